"""Float64 oracle of the Bokenex family: one plain function per mechanism, whole sequences only, no cache.

It shares nothing with the product path (dnet_b200/core/models/seqmix.py, libdnet_b200_seq): attention walks the rows
one by one over an explicit list of visible positions, experts are applied token by token.

Notation: T tokens, W width, H query heads on G key / value heads, ``m`` the residual factor.

    x0 = embed[token] + pos[position]
    h = g x / rms(x);   x <- x + m (mixer(h) + ff(h))       (one norm a layer, both sublayers read its output)
    logits = head . (g_f x / rms(x))
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F64 = torch.float64


# -- norms -----------------------------------------------------------------------------------------------------------
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def scalar_rms_norm(x: torch.Tensor, g: torch.Tensor, eps: float) -> torch.Tensor:
    """one number g for all coordinates"""
    return unit_rms(x, eps) * g.reshape(())


def head_rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """x [T, heads, d], one weight [d] for all heads"""
    return unit_rms(x, eps) * w


# -- embedding ---------------------------------------------------------------------------------------------------------
def embed(tokens: List[int], table: torch.Tensor, pos: torch.Tensor) -> torch.Tensor:
    return torch.stack([table[t] + pos[i] for i, t in enumerate(tokens)])


# -- short causal convolution --------------------------------------------------------------------------------------------
def short_convolution(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start"""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


# -- attention -----------------------------------------------------------------------------------------------------------
def visible(i: int, size: int) -> List[int]:
    """positions that the query at i sees: itself and the size - 1 before it (size 0: all before it)"""
    return [j for j in range(i + 1) if size <= 0 or i - j < size]


def distance_bias(d: torch.Tensor, r1: torch.Tensor, r2: torch.Tensor) -> torch.Tensor:
    """d [n] distances -> [H, n], what is taken off the scores"""
    return r1[:, None] * torch.log(1.0 + r2[:, None] * d[None, :])


def key_weights(scores: torch.Tensor, pb: torch.Tensor) -> torch.Tensor:
    """scores [H, n] of the visible keys -> their weights: a sigmoid each, nothing is divided by a sum"""
    return 1.0 / (1.0 + torch.exp(-(scores + pb[:, None])))


def sigmoid_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, size: int, r1, r2, pb) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]"""
    T, H, _ = q.shape
    G = k.shape[1]
    of = torch.tensor([h // (H // G) for h in range(H)])
    out = []
    for i in range(T):
        js = visible(i, size)
        kk, vv = k[js][:, of], v[js][:, of]                                   # [n, H, d]
        s = torch.einsum("hd,nhd->hn", q[i], kk) * scale
        s = s - distance_bias(torch.tensor([float(i - j) for j in js], dtype=F64), r1, r2)
        out.append(torch.einsum("hn,nhd->hd", key_weights(s, pb), vv))
    return torch.stack(out)


def attention_mixer(h: torch.Tensor, mx: dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, dk = mx["heads"], mx["kv_heads"], mx["dim"]
    dv = mx.get("vdim", dk)
    u = {c: h @ w[p + c].T for c in "qkv"}
    if mx.get("conv"):
        u = {c: short_convolution(u[c], w[p + c + ".conv"]) for c in "qkv"}
    q = head_rms_norm(u["q"].reshape(T, H, dk), w[p + "q.norm"], eps)
    k = head_rms_norm(u["k"].reshape(T, G, dk), w[p + "k.norm"], eps)
    o = sigmoid_attention(q, k, u["v"].reshape(T, G, dv), float(mx["scale"]), int((mx.get("mask") or {}).get("size", 0)),
                          w[p + "r1"], w[p + "r2"], w[p + "pb"])
    return o.reshape(T, H * dv) @ w[p + "o"].T


# -- feed-forward -----------------------------------------------------------------------------------------------------------
def squared_relu(z: torch.Tensor) -> torch.Tensor:
    return z.clamp_min(0.0) ** 2


def two_layer(h, up, down):
    return squared_relu(h @ up.T) @ down.T


def route(h: torch.Tensor, router: torch.Tensor, top: int, scale: float) -> Tuple[List[int], List[float]]:
    """one token [W] -> the chosen experts and their weights"""
    s = [1.0 / (1.0 + math.exp(-float(z))) for z in router @ h]
    chosen = sorted(range(len(s)), key=lambda e: (-s[e], e))[:top]
    total = sum(s[e] for e in chosen) + 1e-20
    return chosen, [s[e] / total * scale for e in chosen]


def routed(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    r = mlp["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(*route(h[t], w[p + "router"], r["top"], float(r.get("scale", 1.0)))):
            out[t] += a * two_layer(h[t], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
    return out


def feed_forward(h: torch.Tensor, mlp: Optional[dict], w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    if not mlp:
        return torch.zeros_like(h)
    if mlp["kind"] == "moe":
        return routed(h, mlp, w, p)
    return two_layer(h, w[p + "up"], w[p + "down"])


# -- the model ---------------------------------------------------------------------------------------------------------------
def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], layers_out: Optional[list] = None) -> torch.Tensor:
    """logits [T, vocab] in float64; layers_out collects the residual after every layer"""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps, m = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x = embed(tokens, w["embed"], w["pos"])
    for i, L in enumerate(cfg["layers"]):
        h = scalar_rms_norm(x, w[f"l{i}.norm1"], eps)
        x = x + m * (attention_mixer(h, L["mixer"], w, f"l{i}.mix.", eps) + feed_forward(h, L.get("mlp"), w, f"l{i}.mlp."))
        if layers_out is not None:
            layers_out.append(x.clone())
    return scalar_rms_norm(x, w["final.norm"], eps) @ w["head"].T


# -- random checkpoints ---------------------------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    W, V = cfg["width"], cfg["vocab"]
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, W), "pos": (cfg["max_positions"], W), "final.norm": (), "head": (V, W)}
    for i, L in enumerate(cfg["layers"]):
        mx, p = L["mixer"], f"l{i}."
        H, G, dk = mx["heads"], mx["kv_heads"], mx["dim"]
        dv = mx.get("vdim", dk)
        rows = {"q": H * dk, "k": G * dk, "v": G * dv}
        out[p + "norm1"] = ()
        for c in "qkv":
            out[p + "mix." + c] = (rows[c], W)
            if mx.get("conv"):
                out[p + "mix." + c + ".conv"] = (rows[c], mx["conv"])
        out[p + "mix.q.norm"] = out[p + "mix.k.norm"] = (dk,)
        out[p + "mix.r1"] = out[p + "mix.r2"] = out[p + "mix.pb"] = (H,)
        out[p + "mix.o"] = (W, H * dv)
        mlp = L.get("mlp")
        if mlp and mlp["kind"] == "moe":
            out[p + "mlp.router"] = (mlp["router"]["experts"], W)
            for e in range(mlp["router"]["experts"]):
                out[f"{p}mlp.e{e}.up"], out[f"{p}mlp.e{e}.down"] = (mlp["expert"]["ff"], W), (W, mlp["expert"]["ff"])
        elif mlp:
            out[p + "mlp.up"], out[p + "mlp.down"] = (mlp["ff"], W), (W, mlp["ff"])
    return out


def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """fp32 tensors holding bf16 values; scalars of the norms away from one, distance rates and weight offsets of both kinds"""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        leaf = name.split(".", 1)[-1]
        if leaf in ("norm1", "norm") or name == "final.norm":
            t = 0.8 + 0.3 * t.abs()
        elif leaf.endswith(".norm"):
            t = 1.0 + 0.2 * t
        elif leaf == "mix.r1":
            t = 0.3 + 0.4 * t.abs()
        elif leaf == "mix.r2":
            t = 0.1 + 0.5 * t.abs()
        elif leaf == "mix.pb":
            t = -1.0 + 0.7 * t
        elif leaf.endswith(".conv"):
            t = t * 0.5
        elif name in ("embed", "pos"):
            t = t * (0.3 if name == "pos" else 1.0)
        else:
            t = t * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16).float()
    return out
