"""Float64 oracle of the Tuguvik family: one plain function per mechanism, whole sequences only, no cache.

It shares nothing with the product path (dnet_b200/core/models/seqmix.py, libdnet_b200_seq): keys and values are formed
per head from the latent of every position, the two maps of a differential attention are two separate softmaxes over a dense
[T, T] table whose visible places are listed query by query, and nothing is absorbed, permuted or paged.

Notation: T tokens, W width, H query heads on G key / value heads; dyt(x) = tanh(alpha x) w + b; rms(x) = x / sqrt(mean(x^2) + eps).

    x0 = embed[tokens]
    x <- x + ls1 * mixer(dyt1(x));   x <- x + ls2 * ff(dyt2(x))
    x <- x + rms(W_p (gelu(W_g x) * e_i[token])) * w        (a row of a token table per layer)
    logits = head . dyt(x)
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F64 = torch.float64


# -- elementwise ---------------------------------------------------------------------------------------------------------
def dyt(x, w, b, alpha):
    return torch.tanh(alpha * x) * w + b


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# -- rotary ------------------------------------------------------------------------------------------------------------
def plain_frequencies(dims: int, base: float) -> List[float]:
    return [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]


def ramped_frequencies(dims: int, base: float, sc: dict) -> Tuple[List[float], float]:
    """pairs below `lo` keep their frequency, pairs from `hi` on get it divided by the factor, a straight line between;
    the second result multiplies cos and sin"""
    def pair_of(turns: float) -> float:       # the pair that makes this many turns over the original length
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(pair_of(sc["fast"])), 0), min(math.ceil(pair_of(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        r = min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001)))
        out.append(f / sc["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def banded_frequencies(dims: int, base: float, sc: dict) -> List[float]:
    """by wavelength: short ones keep their frequency, long ones are divided by the factor, a blend between"""
    out = []
    for f in plain_frequencies(dims, base):
        wl = 2.0 * math.pi / f
        if wl < sc["original"] / sc["high"]:
            out.append(f)
        elif wl > sc["original"] / sc["low"]:
            out.append(f / sc["factor"])
        else:
            s = (sc["original"] / wl - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - s) * f / sc["factor"] + s * f)
    return out


def turn(x: torch.Tensor, freqs: List[float], mult: float, layout: str) -> torch.Tensor:
    """x [T, ..., d], row t at position t: the first 2 len(freqs) numbers of the last axis turn; pair i is (2i, 2i + 1)
    for 'interleaved' and (i, i + len(freqs)) for 'half'"""
    n = len(freqs)
    if n == 0:
        return x
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * torch.tensor(freqs, dtype=F64)[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [n]
    cs, sn = (torch.cos(ang) * mult).reshape(shape), (torch.sin(ang) * mult).reshape(shape)
    ia = torch.arange(n) * 2 if layout == "interleaved" else torch.arange(n)
    ib = ia + 1 if layout == "interleaved" else ia + n
    out = x.clone()
    u, v = x[..., ia], x[..., ib]
    out[..., ia] = u * cs - v * sn
    out[..., ib] = v * cs + u * sn
    return out


def rotation(rot: Optional[dict]) -> Tuple[List[float], float]:
    """frequencies and multiplier of a mixer's `rot` entry"""
    rot = rot or {}
    dims, base, sc = int(rot.get("dims", 0) or 0), float(rot.get("base", 10000.0)), rot.get("scaling")
    if dims == 0:
        return [], 1.0
    if not sc:
        return plain_frequencies(dims, base), 1.0
    if "fast" in sc:
        return ramped_frequencies(dims, base, sc)
    return banded_frequencies(dims, base, sc), 1.0


# -- which keys a query sees -----------------------------------------------------------------------------------------------
def visible(i: int, mask: Optional[dict]) -> List[int]:
    """size 0 or no mask: every earlier key; keep_first: these positions stay visible behind the window"""
    mask = mask or {}
    size, keep = int(mask.get("size", 0) or 0), int(mask.get("keep_first", 0) or 0)
    return [j for j in range(i + 1) if size <= 0 or i - j < size or j < keep]


def visible_table(T: int, mask: Optional[dict]) -> torch.Tensor:
    """[T, T] bool, row i true at visible(i)"""
    out = torch.zeros(T, T, dtype=torch.bool)
    for i in range(T):
        out[i, visible(i, mask)] = True
    return out


def weights_with_sink(s: torch.Tensor, vis: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """softmax over the visible scores of every row of s [T, T]; the sink adds exp(sink) to every denominator"""
    s = s.masked_fill(~vis, -math.inf)
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + (torch.exp(sink - m) if sink is not None else 0.0))


# -- mixers ------------------------------------------------------------------------------------------------------------------
def latent_rows(w: Dict[str, torch.Tensor], p: str, mx: dict, h: torch.Tensor, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """what a layer's cache holds: the normed latent [T, R] and the rotated key part [T, dr]"""
    R = mx["kv_rank"]
    down = h @ w[p + "mix.dkv"].T
    freqs, mult = rotation(mx.get("rot"))
    return unit_rms(down[:, :R], eps) * w[p + "mix.dkv.norm"], turn(down[:, R:], freqs, mult, "interleaved")


def latent_attention(w, p: str, mx: dict, h: torch.Tensor, eps: float, rows: Tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
    H, dn, dv, dr = mx["heads"], mx["dim"], mx.get("vdim", mx["dim"]), mx["rot_dim"]
    T = h.shape[0]
    lat, k_rot = rows
    q = (unit_rms(h @ w[p + "mix.dq"].T, eps) * w[p + "mix.dq.norm"]) @ w[p + "mix.uq"].T
    q = q.reshape(T, H, dn + dr)
    freqs, mult = rotation(mx.get("rot"))
    q_rot = turn(q[:, :, dn:], freqs, mult, "interleaved")
    k_un = (lat @ w[p + "mix.uk"].T).reshape(T, H, dn)
    val = (lat @ w[p + "mix.uv"].T).reshape(T, H, dv)
    gate = torch.sigmoid(h @ w[p + "mix.g"].T)
    vis = visible_table(T, mx.get("mask"))
    out = torch.zeros(T, H, dv, dtype=F64)
    for hh in range(H):
        s = (q[:, hh, :dn] @ k_un[:, hh].T + q_rot[:, hh] @ k_rot.T) * float(mx["scale"])
        out[:, hh] = weights_with_sink(s, vis, w[p + "mix.sink"][hh]) @ val[:, hh] * gate[:, hh, None]
    return out.reshape(T, H * dv) @ w[p + "mix.o"].T


def diff_lambda(w, p: str, diff: float) -> torch.Tensor:
    return torch.exp((w[p + "mix.lq1"] * w[p + "mix.lk1"]).sum()) - torch.exp((w[p + "mix.lq2"] * w[p + "mix.lk2"]).sum()) + diff


def diff_attention(w, p: str, mx: dict, h: torch.Tensor, eps: float) -> torch.Tensor:
    H, G, dk, dv, diff = mx["heads"], mx["kv_heads"], mx["dim"], mx.get("vdim", mx["dim"]), float(mx["diff"])
    T = h.shape[0]
    freqs, mult = rotation(mx.get("rot"))
    q = turn((h @ w[p + "mix.q"].T).reshape(T, H, 2, dk), freqs, mult, "half")
    k = turn((h @ w[p + "mix.k"].T).reshape(T, G, 2, dk), freqs, mult, "half")
    v = (h @ w[p + "mix.v"].T).reshape(T, G, dv)
    lam = diff_lambda(w, p, diff)
    vis = visible_table(T, mx.get("mask"))
    out = torch.zeros(T, H, dv, dtype=F64)
    for hh in range(H):
        g = hh // (H // G)
        a = [weights_with_sink(q[:, hh, m] @ k[:, g, m].T * float(mx["scale"]), vis, None) @ v[:, g] for m in range(2)]
        out[:, hh] = unit_rms(a[0] - lam * a[1], eps) * (1.0 - diff)
    return out.reshape(T, H * dv) @ w[p + "mix.o"].T


# -- feed-forward and token input -----------------------------------------------------------------------------------------------
def swiglu_ff(w, p: str, h: torch.Tensor) -> torch.Tensor:
    return (silu(h @ w[p + "mlp.gate"].T) * (h @ w[p + "mlp.up"].T)) @ w[p + "mlp.down"].T


def token_input(w, p: str, i: int, dim: int, tokens: torch.Tensor, x: torch.Tensor, eps: float) -> torch.Tensor:
    e = w["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return unit_rms(y, eps) * w[p + "side.norm"]


# -- the model ---------------------------------------------------------------------------------------------------------------
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, layers_out: Optional[list] = None) -> torch.Tensor:
    """logits [T, vocab] of a whole sequence; layers_out collects the residual after every layer"""
    w = {k: v.to(F64) for k, v in w.items()}
    eps = float((cfg.get("norm") or {}).get("eps", 1e-6))
    ids = torch.as_tensor(tokens, dtype=torch.long)
    side = int((cfg.get("token_side") or {}).get("dim", 0))

    def norm(name: str, x):
        return dyt(x, w[name], w[name + ".b"], w[name + ".alpha"])

    x = w["embed"][ids]
    rows: Dict[int, Tuple[torch.Tensor, torch.Tensor]] = {}
    for i, L in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", L["mixer"]
        h = norm(p + "norm1", x)
        if L["type"] == "latent_attention":
            src = mx.get("kv_from")
            if src is None:
                rows[i] = latent_rows(w, p, mx, h, eps)
            y = latent_attention(w, p, mx, h, eps, rows[i if src is None else src])
        else:
            y = diff_attention(w, p, mx, h, eps)
        x = x + y * w[p + "ls1"]
        if L.get("mlp"):
            x = x + swiglu_ff(w, p, norm(p + "norm2", x)) * w[p + "ls2"]
        if side:
            x = x + token_input(w, p, i, side, ids, x, eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm("final.norm", x) @ w["head"].T


# -- checkpoints ---------------------------------------------------------------------------------------------------------------
def tensor_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    W, V = int(cfg["width"]), int(cfg["vocab"])
    side = int((cfg.get("token_side") or {}).get("dim", 0))
    out: Dict[str, Tuple[int, ...]] = {"embed": (V, W), "head": (V, W)}

    def norm(name: str):
        out[name], out[name + ".b"], out[name + ".alpha"] = (W,), (W,), ()

    norm("final.norm")
    if side:
        out["side.embed"] = (V, len(cfg["layers"]) * side)
    for i, L in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", L["mixer"]
        H, dk, dv = mx["heads"], mx["dim"], mx.get("vdim", mx["dim"])
        norm(p + "norm1")
        out[p + "ls1"] = (W,)
        if L["type"] == "latent_attention":
            R, Q, dr = mx["kv_rank"], mx["q_rank"], mx["rot_dim"]
            out[p + "mix.dq"], out[p + "mix.dq.norm"], out[p + "mix.uq"] = (Q, W), (Q,), (H * (dk + dr), Q)
            if mx.get("kv_from") is None:
                out[p + "mix.dkv"], out[p + "mix.dkv.norm"] = (R + dr, W), (R,)
            out[p + "mix.uk"], out[p + "mix.uv"] = (H * dk, R), (H * dv, R)
            out[p + "mix.sink"], out[p + "mix.g"] = (H,), (H, W)
        else:
            G = mx["kv_heads"]
            out[p + "mix.q"], out[p + "mix.k"], out[p + "mix.v"] = (H * 2 * dk, W), (G * 2 * dk, W), (G * dv, W)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                out[p + "mix." + n] = (dk,)
        out[p + "mix.o"] = (W, H * dv)
        if L.get("mlp"):
            F = int(L["mlp"]["ff"])
            norm(p + "norm2")
            out[p + "ls2"] = (W,)
            out[p + "mlp.gate"] = out[p + "mlp.up"] = (F, W)
            out[p + "mlp.down"] = (W, F)
        if side:
            out[p + "side.gate"], out[p + "side.proj"], out[p + "side.norm"] = (side, W), (W, side), (W,)
    return out


def random_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """fp32 tensors whose values are exact in bf16: matrices ~ N(0, 1/fan_in), norm weights and layer scales around one,
    alphas around 0.7 and different in every norm, sinks of the size of a score"""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        if name.endswith(".alpha"):
            t = 0.7 + 0.2 * r
        elif name.endswith((".dkv.norm", ".dq.norm", "norm1", "norm2", "final.norm")):
            t = 1.0 + 0.2 * r
        elif name.endswith((".ls1", ".ls2")):
            t = 0.8 + 0.3 * r
        elif name.endswith("side.norm"):
            t = 0.5 + 0.2 * r
        elif name.endswith("norm.b") or name.endswith((".norm1.b", ".norm2.b")):
            t = 0.2 * r
        elif name.endswith(".sink"):
            t = 1.0 + 0.7 * r
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = 0.6 * r / math.sqrt(shape[0]) + 0.1
        elif name in ("embed", "side.embed"):
            t = r
        elif name.endswith(("mix.uq", "mix.q", "mix.k")):
            t = 1.6 * r / math.sqrt(shape[-1])
        else:
            t = r / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out
