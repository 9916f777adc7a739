"""The Tuguvik family (core/models/seqmix.py TuguvikRingModel, shard/batching.py, libdnet_b200_seq) against the float64 oracle
(oracle/tuguvik_oracle.py): every mechanism alone with the residual after each layer, then portions, batches, page and slot
reuse, keys at the edges of the windows, among the kept first tokens and far away with scores made to stand out, sinks, lambda,
rotation, long decoding and greedy generation through the batcher's token loop.  fp32 runs are held to 2e-4 of the logits'
spread row by row; bf16 runs to 4e-2 of the spread over all rows together."""
from __future__ import annotations

import copy

import pytest
import torch

from oracle import tuguvik_oracle as to

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-4, "bfloat16": 4e-2}

DENSE = {"kind": "dense", "ff": 72}
RAMP = {"factor": 3.0, "original": 40, "fast": 8.0, "slow": 0.5}
BANDS = {"factor": 5.0, "low": 1.0, "high": 3.0, "original": 60}


def rot(base, dims, scaling=None):
    return {"base": base, "dims": dims, **({"scaling": scaling} if scaling else {})}


def lat(mlp=None, **kw):
    mx = {"heads": 3, "dim": 24, "rot_dim": 8, "vdim": 16, "kv_rank": 40, "q_rank": 28, "scale": 0.2, "rot": rot(500.0, 8, RAMP), "mask": {"size": 21}}
    mx.update(kw)
    if "rot_dim" in kw and "rot" not in kw:
        mx["rot"] = rot(500.0, kw["rot_dim"], RAMP)
    return {"type": "latent_attention", "mixer": {k: v for k, v in mx.items() if v is not None}, "mlp": mlp}


def dif(mlp=None, size=26, keep=3, **kw):
    mx = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.25, "diff": 0.35, "rot": rot(300.0, 12, BANDS)}
    if size:
        mx["mask"] = {"size": size, "keep_first": keep}
    mx.update(kw)
    return {"type": "attention", "mixer": {k: v for k, v in mx.items() if v is not None}, "mlp": mlp}


def config(layers, width=48, vocab=96, eps=1e-5, side=10):
    return {"architecture": "Tuguvik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            **({"token_side": {"dim": side}} if side else {})}


FULL = config([dif(DENSE), lat(DENSE), lat(None, kv_from=1, heads=2, mask={"size": 70}, vdim=24), dif(None, size=70, keep=9, heads=2, kv_heads=2, dim=12, rot=rot(300.0, 12)),
               lat(DENSE, kv_from=1, dim=10, q_rank=17)])


class Rig:
    """a model + batcher on the GPU and the oracle's view of the same weights"""

    def __init__(self, cfg, dtype="float32", seed=1, max_tokens=1024, max_seqs=4, max_batch_tokens=512, weights=None):
        from dnet_b200.shard.batching import SequenceBatcher, load_model
        from dnet_b200.utils.model import HostDictSource

        self.cfg, self.dtype = cfg, dtype
        self.w = weights if weights is not None else to.random_weights(cfg, seed)
        self.model = load_model(HostDictSource({k: v.to(torch.bfloat16) for k, v in self.w.items()}, cfg), dtype, max_tokens=max_tokens,
                                max_seqs=max_seqs, max_batch_tokens=max_batch_tokens)
        self.eng = SequenceBatcher(self.model)

    def oracle(self, tokens, layers_out=None):
        return to.forward(self.cfg, self.w, tokens, layers_out)

    def close(self):
        self.eng.close()
        self.model.destroy()

    def __enter__(self):
        return self

    def __exit__(self, *a):
        self.close()


def err(got: torch.Tensor, ref: torch.Tensor) -> float:
    """worst row of: rms of the difference (mean removed) over the rms spread of the reference row"""
    d = got.double().cpu() - ref.double()
    d = d - d.mean(-1, keepdim=True)
    r = ref.double() - ref.double().mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / r.pow(2).mean(-1).sqrt().clamp_min(1e-9)).max())


def err16(got: torch.Tensor, ref: torch.Tensor) -> float:
    """rms of the difference (row means removed) over the rms spread of the reference, all rows together"""
    d = got.double().cpu() - ref.double()
    d = d - d.mean(-1, keepdim=True)
    r = ref.double() - ref.double().mean(-1, keepdim=True)
    return float(d.pow(2).mean().sqrt() / r.pow(2).mean().sqrt())


def off(dtype):
    return err16 if dtype == "bfloat16" else err


def toks(n, vocab=96, seed=0):
    g = torch.Generator().manual_seed(12000 + seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def run_schedule(rig: Rig, tokens, cuts, rid="r"):
    """feed tokens in portions of the given sizes (the rest one by one); logits of every position"""
    out, at = [], 0
    for c in list(cuts) + [1] * len(tokens):
        if at >= len(tokens):
            break
        part = tokens[at:at + c]
        out.append(rig.eng.step([(rid, part, list(range(len(part))))]))
        at += len(part)
    rig.eng.finish(rid)
    return torch.cat(out)


# -- each mechanism alone -----------------------------------------------------------------------------------------------
MECHANISMS = {
    "latent": config([lat()], side=None),
    "latent_one_head": config([lat(heads=1, dim=32, vdim=40)], side=None),
    "latent_odd_sizes": config([lat(heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=21, q_rank=11), lat(heads=2, dim=5, rot_dim=2, vdim=9, kv_rank=13, q_rank=5)], side=None),
    "latent_equal_sizes": config([lat(heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=16, q_rank=16)], side=None),
    "latent_wide": config([lat(heads=2, dim=8, kv_rank=288, vdim=24), lat(heads=2, dim=160, rot_dim=64, vdim=136, kv_rank=96, q_rank=70)], width=64, side=None),
    "latent_unscaled_rotation": config([lat(rot=rot(500.0, 8))], side=None),
    "latent_ramp_of_one_factor": config([lat(rot=rot(500.0, 8, {**RAMP, "factor": 1.0}))], side=None),
    "latent_ramp_below_and_beyond_the_pairs": config([lat(rot_dim=16, rot=rot(10.0, 16, {"factor": 4.0, "original": 4000, "fast": 900.0, "slow": 1e-3})),
                                                      lat(rot_dim=16, rot=rot(1e6, 16, {"factor": 4.0, "original": 30, "fast": 32.0, "slow": 1.0}))], side=None),
    "latent_windows": config([lat(mask={"size": 1}), lat(mask={"size": 64}), lat(mask={"size": 65}), lat(mask={"size": 4000}), lat(mask=None)], side=None),
    "latent_borrowed_rows": config([lat(), dif(), lat(kv_from=0, heads=5, dim=12, vdim=8, q_rank=9, mask={"size": 50}, scale=0.4), lat(), lat(kv_from=0), lat(kv_from=3)], side=None),
    "differential": config([dif()], side=None),
    "differential_one_head": config([dif(heads=1, kv_heads=1, dim=32, vdim=40)], side=None),
    "differential_one_key_head": config([dif(heads=6, kv_heads=1)], side=None),
    "differential_as_many_key_heads": config([dif(heads=3, kv_heads=3, dim=8, vdim=8, rot=rot(300.0, 8, BANDS))], side=None),
    "differential_odd_sizes": config([dif(heads=3, kv_heads=1, dim=7, vdim=5, rot=rot(30.0, 6, BANDS)), dif(heads=2, kv_heads=2, dim=10, vdim=11, rot=rot(30.0, 2, BANDS))], side=None),
    "differential_large_heads": config([dif(heads=2, kv_heads=1, dim=64, vdim=128, scale=0.12), dif(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.1),
                                        dif(heads=2, kv_heads=1, dim=96, vdim=200, scale=0.1)], width=64, side=None),
    "differential_no_rotation": config([dif(rot=None)], side=None),
    "differential_whole_head_turns": config([dif(rot=rot(300.0, 16, BANDS))], side=None),
    "differential_unscaled_rotation": config([dif(rot=rot(300.0, 12))], side=None),
    "differential_narrow_bands": config([dif(rot=rot(300.0, 12, {"factor": 2.0, "low": 1.0, "high": 1.25, "original": 200}))], side=None),
    "differential_all_pairs_long_or_short": config([dif(rot=rot(300.0, 12, {"factor": 2.0, "low": 1.0, "high": 4.0, "original": 4})),
                                                    dif(rot=rot(300.0, 12, {"factor": 2.0, "low": 1.0, "high": 4.0, "original": 90000}))], side=None),
    "differential_diff_zero": config([dif(diff=0.0)], side=None),
    "window_of_one": config([dif(size=1, keep=0), dif(size=1, keep=1), dif(size=2, keep=5)], side=None),
    "windows_about_a_page": config([dif(size=64, keep=1), dif(size=65, keep=64), dif(size=63, keep=65)], side=None),
    "kept_tokens_beyond_the_window": config([dif(size=5, keep=100), dif(size=20, keep=40)], side=None),
    "window_wider_than_the_prompt": config([dif(size=4000, keep=4)], side=None),
    "no_window": config([dif(size=None)], side=None),
    "dense": config([lat(DENSE), dif(DENSE)], side=None),
    "dense_wide": config([dif({"kind": "dense", "ff": 200})], side=None),
    "token_side": config([dif(), lat(DENSE), dif(DENSE)]),
    "token_side_of_one": config([dif(DENSE), lat()], side=1),
    "token_side_wide": config([lat(DENSE), dif()], side=64),
    "large_eps": config([dif(DENSE), lat(None)], eps=0.3),
    "every_kind_of_layer": FULL,
}


@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_alone_fp32(name):
    cfg = MECHANISMS[name]
    t = toks(150, seed=3)
    with Rig(cfg, "float32", seed=sum(map(ord, name))) as rig:
        layers = []
        ref = rig.oracle(t, layers)
        got, trace = rig.eng.step([("a", t, list(range(len(t))))], layer_trace=True)
        assert trace.shape[0] == len(layers)
        for i, l in enumerate(layers):
            assert err(trace[i], l) < TOL["float32"], f"{name}: residual after layer {i}"
        assert err(got, ref) < TOL["float32"]
        rig.eng.finish("a")
        assert err(run_schedule(rig, t[:100], [30, 7, 2, 41]), ref[:100]) < TOL["float32"], f"{name}: portions and decoding"


@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_alone_bf16(name):
    """(two sharp layers in a row amplify rounding: 2 x the tolerance)"""
    cfg = MECHANISMS[name]
    t = toks(150, seed=4)
    with Rig(cfg, "bfloat16", seed=sum(map(ord, name))) as rig:
        ref = rig.oracle(t)
        assert err16(run_schedule(rig, t, [150]), ref) < 2 * TOL["bfloat16"]
        assert err16(run_schedule(rig, t, [50, 17, 2, 41]), ref) < 2 * TOL["bfloat16"]


# -- sizes --------------------------------------------------------------------------------------------------------------
def test_sizes_on_the_tensor_core_products():
    """width and projection sizes in multiples of 64: bf16 prompt portions take the tcgen05 products with their joining epilogues and
    the MMA attention"""
    cfg = config([lat({"kind": "dense", "ff": 256}, heads=4, dim=64, rot_dim=32, vdim=32, kv_rank=96, q_rank=64, mask={"size": 100}),
                  dif({"kind": "dense", "ff": 192}, heads=4, kv_heads=2, dim=32, vdim=64, size=33, keep=5, rot=rot(300.0, 32, BANDS)),
                  lat(None, heads=8, dim=32, rot_dim=32, vdim=64, kv_rank=96, q_rank=128, kv_from=0)], width=128, vocab=192, side=64)
    t = toks(300, vocab=192, seed=6)
    with Rig(cfg, "bfloat16") as rig:
        ref = rig.oracle(t)
        assert err16(run_schedule(rig, t, [300]), ref) < TOL["bfloat16"]
        assert err16(run_schedule(rig, t, [130, 17, 64, 2, 70]), ref) < TOL["bfloat16"]


@pytest.mark.parametrize("dk,dv", [(16, 16), (32, 48), (24, 128), (56, 24), (64, 64), (48, 96), (96, 32), (128, 64), (64, 128), (112, 120), (128, 128)])
def test_every_pair_of_head_sizes_of_the_tiles(dk, dv):
    cfg = config([dif(size=75, keep=6, heads=4, kv_heads=2, dim=dk, vdim=dv, scale=1.2 * dk ** -0.5, rot=rot(200.0, dk // 2, BANDS))], width=64, side=None)
    t = toks(180, seed=17)
    with Rig(cfg, "bfloat16") as rig:
        ref = rig.oracle(t)
        assert err16(run_schedule(rig, t, [180]), ref) < TOL["bfloat16"]
        assert err16(run_schedule(rig, t, [100, 2, 70]), ref) < TOL["bfloat16"]


@pytest.mark.parametrize("H,G,dk,dv,size,keep", [(1, 1, 64, 64, 50, 3), (4, 2, 128, 64, 200, 4), (6, 2, 64, 128, 64, 64), (6, 1, 64, 128, 65, 130), (16, 1, 64, 64, 33, 1),
                                                 (20, 1, 64, 64, 300, 7), (8, 8, 64, 64, None, 0), (34, 2, 64, 128, 130, 20), (4, 1, 128, 128, 1, 2)])
def test_prompt_attention_of_wide_heads(H, G, dk, dv, size, keep):
    """heads of 64 / 128 with one, some and many query heads a key head, windows of one token, about a page, several tiles and none, kept
    tokens inside a page and beyond two; whole, in portions that start inside pages and tiles, and unequal entries side by side"""
    cfg = config([dif(size=size, keep=keep, heads=H, kv_heads=G, dim=dk, vdim=dv, scale=1.2 * dk ** -0.5, rot=rot(400.0, dk // 2, BANDS))], width=64, side=None)
    t = toks(330, seed=500 + H)
    with Rig(cfg, "bfloat16", max_tokens=2048, max_batch_tokens=1024) as rig:
        ref = rig.oracle(t)
        assert err16(run_schedule(rig, t, [330]), ref) < TOL["bfloat16"]
        assert err16(run_schedule(rig, t, [37, 16, 2, 90, 129, 50]), ref) < TOL["bfloat16"]
        rig.eng.step([("a", t[:100], []), ("b", t[:20], [])])
        lg = rig.eng.step([("a", t[100:231], list(range(131))), ("b", t[20:21], [0]), ("c", t[:17], list(range(17)))])
        assert err16(lg, torch.cat([ref[100:231], ref[20:21], ref[:17]])) < TOL["bfloat16"]


def test_prompt_attention_in_pages_that_were_used():
    """the last page of a prompt holds rows of the request that had it before: they must not enter (values four times as large)"""
    cfg = config([dif(DENSE, size=200, keep=4, heads=4, kv_heads=2, dim=64, vdim=64, scale=0.15), lat(None, mask={"size": 90})], width=64)
    w = to.random_weights(cfg, 520)
    w["l0.mix.v"] = w["l0.mix.v"] * 4
    with Rig(cfg, "bfloat16", weights=w, max_tokens=256, max_seqs=2) as rig:
        for n, k in ((250, 0), (17, 1), (70, 2), (129, 3), (190, 4)):
            t = toks(n, seed=521 + k)
            assert err16(run_schedule(rig, t, [n]), rig.oracle(t)) < TOL["bfloat16"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_allow_no_wide_loads(dtype):
    """width, head, rank, feed-forward, side and vocabulary sizes that are multiples of neither 4 nor 8: the scalar forms of every kernel"""
    cfg = config([dif({"kind": "dense", "ff": 35}, size=19, heads=3, kv_heads=1, dim=7, vdim=5, rot=rot(30.0, 6, BANDS)),
                  lat({"kind": "dense", "ff": 9}, heads=2, dim=9, rot_dim=6, vdim=13, kv_rank=21, q_rank=11)], width=50, vocab=77, side=7)
    t = toks(120, vocab=77, seed=160)
    with Rig(cfg, dtype) as rig:
        ref = rig.oracle(t)
        assert off(dtype)(run_schedule(rig, t, [120]), ref) < TOL[dtype]
        assert off(dtype)(run_schedule(rig, t, [70, 2, 20]), ref) < TOL[dtype]


LAYER_SIZED = {
    "w384": config([dif({"kind": "dense", "ff": 640}, size=90, keep=5, heads=6, kv_heads=2, dim=64, vdim=48, scale=0.11, rot=rot(1e4, 32, BANDS)),
                    lat({"kind": "dense", "ff": 512}, heads=6, dim=48, rot_dim=32, vdim=64, kv_rank=128, q_rank=192, scale=0.12, mask={"size": 70}),
                    dif(None, size=64, keep=64, heads=4, kv_heads=1, dim=96, vdim=64, scale=0.1, rot=rot(1e4, 48))], width=384, vocab=640, side=64),
    "w512": config([lat({"kind": "dense", "ff": 1024}, heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=320, scale=0.07, mask={"size": 150}),
                    dif({"kind": "dense", "ff": 768}, size=150, keep=2, heads=4, kv_heads=2, dim=64, vdim=128, scale=0.12, rot=rot(1e5, 64, BANDS)),
                    lat(None, heads=8, dim=64, rot_dim=64, vdim=64, kv_rank=512, q_rank=256, scale=0.09, kv_from=0, mask={"size": 33}),
                    dif({"kind": "dense", "ff": 512}, size=None, heads=8, kv_heads=4, dim=64, vdim=64, scale=0.12)], width=512, vocab=1000, side=128),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(LAYER_SIZED))
def test_layer_sized_models(name, dtype):
    cfg = LAYER_SIZED[name]
    V = cfg["vocab"]
    t = toks(210, vocab=V, seed=300)
    w = to.random_weights(cfg, 301)
    with Rig(cfg, dtype, weights=w) as rig:
        ref = to.forward(cfg, w, t)
        e = off(dtype)
        whole = run_schedule(rig, t, [len(t)])
        assert e(whole, ref) < TOL[dtype]
        cut = run_schedule(rig, t, [100, 2, 64, 17, 5])
        assert e(cut, ref) < TOL[dtype]
        rig.eng.step([("a", t[:100], [])])
        rig.eng.step([("b", t[:37], [])])
        lg = rig.eng.step([("a", t[100:130], list(range(30))), ("b", t[37:38], [0])])      # a portion beside a decoded token
        assert e(lg[:30], ref[100:130]) < TOL[dtype] and e(lg[30:], ref[37:38]) < 2 * TOL[dtype]
        if dtype == "bfloat16":       # and the schedules agree with each other about as well
            assert err16(cut, whole.cpu()) < TOL[dtype] and err16(lg[:30], whole[100:130].cpu()) < TOL[dtype]


# -- schedules ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_against_token_by_token(dtype):
    t = toks(90, seed=7)
    with Rig(FULL, dtype) as rig:
        ref = rig.oracle(t)
        tol = TOL[dtype] * (2 if dtype == "bfloat16" else 1)
        assert off(dtype)(run_schedule(rig, t, []), ref) < tol              # every token alone, from the first
        assert off(dtype)(run_schedule(rig, t, [50]), ref) < tol            # a prompt, then decoding


@pytest.mark.parametrize("cuts", [[2, 2, 2, 3, 5, 64, 1, 2, 40], [39, 2, 41, 2, 63, 1, 64], [128, 2], [1, 1, 1, 2, 200], [20, 1, 21, 22, 2, 19], [12, 9, 14, 30, 11]])
def test_portions_of_any_size(cuts):
    t = toks(230, seed=11)
    with Rig(FULL, "float32") as rig:
        assert err(run_schedule(rig, t, cuts), rig.oracle(t)) < TOL["float32"]


def test_unequal_requests_in_one_batch_equal_each_alone():
    lens = [5, 77, 140, 33]
    seqs = [toks(n, seed=20 + i) for i, n in enumerate(lens)]
    with Rig(FULL, "float32") as rig:
        refs = [rig.oracle(s) for s in seqs]
        at = [0] * 4
        portions = [[2, 3], [40, 2, 35], [64, 64, 12], [1] * 33]
        got = [[] for _ in seqs]
        step = 0
        while any(at[i] < lens[i] for i in range(4)):
            entries = []
            for i in range(4):
                if at[i] < lens[i] and (step + i) % 3 != 2:              # requests sit out some steps
                    n = portions[i][0] if portions[i] else 1
                    portions[i] = portions[i][1:]
                    part = seqs[i][at[i]:at[i] + n]
                    entries.append((f"q{i}", part, list(range(len(part)))))
                    at[i] += len(part)
            step += 1
            if not entries:
                continue
            lg = rig.eng.step(entries)
            row = 0
            for rid, part, _ in entries:
                got[int(rid[1:])].append(lg[row:row + len(part)])
                row += len(part)
        for i in range(4):
            assert err(torch.cat(got[i]), refs[i]) < TOL["float32"], f"request {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [3, 8, 9, 13, 20])
def test_decoding_many_sequences_together(n, dtype):
    """steps of 1 .. 20 single tokens: the few-row products, the tiles, and the decode kernels of both mixers"""
    seqs = [toks(20 + 5 * i, seed=400 + i) for i in range(n)]
    with Rig(FULL, dtype, max_tokens=64 * 3 * n, max_seqs=n) as rig:
        refs = torch.stack([rig.oracle(s)[-3:] for s in seqs])
        rig.eng.step([(f"s{i}", s[:-3], []) for i, s in enumerate(seqs[:n // 2 + 1])])
        for i, s in enumerate(seqs):
            if i > n // 2:
                rig.eng.step([(f"s{i}", s[:-3], [])])
        got = torch.stack([rig.eng.step([(f"s{i}", [s[k]], [0]) for i, s in enumerate(seqs)]) for k in (-3, -2, -1)], dim=1)
        assert off(dtype)(got.flatten(0, 1), refs.flatten(0, 1)) < TOL[dtype] * (2 if dtype == "bfloat16" else 1)


def test_pages_and_slots_are_reused():
    """a pool of 4 pages and 2 slots serves 6 requests two at a time; a request that does not fit is refused without
    disturbing the live ones; a page's old rows never show in its next user"""
    from dnet_b200._cabi import DnError

    with Rig(FULL, "float32", max_tokens=256, max_seqs=2, max_batch_tokens=256) as rig:
        for rnd in range(3):
            a, b = toks(100 + rnd, seed=30 + rnd), toks(120 - rnd, seed=40 + rnd)
            assert rig.eng.step([("a", a[:70], []), ("b", b[:3], [])]) is None
            la = rig.eng.step([("a", a[70:], list(range(len(a) - 70))), ("b", b[3:], list(range(len(b) - 3)))])
            assert err(la[:len(a) - 70], rig.oracle(a)[70:]) < TOL["float32"]
            assert err(la[len(a) - 70:], rig.oracle(b)[3:]) < TOL["float32"]
            assert rig.model.free_pages == 0 and rig.model.free_slots == 0
            with pytest.raises(DnError):
                rig.eng.step([("a", toks(60), [])])                        # a fifth page does not exist
            with pytest.raises(DnError):
                rig.eng.step([("c", [1], [])])                            # nor a third slot
            rig.eng.live.pop("c", None)
            la = rig.eng.step([("a", [7], [0])])                           # the refused steps changed nothing of "a"
            assert err(la, rig.oracle(a + [7])[-1:]) < TOL["float32"]
            rig.eng.finish("a")
            rig.eng.finish("b")
            assert rig.model.free_pages == 4 and rig.model.free_slots == 2


def test_a_layer_that_borrows_rows_takes_no_pages_of_its_own():
    """two models of the same layers, one of which borrows: the borrowing one has one page pool less"""
    a, b = config([lat(), lat()], side=None), config([lat(), lat(kv_from=0)], side=None)
    used = []
    for cfg in (a, b):
        torch.cuda.synchronize()
        free0 = torch.cuda.mem_get_info()[0]
        with Rig(cfg, "float32", max_tokens=64 * 4096):
            used.append(free0 - torch.cuda.mem_get_info()[0])
    row = (40 + 8) * 4
    assert used[0] - used[1] > 0.9 * 64 * 4096 * row


# -- keys at the window's edges, among the kept tokens and far away, with scores made to stand out ------------------------------------
def opposite_setup(layer, seed, vocab=64):
    """One layer in which a query finds the token whose input points the other way: the first head's keys are minus its queries, the
    norm before the mixer has no bias (so it is odd), nothing rotates; a token scores about minus its query's square against itself
    and plus that against a token with the opposite embedding (token 63 is minus token 62)."""
    cfg = config([layer], vocab=vocab, side=None)
    mx = layer["mixer"]
    w = to.random_weights(cfg, seed)
    e = w["embed"].clone()
    e[63] = -e[62]
    w["embed"] = e
    w["l0.norm1.b"] = torch.zeros_like(w["l0.norm1.b"])
    dk = mx["dim"]
    if layer["type"] == "attention":
        w["l0.mix.k"][:dk] = -w["l0.mix.q"][:dk]
    else:
        R, dr = mx["kv_rank"], mx["rot_dim"]
        assert mx["q_rank"] == R
        w["l0.mix.dkv"][:R] = w["l0.mix.dq"]
        w["l0.mix.dkv"][R:] = 0
        w["l0.mix.dq.norm"] = w["l0.mix.dkv.norm"] = torch.ones(R)
        w["l0.mix.uk"][:dk] = -w["l0.mix.uq"][:dk]
    return cfg, w


def edge_layer(kind, size, keep=0, **kw):
    if kind == "latent":
        return lat(heads=2, dim=24, kv_rank=40, q_rank=40, scale=0.35, mask={"size": size} if size else None, **kw)
    return dif(size=size, keep=keep, heads=2, kv_heads=1, **{"dim": 32, "vdim": 16, "scale": 0.3, "rot": None, **kw})


WIDE = {"dim": 64, "vdim": 64, "scale": 0.16}


def edge_setup(kind, size, token_marks=(0, 40, 64, 104, 127, 170), keep=0, **kw):
    """token 63 stands at every position of `token_marks`, token 62 at mark + size - 1 (it just sees the 63) and at mark + size
    (it just does not); all other tokens are below 62"""
    cfg, w = opposite_setup(edge_layer(kind, size, keep, **kw), 70 + size)
    n = max(token_marks) + size + 8
    g = torch.Generator().manual_seed(71 + size)
    t = torch.randint(0, 62, (n,), generator=g).tolist()
    for m in token_marks:
        t[m] = 63
    rows = []
    for m in token_marks:
        for p in (m + size - 1, m + size):
            if p < n and t[p] != 63:
                t[p] = 62
                rows.append(p)
    return cfg, w, t, sorted(set(rows))


@pytest.mark.parametrize("kind,kw", [("latent", {}), ("differential", {}), ("differential", WIDE)])
@pytest.mark.parametrize("size", [24, 64, 65, 40, 129])
def test_keys_just_inside_and_just_outside_the_window(size, kind, kw, monkeypatch):
    """marks at the sequence's start, in the middle of pages and where an edge falls on a page border; a window that is one token off in
    either direction changes the marked rows by far more than the tolerance.  In prompts (cut at, before and after the edges) and
    decoded one by one, fp32 and bf16."""
    cfg, w, t, rows = edge_setup(kind, size, **kw)
    ref = to.forward(cfg, w, t)
    real = to.visible
    for d in (-1, 1):
        monkeypatch.setattr(to, "visible", lambda i, m, d=d: real(i, {**m, "size": m["size"] + d}))
        assert err(to.forward(cfg, w, t)[rows], ref[rows]) > 100 * TOL["float32"], d
        monkeypatch.undo()
    first = rows[0]
    for dtype in ("float32", "bfloat16"):
        e = off(dtype)
        with Rig(cfg, dtype, weights=w, max_tokens=1024, max_batch_tokens=1024) as rig:
            got = run_schedule(rig, t, [len(t)])
            assert e(got, ref) < TOL[dtype] and e(got[rows], ref[rows]) < TOL[dtype]
            got = run_schedule(rig, t, [first, 2, size - 1, 2, size, 17, 2, 64, 2, 100, 3, len(t)])      # portions that start and end at the edges
            assert e(got, ref) < TOL[dtype] and e(got[rows], ref[rows]) < TOL[dtype]
            got = run_schedule(rig, t, [max(1, first - 3)])                               # every edge row decoded alone
            assert e(got, ref) < TOL[dtype] and e(got[rows], ref[rows]) < TOL[dtype]


@pytest.mark.parametrize("kw", [{}, WIDE])
@pytest.mark.parametrize("size,keep", [(20, 1), (20, 4), (70, 4), (64, 64), (30, 65), (100, 63), (10, 128), (40, 130)])
def test_first_tokens_that_the_window_keeps(size, keep, kw, monkeypatch):
    """the marked token at the last kept place is seen from any distance, at the next place only inside the window"""
    for at in (keep - 1, keep):
        cfg, w = opposite_setup(edge_layer("differential", size, keep, **kw), 200 + keep)
        n = keep + size + 90
        g = torch.Generator().manual_seed(201 + size + at)
        t = torch.randint(0, 62, (n,), generator=g).tolist()
        t[at] = 63
        rows = [p for p in (at + 1, at + size - 1, at + size, at + size + 1, at + size + 40, n - 3, n - 1) if at < p]
        for p in rows:
            t[p] = 62
        ref = to.forward(cfg, w, t)
        real = to.visible
        d = -1 if at == keep - 1 else 1
        monkeypatch.setattr(to, "visible", lambda i, m: real(i, {**m, "keep_first": m["keep_first"] + d}))
        far = [p for p in rows if p >= at + size]
        assert err(to.forward(cfg, w, t)[far], ref[far]) > 100 * TOL["float32"]
        monkeypatch.undo()
        for dtype in ("float32", "bfloat16"):
            e = off(dtype)
            with Rig(cfg, dtype, weights=w) as rig:
                for cuts in ([n], [max(1, keep), 2, size, 2, 33, 17, n], [max(1, n - 45)]):
                    got = run_schedule(rig, t, cuts)
                    assert e(got, ref) < TOL[dtype] and e(got[rows], ref[rows]) < TOL[dtype]


@pytest.mark.parametrize("kind,kw", [("latent", {}), ("differential", {}), ("differential", WIDE)])
@pytest.mark.parametrize("size", [None, 704])
def test_far_key_among_hundreds(size, kind, kw):
    """the marked token at position 3 is seen from 700 positions on, through the prompt kernels and through decode rows split
    over several blocks"""
    n = 706
    cfg, w = opposite_setup(edge_layer(kind, size, **kw), 170)
    g = torch.Generator().manual_seed(171)
    t = torch.randint(0, 62, (n,), generator=g).tolist()
    t[3] = 63
    for p in range(n - 6, n):
        t[p] = 62
    ref = to.forward(cfg, w, t)
    t_without = list(t)
    t_without[3] = 5
    assert err(to.forward(cfg, w, t_without)[-6:], ref[-6:]) > 100 * TOL["float32"]       # the far key matters
    for dtype in ("float32", "bfloat16"):
        with Rig(cfg, dtype, weights=w, max_batch_tokens=1024) as rig:
            for cuts in ([n], [300, 2, 250, 148]):                                        # the last six decoded one by one
                got = run_schedule(rig, t, cuts)
                assert off(dtype)(got, ref) < TOL[dtype] and off(dtype)(got[-6:], ref[-6:]) < TOL[dtype]


@pytest.mark.parametrize("level", [-30.0, 0.0, 3.0, 12.0])
def test_sink_counts_once_and_unscaled(level):
    """sinks far below, about and far above the scores; left out, counted twice or scaled they change every row"""
    cfg = config([lat(mask={"size": 90}, scale=0.5)], side=None)
    w = to.random_weights(cfg, 61)
    w["l0.mix.sink"] = torch.tensor([level, level + 0.5, level - 0.25])
    t = toks(170, seed=62)
    ref = to.forward(cfg, w, t)
    if level >= 0:
        for f in (lambda s: s - 100, lambda s: s + 0.6931, lambda s: s * 0.5 - 0.3):
            assert err(to.forward(cfg, {**w, "l0.mix.sink": f(w["l0.mix.sink"])}, t)[:40], ref[:40]) > 20 * TOL["float32"]
    for dtype in ("float32", "bfloat16"):
        with Rig(cfg, dtype, weights=w) as rig:
            for cuts in ([170], [60, 2, 50, 33]):
                assert off(dtype)(run_schedule(rig, t, cuts), ref) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_lambda_far_from_its_constant(dtype):
    """lambda of about -3 and +4: its vectors matter, also when they are bound again"""
    cfg = config([dif(DENSE), dif(heads=2, kv_heads=2)], side=None)
    t = toks(90, seed=64)
    for k, (a, b) in enumerate(((0.1, 1.2), (1.5, 0.2))):
        w = to.random_weights(cfg, 63 + k)
        for l in range(2):
            for n, v in (("lq1", a), ("lk1", 1.0), ("lq2", b), ("lk2", 1.0)):
                w[f"l{l}.mix.{n}"] = torch.full((16,), v / 16 if n[1] == "q" else v).to(torch.bfloat16).float()
        lam = float(to.diff_lambda({n: v.double() for n, v in w.items()}, "l0.", 0.35))
        assert (lam < -1.5) if k == 0 else (lam > 3)
        with Rig(cfg, dtype, weights=w) as rig:
            ref = rig.oracle(t)
            for cuts in ([90], [40, 2, 20]):
                assert off(dtype)(run_schedule(rig, t, cuts), ref) < TOL[dtype]
            if dtype == "float32":
                q = rig.model._bound["l0.mix.lq1"]
                new = (w["l0.mix.lq1"] + 0.0625).to(torch.bfloat16).float()
                w2 = {**w, "l0.mix.lq1": new}
                rig.model.load_weights({"l0.mix.lq1": new.to(q.device, q.dtype)})
                assert err(run_schedule(rig, t, [40]), to.forward(cfg, w2, t)) < TOL[dtype]


def test_rotation_follows_the_true_position():
    """far into a sequence, with slow and fast pairs: scaled frequencies, the multiplier of the rotated part and positions that continue
    over portions (sharp scores)"""
    cfg = config([lat(rot_dim=16, rot=rot(1000.0, 16, {"factor": 6.0, "original": 100, "fast": 10.0, "slow": 1.0}), mask={"size": 300}, scale=0.5),
                  dif(size=50, keep=4, rot=rot(2000.0, 16, {"factor": 7.0, "low": 1.0, "high": 5.0, "original": 120}), scale=0.6)], side=None)
    t = toks(420, seed=68)
    w = to.random_weights(cfg, 69)
    ref = to.forward(cfg, w, t)
    for i, sc in enumerate(({"factor": 6.5}, {"original": 60})):       # the scaling shows
        c2 = copy.deepcopy(cfg)
        c2["layers"][i]["mixer"]["rot"]["scaling"].update(sc)
        assert err(to.forward(c2, w, t), ref) > 50 * TOL["float32"]
    with Rig(cfg, "float32", weights=w) as rig:
        assert err(run_schedule(rig, t, [420]), ref) < TOL["float32"]
        assert err(run_schedule(rig, t, [333, 2, 60]), ref) < TOL["float32"]


def test_long_rows_split_over_blocks_in_decoding():
    """decoding past 512 and 1024 visible keys, under windows that need one, two and three blocks a row and without one, with head sizes
    for either decode kernel"""
    cfg = config([dif(size=None, heads=2, kv_heads=1, dim=16, vdim=16, scale=0.4), dif(size=600, keep=70, heads=2, kv_heads=2, dim=16, vdim=40, scale=0.4),
                  lat(mask={"size": 1100}, heads=2), dif(size=512, keep=1, heads=4, kv_heads=1, dim=9, vdim=7, rot=rot(50.0, 8, BANDS))], side=None)
    t = toks(1300, seed=165)
    with Rig(cfg, "float32", max_tokens=1344, max_batch_tokens=1344) as rig:
        ref = rig.oracle(t)
        for first, n in ((508, 8), (1020, 8), (596, 8), (1290, 8)):
            lg = run_schedule(rig, t[:first + n], [first])
            assert err(lg[first:], ref[first:first + n]) < TOL["float32"]


def test_first_tokens_of_a_sequence():
    """the first token sees itself alone; so does the first token of the next user of its slot"""
    for dtype in ("float32", "bfloat16"):
        with Rig(FULL, dtype) as rig:
            for n in (1, 2, 3, 4, 6, 17):
                t = toks(n, seed=80 + n)
                tol = TOL[dtype] * (2 if dtype == "bfloat16" else 1)
                assert off(dtype)(run_schedule(rig, t, [n]), rig.oracle(t)) < tol
                assert off(dtype)(run_schedule(rig, t, []), rig.oracle(t)) < tol


def test_token_rows_belong_to_the_layer():
    """the token table's columns of another layer, or another token's row, are far off"""
    cfg = config([dif(DENSE), lat(DENSE), dif(None)], side=12)
    w = to.random_weights(cfg, 91)
    for i in range(3):
        w[f"l{i}.side.norm"] = w[f"l{i}.side.norm"] * 4
    t = toks(80, seed=92)
    ref = to.forward(cfg, w, t)
    assert err(to.forward(cfg, {**w, "side.embed": w["side.embed"].roll(12, 1)}, t), ref) > 100 * TOL["float32"]
    assert err(to.forward(cfg, {**w, "side.embed": w["side.embed"].roll(1, 0)}, t), ref) > 100 * TOL["float32"]
    with Rig(cfg, "float32", weights=w) as rig:
        rig.eng.step([("x", toks(17, seed=93), [])])
        assert err(run_schedule(rig, t, [20, 2, 33]), ref) < TOL["float32"]


def test_long_decoding():
    t = toks(300, seed=90)
    with Rig(FULL, "float32") as rig:
        assert err(run_schedule(rig, t, [20]), rig.oracle(t)) < TOL["float32"]


def test_a_step_larger_than_the_batch_buffer_is_cut_inside():
    t = toks(300, seed=95)
    with Rig(FULL, "float32", max_batch_tokens=64) as rig:
        got = rig.eng.step([("a", t[:290], [0, 63, 64, 289]), ("b", t[:70], [69])])
        ref = rig.oracle(t)
        assert err(got[:4], ref[[0, 63, 64, 289]]) < TOL["float32"]
        assert err(got[4:], ref[[69]]) < TOL["float32"]


def test_graph_replay_equals_launch_by_launch_decoding():
    t = toks(60, seed=97)
    with Rig(FULL, "bfloat16") as rig:
        a = run_schedule(rig, t, [20])
        rig.model.set_graphs(False)
        b = run_schedule(rig, t, [20])
        assert torch.equal(a, b)


# -- the mechanisms in other company ---------------------------------------------------------------------------------------------
def made_up(name, family):
    """a family of this test: registered under `name` like any other"""
    from dnet_b200.core.models.seqmix import SeqMixRingModel

    return type(name, (SeqMixRingModel,), {"model_type": name.lower(), "family": family})


def random_for(cls, cfg, seed):
    """random weights for what the class expects of the config (fp32 holding bf16 values)"""
    from dnet_b200.core.models.seqmix import parse_layer_list

    m = cls.__new__(cls)
    sc, layers = parse_layer_list(cfg, cls.family)
    m.config, m._cfg_struct, m._layer_structs, m.hidden_size, m.vocab_size = cfg, sc, layers, sc.width, sc.vocab
    g = torch.Generator().manual_seed(seed)
    out = {}
    for k, s in m.expected_tensors().items():
        t = torch.randn(s, generator=g)
        if "norm" in k:
            t = 0.2 * t
        elif "ls" in k:
            t = 0.7 + 0.3 * t
        elif len(s) == 2 and k not in ("embed", "side.embed"):
            t = t * s[-1] ** -0.5
        out[k] = t.to(torch.bfloat16).float()
    return out


def test_kept_tokens_under_sigmoid_weights_and_scaled_outputs_behind_rms_norms():
    """a window that keeps the first tokens with sigmoid weights, a distance bias and gated heads; channel scales, a residual factor and the
    token input behind one-plus RMS norms, whose next norm is a launch of its own; relu-squared feed-forward with biases, capped logits"""
    cls = made_up("TestKeptSigmoid", {"norm": "rms", "layer_scale": True, "qk_norm": "head", "mask": "window", "attn_weight": "sigmoid", "dist_bias": True, "head_gate": True,
                                      "ff_act": "relu2"})
    H, G, size, keep, side = 4, 2, 20, 5, 12
    for d in (16, 64):
        mx = {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": 0.2, "mask": {"size": size, "keep_first": keep}}
        cfg = {"architecture": "TestKeptSigmoid", "vocab": 64, "width": 48, "norm": {"eps": 1e-5}, "residual_mult": 0.6, "logit_softcap": 5.0, "token_side": {"dim": side},
               "layers": [{"type": "attention", "mixer": mx, "mlp": {"kind": "dense", "ff": 40}}, {"type": "attention", "mixer": mx, "mlp": None}]}
        w = random_for(cls, cfg, 501)
        for i in range(2):
            for r in ("mix.r1", "mix.r2"):
                w[f"l{i}.{r}"] = w[f"l{i}.{r}"].abs()
        t = toks(130, vocab=64, seed=502)
        D = {k: v.double() for k, v in w.items()}
        x = D["embed"][t]

        def rms1p(x, w):
            return to.unit_rms(x, 1e-5) * (1 + w)

        for i, L in enumerate(cfg["layers"]):
            p = f"l{i}."
            h = rms1p(x, D[p + "norm1"])
            q, k, v = (h @ D[p + "mix." + c].T for c in "qkv")
            q, k, v = q.view(-1, H, d), k.view(-1, G, d), v.view(-1, G, d)
            q, k = to.unit_rms(q, 1e-5) * D[p + "mix.q.norm"], to.unit_rms(k, 1e-5) * D[p + "mix.k.norm"]
            gate = torch.sigmoid(h @ D[p + "head_gate"].T)
            rows = []
            for j in range(len(t)):
                js = to.visible(j, mx["mask"])
                of = [a // (H // G) for a in range(H)]
                s = torch.einsum("hd,nhd->hn", q[j], k[js][:, of]) * 0.2
                dist = torch.tensor([float(j - a) for a in js], dtype=torch.float64)
                s = s - D[p + "mix.r1"][:, None] * torch.log1p(D[p + "mix.r2"][:, None] * dist[None])
                a = torch.sigmoid(s + D[p + "mix.pb"][:, None]) * gate[j][:, None]
                rows.append(torch.einsum("hn,nhd->hd", a, v[js][:, of]).reshape(-1))
            x = x + 0.6 * D[p + "ls1"] * (torch.stack(rows) @ D[p + "mix.o"].T)
            if L["mlp"]:
                h = rms1p(x, D[p + "norm2"])
                f = torch.relu(h @ D[p + "mlp.up"].T + D[p + "mlp.up.b"]) ** 2 @ D[p + "mlp.down"].T + D[p + "mlp.down.b"]
                x = x + 0.6 * D[p + "ls2"] * f
            x = x + to.token_input({**D}, p, i, side, torch.tensor(t), x, 1e-5)
        z = rms1p(x, D["final.norm"]) @ D["head"].T
        ref = 5.0 * torch.tanh(z / 5.0)
        for dtype in ("float32", "bfloat16"):
            with Rig(cfg, dtype, weights=w) as rig:
                assert off(dtype)(run_schedule(rig, t, [130]), ref) < TOL[dtype]
                assert off(dtype)(run_schedule(rig, t, [50, 2, 40]), ref) < TOL[dtype]


# -- the token loop, the command lines, the runtime ----------------------------------------------------------------------------
def greedy_agrees(cfg, w, prompt, got, margin=1e-3):
    seq = list(prompt)
    for tok in got:
        lg = to.forward(cfg, w, seq)[-1]
        top2 = torch.topk(lg, 2).values
        if float(top2[0] - top2[1]) > margin:           # a near tie may fall either way
            assert tok == int(lg.argmax()), f"at length {len(seq)}"
        seq.append(tok)


def test_greedy_generation_through_the_batcher():
    from dnet_b200.shard.batching import GenRequest

    with Rig(FULL, "float32", max_tokens=320, max_seqs=2) as rig:
        rig.eng.step_tokens = 48
        reqs = [GenRequest(f"g{i}", toks(n, seed=100 + i), max_new_tokens=m) for i, (n, m) in enumerate([(30, 6), (100, 4), (3, 9), (65, 5)])]
        out = rig.eng.generate(reqs)
        assert rig.model.free_slots == 2 and rig.model.free_pages == 5
        for r in reqs:
            greedy_agrees(FULL, rig.w, r.prompt, out[r.id])


def test_command_lines_on_a_checkpoint_folder(tmp_path):
    """bin/trace_run and bin/generate on a folder with config.json and model.safetensors: the class is picked by the
    config's architecture; alphas are scalars in the file"""
    import json
    import os
    import struct
    import subprocess
    import sys

    import numpy as np

    cfg = config([dif(DENSE), lat(DENSE), lat(None, kv_from=1)])
    w = to.random_weights(cfg, 110)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    header, blobs, at = {}, [], 0
    for k, v in w.items():
        raw = v.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        header[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    t = toks(70, seed=111)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:50], "want": [49]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": t[50:52], "want": [0, 1]}, {"id": "b", "tokens": t[:9], "want": [8]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": t[52:], "want": [17]}], "end": ["a"]}]
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    ref = to.forward(cfg, w, t)
    got = [torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"]) for i in range(3)]
    assert err(got[0], ref[[49]]) < TOL["float32"]
    assert err(got[1], torch.cat([ref[[50, 51]], to.forward(cfg, w, t[:9])[[8]]])) < TOL["float32"]
    assert err(got[2], ref[[69]]) < TOL["float32"]
    reqs = [{"id": "x", "prompt": t[:40], "max_new_tokens": 5}, {"id": "y", "prompt": t[:7], "max_new_tokens": 3}]
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "generate"), "--model", str(folder), "--dtype", "float32", "--max-tokens", "192",
                        "--step-tokens", "16"], input="\n".join(json.dumps(r) for r in reqs) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    outs = {o["id"]: o["tokens"] for o in map(json.loads, p.stdout.strip().splitlines())}
    for r in reqs:
        assert len(outs[r["id"]]) == r["max_new_tokens"]
        greedy_agrees(cfg, w, r["prompt"], outs[r["id"]])


def test_served_by_the_shard_runtime():
    """load_model_core finds the class by the config's architecture and serves it with the batched policy: frames of
    tokens in, sampled tokens out, chunked prompts, slots and pages returned at release"""
    import queue

    from dnet_b200.shard.models import ShardLoadModelRequest
    from dnet_b200.shard.policies.batched import BatchedStepPolicy
    from dnet_b200.shard.runtime import ShardRuntime
    from dnet_b200.utils.model import HostDictSource
    from tests.helpers import ring_generate, token_message

    w = to.random_weights(FULL, 21)
    n = len(FULL["layers"])
    rt = ShardRuntime(shard_id="s0", queue_size=64)
    rt.kv_cache_config.max_tokens = 256
    src = HostDictSource({k: v.to(torch.bfloat16) for k, v in w.items()}, FULL)
    rt.load_model_core(ShardLoadModelRequest(model_path=src, total_layers=n, layers=list(range(n)), window_size=n, residency_size=n, kv_bits="fp16"))
    try:
        assert isinstance(rt.policy, BatchedStepPolicy)
        a, b = toks(45, seed=180), toks(70, seed=181)
        out_a = [t for t, _, _ in ring_generate([rt], "na", a, 5)]
        greedy_agrees(FULL, w, a, out_a, margin=0.1 * float(to.forward(FULL, w, a)[-1].std()))
        for part in (b[:30], b[30:64]):
            rt.policy.process(token_message(rt, "nb", part, more=True))
            with pytest.raises(queue.Empty):
                rt.activation_send_queue.get_nowait()
        out_b = [t for t, _, _ in ring_generate([rt], "nb", b[64:], 4)]
        greedy_agrees(FULL, w, b, out_b, margin=0.1 * float(to.forward(FULL, w, b)[-1].std()))
        rt.release_nonce("na")
        rt.release_nonce_deferred("nb")
        assert rt.model.free_pages == rt.model.pool_pages
    finally:
        assert rt.unload_model_core().success
