"""The Bokenex family (core/models/seqmix.py BokenexRingModel, shard/batching.py, libdnet_b200_seq) against the float64
oracle (oracle/bokenex_oracle.py): every mechanism alone with the residual after each layer, then portions, batches,
page and slot reuse, keys at the edges of the sliding window and far away with scores made to stand out, carried
convolution inputs that must not survive a slot, the position table's end, long decoding and greedy generation through
the batcher's token loop.  fp32 runs are held to 2e-4 of the logits' spread row by row; bf16 runs to 4e-2 of the spread
over all rows together.  The family's mechanisms are also run in other company (families made up here)."""
from __future__ import annotations

import math

import pytest
import torch

from oracle import bokenex_oracle as bo

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-4, "bfloat16": 4e-2}

DENSE = {"kind": "dense", "ff": 72}


def moe(experts=5, top=2, scale=1.6, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}}


def att(mlp=None, size=21, **kw):
    mx = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "conv": 3, "scale": 0.3}
    if size is not None:
        mx["mask"] = {"size": size}
    mx.update(kw)
    return {"type": "attention", "mixer": {k: v for k, v in mx.items() if v is not None}, "mlp": mlp}


def config(layers, width=48, vocab=96, eps=1e-5, mult=0.4, positions=1400):
    return {"architecture": "Bokenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "max_positions": positions,
            "layers": layers}


FULL = config([att(DENSE), att(moe()), att(None, heads=2, kv_heads=1, dim=8, conv=2), att(moe(3, 3, 0.7, 40), size=70, heads=6, kv_heads=3, vdim=8),
               att(DENSE, size=None, heads=3, kv_heads=3, dim=24, vdim=24, conv=5)])


class Rig:
    """a model + batcher on the GPU and the oracle's view of the same weights"""

    def __init__(self, cfg, dtype="float32", seed=1, max_tokens=1024, max_seqs=4, max_batch_tokens=512, weights=None):
        from dnet_b200.shard.batching import SequenceBatcher, load_model
        from dnet_b200.utils.model import HostDictSource

        self.cfg, self.dtype = cfg, dtype
        self.w = weights if weights is not None else bo.random_weights(cfg, seed)
        self.model = load_model(HostDictSource({k: v.to(torch.bfloat16) for k, v in self.w.items()}, cfg), dtype, max_tokens=max_tokens,
                                max_seqs=max_seqs, max_batch_tokens=max_batch_tokens)
        self.eng = SequenceBatcher(self.model)

    def oracle(self, tokens, layers_out=None):
        return bo.forward(self.cfg, self.w, tokens, layers_out)

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
    g = torch.Generator().manual_seed(9000 + seed)
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
    "attention": config([att()]),
    "no_convolution": config([att(conv=None)]),
    "convolution_of_one_tap": config([att(conv=1), att(DENSE, conv=1)]),
    "convolution_of_two_taps": config([att(conv=2)]),
    "convolution_of_nine_taps": config([att(conv=9), att(conv=9)]),
    "one_head": config([att(heads=1, kv_heads=1, dim=32, vdim=40)]),
    "as_many_key_heads": config([att(heads=3, kv_heads=3, dim=8, vdim=8)]),
    "one_key_head": config([att(heads=6, kv_heads=1, dim=24, vdim=16)]),
    "values_narrower_than_keys": config([att(dim=40, vdim=8)]),
    "odd_sizes": config([att(heads=3, kv_heads=1, dim=7, vdim=5), att(heads=2, kv_heads=2, dim=10, vdim=11)]),
    "large_heads": config([att(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.1), att(heads=1, kv_heads=1, dim=200, vdim=160, scale=0.1)], width=64),
    "window_of_one": config([att(size=1), att(size=2)]),
    "window_of_a_page": config([att(size=64), att(size=65), att(size=63)]),
    "window_of_two_pages": config([att(size=128), att(size=127)]),
    "window_wider_than_the_prompt": config([att(size=4000)]),
    "no_window": config([att(size=None)]),
    "scale_of_one": config([att(scale=1.0)]),
    "factor_of_one": config([att(DENSE), att(moe())], mult=1.0),
    "factor_above_one": config([att(DENSE)], mult=1.7),
    "large_eps": config([att(DENSE), att(None)], eps=0.3),
    "dense": config([att(DENSE)]),
    "dense_wide": config([att({"kind": "dense", "ff": 200})]),
    "experts": config([att(moe())]),
    "experts_top_one": config([att(moe(7, 1, 2.5))]),
    "experts_all_chosen": config([att(moe(4, 4, 1.0))]),
    "one_expert": config([att(moe(1, 1, 0.5))]),
    "experts_many": config([att(moe(70, 9, 3.0, 8))]),
    "experts_of_odd_width": config([att(moe(5, 3, 1.25, 13))], width=50),
    "no_feed_forward_between": config([att(DENSE), att(None), att(moe()), att(None)]),
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_full_model_whole_prompt(dtype):
    t = toks(200, seed=5)
    with Rig(FULL, dtype) as rig:
        assert off(dtype)(rig.eng.step([("a", t, list(range(len(t))))]), rig.oracle(t)) < TOL[dtype]


def test_positions_matter_and_come_from_the_sequence():
    """the position row is the sequence's, not the step's: with position rows ten times the embeddings a token fed at a wrong
    position is far off"""
    cfg = config([att(DENSE)])
    w = bo.random_weights(cfg, 8)
    w["pos"] = (w["pos"] * 30).to(torch.bfloat16).float()
    t = toks(80, seed=9)
    with Rig(cfg, "float32", weights=w) as rig:
        ref = rig.oracle(t)
        assert err(rig.oracle(t[1:]), ref[1:]) > 100 * TOL["float32"]
        rig.eng.step([("x", toks(17, seed=10), [])])
        assert err(run_schedule(rig, t, [20, 2, 33]), ref) < TOL["float32"]


def test_the_position_table_ends_a_sequence():
    """a sequence may fill the table to its last row; a token beyond is refused and changes nothing"""
    from dnet_b200._cabi import DnError

    cfg = config([att(DENSE), att(moe())], positions=90)
    t = toks(91, seed=12)
    with Rig(cfg, "float32") as rig:
        ref = rig.oracle(t[:90])
        assert err(rig.eng.step([("a", t[:88], list(range(88)))]), ref[:88]) < TOL["float32"]
        with pytest.raises(DnError, match="90 positions"):
            rig.eng.step([("a", t[88:91], [0])])
        assert err(rig.eng.step([("a", t[88:90], [0, 1])]), ref[88:]) < TOL["float32"]
        with pytest.raises(DnError, match="90 positions"):
            rig.eng.step([("a", t[90:], [0])])
        rig.eng.finish("a")
        assert err(run_schedule(rig, t[:90], [50, 35]), ref) < TOL["float32"]      # and the last rows by decoding


# -- sizes --------------------------------------------------------------------------------------------------------------
def test_sizes_on_the_tensor_core_products():
    """width and projection sizes in multiples of 64: bf16 prompt portions take the tcgen05 products (grouped ones for the
    experts, in tiles of 64 rows) and the MMA attention tiles"""
    cfg = config([att({"kind": "dense", "ff": 256}, size=33, heads=4, kv_heads=2, dim=64, vdim=32, scale=0.1, conv=4),
                  att(moe(4, 2, 1.5, 64), size=90, heads=8, kv_heads=2, dim=32, vdim=64)], width=128, vocab=192)
    t = toks(300, vocab=192, seed=6)
    with Rig(cfg, "bfloat16") as rig:
        ref = rig.oracle(t)
        assert err16(rig.eng.step([("a", t, list(range(len(t))))]), ref) < TOL["bfloat16"]
        rig.eng.finish("a")
        assert err16(run_schedule(rig, t, [130, 17, 64, 2, 70]), ref) < TOL["bfloat16"]


def test_experts_in_tiles_of_128_rows():
    """two experts, both chosen by every token: 300 rows each take the wide token tiles of the grouped products"""
    cfg = config([att(moe(2, 2, 1.0, 192), heads=2, kv_heads=1, dim=64, vdim=64, scale=0.1)], width=128, vocab=64)
    t = toks(300, vocab=64, seed=16)
    with Rig(cfg, "bfloat16") as rig:
        assert err16(rig.eng.step([("a", t, list(range(len(t))))]), rig.oracle(t)) < TOL["bfloat16"]


@pytest.mark.parametrize("dk,dv", [(16, 16), (32, 48), (24, 128), (56, 24), (64, 64), (48, 96), (96, 32), (128, 64), (112, 120)])
def test_every_pair_of_head_sizes_of_the_tiles(dk, dv):
    cfg = config([att(size=75, heads=4, kv_heads=2, dim=dk, vdim=dv, scale=dk ** -0.5, conv=2)], width=64)
    t = toks(180, seed=17)
    with Rig(cfg, "bfloat16") as rig:
        ref = rig.oracle(t)
        assert err16(run_schedule(rig, t, [180]), ref) < TOL["bfloat16"]
        assert err16(run_schedule(rig, t, [100, 2, 70]), ref) < TOL["bfloat16"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_allow_no_wide_loads(dtype):
    """width, head, feed-forward and vocabulary sizes that are multiples of neither 4 nor 8: the scalar forms of every kernel"""
    cfg = config([att({"kind": "dense", "ff": 35}, size=19, heads=3, kv_heads=1, dim=7, vdim=5), att(moe(3, 2, 1.3, 9), heads=2, kv_heads=2, dim=9, vdim=13)],
                 width=50, vocab=77)
    t = toks(120, vocab=77, seed=160)
    with Rig(cfg, dtype) as rig:
        ref = rig.oracle(t)
        assert off(dtype)(run_schedule(rig, t, [120]), ref) < TOL[dtype]
        assert off(dtype)(run_schedule(rig, t, [70, 2, 20]), ref) < TOL[dtype]


@pytest.mark.parametrize("H,G,dk,dv,size", [(1, 1, 64, 64, 50), (4, 2, 128, 64, 200), (6, 2, 64, 128, 64), (6, 1, 128, 128, 65), (16, 1, 64, 64, 33),
                                            (20, 1, 64, 64, 300), (8, 8, 64, 64, None), (34, 2, 64, 128, 130), (4, 1, 128, 128, 1)])
def test_prompt_attention_on_tcgen05(H, G, dk, dv, size):
    """heads of 64 / 128: one, some and more than 16 query heads a key head (token blocks of 128 down to 8), windows of one token, about
    a page, several tiles and none; whole, in portions that start inside pages and tiles, and unequal entries side by side"""
    cfg = config([att(size=size, heads=H, kv_heads=G, dim=dk, vdim=dv, scale=1.5 * dk ** -0.5, conv=2)], width=64)
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
    cfg = config([att(DENSE, size=200, heads=4, kv_heads=2, dim=64, vdim=64, scale=0.15)], width=64)
    w = bo.random_weights(cfg, 520)
    w["l0.mix.v"] = w["l0.mix.v"] * 4
    with Rig(cfg, "bfloat16", weights=w, max_tokens=256, max_seqs=2) as rig:
        for n, k in ((250, 0), (17, 1), (70, 2), (129, 3), (190, 4)):
            t = toks(n, seed=521 + k)
            assert err16(run_schedule(rig, t, [n]), rig.oracle(t)) < TOL["bfloat16"]


LAYER_SIZED = {
    "w384": config([att({"kind": "dense", "ff": 640}, size=90, heads=6, kv_heads=2, dim=64, vdim=48, scale=0.11, conv=4),
                    att(moe(6, 2, 2.0, 128), size=40, heads=12, kv_heads=4, dim=32, vdim=32, conv=4),
                    att(None, size=64, heads=4, kv_heads=1, dim=96, vdim=64, scale=0.1, conv=4)], width=384, vocab=640, mult=0.35),
    "w512": config([att({"kind": "dense", "ff": 1024}, size=150, heads=4, kv_heads=1, dim=128, vdim=128, scale=0.09),
                    att(moe(10, 4, 1.8, 192), size=33, heads=8, kv_heads=1, dim=128, vdim=64, scale=0.08, conv=2),
                    att({"kind": "dense", "ff": 768}, size=None, heads=16, kv_heads=4, dim=32, vdim=32, scale=0.17)], width=512, vocab=1000),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(LAYER_SIZED))
def test_layer_sized_models(name, dtype):
    cfg = LAYER_SIZED[name]
    V = cfg["vocab"]
    t = toks(210, vocab=V, seed=300)
    w = bo.random_weights(cfg, 301)
    with Rig(cfg, dtype, weights=w) as rig:
        ref = bo.forward(cfg, w, t)
        e = off(dtype)
        whole = run_schedule(rig, t, [len(t)])
        assert e(whole, ref) < TOL[dtype]
        cut = run_schedule(rig, t, [100, 2, 64, 17, 5])
        assert e(cut, ref) < TOL[dtype]
        rig.eng.step([("a", t[:100], [])])
        rig.eng.step([("b", t[:37], [])])
        lg = rig.eng.step([("a", t[100:130], list(range(30))), ("b", t[37:38], [0])])      # a portion beside a decoded token
        assert e(lg[:30], ref[100:130]) < TOL[dtype] and e(lg[30:], ref[37:38]) < 2 * TOL[dtype]
        if dtype == "bfloat16":       # and the schedules agree with each other better than with the oracle
            assert err16(cut, whole.cpu()) < 0.75 * TOL[dtype] and err16(lg[:30], whole[100:130].cpu()) < 0.75 * TOL[dtype]


# -- schedules ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_against_token_by_token(dtype):
    t = toks(90, seed=7)
    with Rig(FULL, dtype) as rig:
        ref = rig.oracle(t)
        assert off(dtype)(run_schedule(rig, t, []), ref) < TOL[dtype]              # every token alone, from the first
        assert off(dtype)(run_schedule(rig, t, [50]), ref) < TOL[dtype]            # a prompt, then decoding


@pytest.mark.parametrize("cuts", [[2, 2, 2, 3, 5, 64, 1, 2, 40], [39, 2, 41, 2, 63, 1, 64], [128, 2], [1, 1, 1, 2, 200], [20, 1, 21, 22, 2, 19]])
def test_portions_of_any_size(cuts):
    t = toks(230, seed=11)
    with Rig(FULL, "float32") as rig:
        assert err(run_schedule(rig, t, cuts), rig.oracle(t)) < TOL["float32"]


def test_results_do_not_depend_on_the_cut_beyond_rounding():
    t = toks(130, seed=13)
    with Rig(FULL, "bfloat16") as rig:
        a = run_schedule(rig, t, [130])
        b = run_schedule(rig, t, [3, 61, 2, 30])
        assert err16(b, a.cpu()) < 2e-2


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
    """steps of 1 .. 20 single tokens: the few-row products, the tiles, and the convolutions carried inside the prep kernel"""
    seqs = [toks(20 + 5 * i, seed=400 + i) for i in range(n)]
    with Rig(FULL, dtype, max_tokens=64 * 3 * n, max_seqs=n) as rig:
        refs = torch.stack([rig.oracle(s)[-3:] for s in seqs])
        rig.eng.step([(f"s{i}", s[:-3], []) for i, s in enumerate(seqs[:n // 2 + 1])])
        for i, s in enumerate(seqs):
            if i > n // 2:
                rig.eng.step([(f"s{i}", s[:-3], [])])
        got = torch.stack([rig.eng.step([(f"s{i}", [s[k]], [0]) for i, s in enumerate(seqs)]) for k in (-3, -2, -1)], dim=1)
        assert off(dtype)(got.flatten(0, 1), refs.flatten(0, 1)) < TOL[dtype]


def test_pages_and_slots_are_reused():
    """a pool of 4 pages and 2 slots serves 6 requests two at a time; a request that does not fit is refused without
    disturbing the live ones; a page's old rows and a slot's old convolution inputs never show in its next user"""
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


# -- keys at the window's edges and far away, with scores made to stand out ------------------------------------------------------
def opposite_setup(layer, seed, vocab=64):
    """One layer in which a query finds the token whose input points the other way: the first head's keys are minus its
    queries (k projection = minus q projection), q / k norm weights are one, position rows are zero, so a token scores about
    -dim scale against itself and +dim scale against a token with the opposite embedding (token 63 is minus token 62).  With an
    offset of minus half of that only such a key gets a weight near one; everything else weighs next to nothing."""
    dk, scale = layer["mixer"]["dim"], layer["mixer"]["scale"]
    cfg = config([layer], vocab=vocab)
    w = bo.random_weights(cfg, seed)
    e = w["embed"].clone()
    e[63] = -e[62]
    w["embed"] = e
    w["pos"] = torch.zeros_like(w["pos"])
    G = layer["mixer"]["kv_heads"]
    w["l0.mix.k"][:dk] = -w["l0.mix.q"][:dk]
    w["l0.mix.q.norm"] = torch.ones(dk)
    w["l0.mix.k.norm"] = torch.ones(dk)
    H = layer["mixer"]["heads"]
    w["l0.mix.pb"] = torch.full((H,), -0.5 * dk * scale)
    w["l0.mix.r1"] = torch.full((H,), 0.25)
    for c in "qkv":      # a convolution that passes the token's own input
        if layer["mixer"].get("conv"):
            cw = torch.zeros_like(w[f"l0.mix.{c}.conv"])
            cw[:, -1] = 1.0
            w[f"l0.mix.{c}.conv"] = cw
    assert G >= 1
    return cfg, w


def edge_setup(size, token_marks=(0, 40, 64, 104, 127, 170), dk=32, dv=16):
    """token 63 stands at every position of `token_marks`, token 62 at mark + size - 1 (it just sees the 63) and at mark + size
    (it just does not); all other tokens are below 62"""
    cfg, w = opposite_setup(att(size=size, heads=2, kv_heads=1, dim=dk, vdim=dv, scale=16.0 / dk), 70 + size)
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


@pytest.mark.parametrize("dk,dv", [(32, 16), (64, 64)])      # the warp-level tiles, the tcgen05 kernel
@pytest.mark.parametrize("size", [24, 64, 65, 40, 129])
def test_keys_just_inside_and_just_outside_the_window(size, dk, dv, monkeypatch):
    """marks at the sequence's start (the first tokens a window keeps and loses), in the middle of pages and where an edge
    falls on a page border; a window that is one token off in either direction changes the marked rows by far more than the
    tolerance.  In prompts (cut at, before and after the edges) and decoded one by one, fp32 and bf16."""
    cfg, w, t, rows = edge_setup(size, dk=dk, dv=dv)
    ref = bo.forward(cfg, w, t)
    real = bo.visible
    for d in (-1, 1):
        monkeypatch.setattr(bo, "visible", lambda i, s, d=d: real(i, s + d))
        assert err(bo.forward(cfg, w, t)[rows], ref[rows]) > 100 * TOL["float32"], d
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


@pytest.mark.parametrize("dk,dv", [(32, 16), (64, 128)])
@pytest.mark.parametrize("size", [None, 704])
def test_far_key_among_hundreds(size, dk, dv):
    """the marked token at position 3 is seen from 700 positions on, through the prompt kernels and through decode rows split
    over several blocks"""
    n = 706
    cfg, w = opposite_setup(att(size=size, heads=2, kv_heads=1, dim=dk, vdim=dv, scale=16.0 / dk), 170)
    g = torch.Generator().manual_seed(171)
    t = torch.randint(0, 62, (n,), generator=g).tolist()
    t[3] = 63
    for p in range(n - 6, n):
        t[p] = 62
    ref = bo.forward(cfg, w, t)
    t_without = list(t)
    t_without[3] = 5
    assert err(bo.forward(cfg, w, t_without)[-6:], ref[-6:]) > 100 * TOL["float32"]       # the far key matters
    for dtype in ("float32", "bfloat16"):
        with Rig(cfg, dtype, weights=w, max_batch_tokens=1024) as rig:
            for cuts in ([n], [300, 2, 250, 148]):                                        # the last six decoded one by one
                got = run_schedule(rig, t, cuts)
                assert off(dtype)(got, ref) < TOL[dtype] and off(dtype)(got[-6:], ref[-6:]) < TOL[dtype]


@pytest.mark.parametrize("d", [16, 64])
def test_distance_bias_and_offset_show(d, monkeypatch):
    """equal scores everywhere (zero queries): a key's weight is sigmoid(offset - r1 ln(1 + r2 d)) alone, so a distance that is
    one off, a bias without its logarithm or a lost offset shows in every row"""
    cfg = config([att(size=90, heads=3, kv_heads=1, dim=d, vdim=d, conv=2)])
    w = bo.random_weights(cfg, 61)
    w["l0.mix.q.norm"] = torch.zeros(d)
    w["l0.mix.r1"] = torch.tensor([2.5, 0.75, 1.5])
    w["l0.mix.r2"] = torch.tensor([0.125, 4.0, 0.015625])
    w["l0.mix.pb"] = torch.tensor([1.0, -0.5, -2.0])
    w["l0.mix.v"] = w["l0.mix.v"] * 4
    t = toks(170, seed=62)
    ref = bo.forward(cfg, w, t)
    real = bo.distance_bias
    for wrong in (lambda d, a, b: real(d + 1, a, b), lambda d, a, b: real(d, a, b) * 0, lambda d, a, b: real(d, b, a)):
        monkeypatch.setattr(bo, "distance_bias", wrong)
        assert err(bo.forward(cfg, w, t)[5:], ref[5:]) > 50 * TOL["float32"]
        monkeypatch.undo()
    assert err(bo.forward(cfg, {**w, "l0.mix.pb": torch.zeros(3)}, t), ref) > 100 * TOL["float32"]
    for dtype in ("float32", "bfloat16"):
        with Rig(cfg, dtype, weights=w) as rig:
            assert off(dtype)(run_schedule(rig, t, [170]), ref) < TOL[dtype]
            assert off(dtype)(run_schedule(rig, t, [60, 2, 50, 33]), ref) < TOL[dtype]


@pytest.mark.parametrize("d", [16, 64])
def test_weights_far_from_one_half(d):
    """offsets that push the sigmoids to both ends: weights near zero do not overflow, weights near one do not sum to one"""
    cfg = config([att(size=80, heads=3, kv_heads=1, dim=d, vdim=d, scale=2.0)])
    w = bo.random_weights(cfg, 63)
    w["l0.mix.pb"] = torch.tensor([40.0, -40.0, -120.0])
    t = toks(150, seed=64)
    ref = bo.forward(cfg, w, t)
    for dtype in ("float32", "bfloat16"):
        with Rig(cfg, dtype, weights=w) as rig:
            for cuts in ([150], [70, 2, 40]):
                got = run_schedule(rig, t, cuts)
                assert bool(torch.isfinite(got).all()) and off(dtype)(got, ref) < TOL[dtype]


def test_long_rows_split_over_blocks_in_decoding():
    """decoding past 512 and 1024 visible keys, under windows that need one, two and three blocks a row and without one: a row's
    attention is computed by several blocks and their partial sums are added"""
    cfg = config([att(size=None, heads=2, kv_heads=1, dim=16, vdim=16, scale=0.4), att(size=600, heads=2, kv_heads=2, dim=16, vdim=40, scale=0.4),
                  att(size=1100, heads=2, kv_heads=1, dim=16, vdim=16), att(size=512, heads=2, kv_heads=1, dim=16, vdim=16)])
    t = toks(1300, seed=165)
    with Rig(cfg, "float32", max_tokens=1344, max_batch_tokens=1344) as rig:
        ref = rig.oracle(t)
        for first, n in ((508, 8), (1020, 8), (596, 8), (1290, 8)):
            lg = run_schedule(rig, t[:first + n], [first])
            assert err(lg[first:], ref[first:first + n]) < TOL["float32"]


def test_first_tokens_of_a_sequence():
    """the first token convolves with zeros and sees itself alone; so does the first token of the next user of its slot"""
    with Rig(FULL, "float32") as rig:
        for n in (1, 2, 3, 4, 6):
            t = toks(n, seed=80 + n)
            assert err(run_schedule(rig, t, [n]), rig.oracle(t)) < TOL["float32"]
            assert err(run_schedule(rig, t, []), rig.oracle(t)) < TOL["float32"]


def test_convolution_inputs_are_carried():
    """convolutions whose oldest tap is the strongest: inputs that are lost, doubled or taken from a neighbour at a cut show in
    the next `taps - 1` rows"""
    cfg = config([att(size=12, conv=4), att(DENSE, size=12, conv=4)])
    w = bo.random_weights(cfg, 65)
    for k in w:
        if k.endswith(".conv"):
            w[k][:, 0] = 2.0
    t = toks(60, seed=66)
    ref = bo.forward(cfg, w, t)
    with Rig(cfg, "float32", weights=w) as rig:
        rig.eng.step([("x", toks(9, seed=67), [])])
        for cuts in ([1, 1, 1, 2, 3, 2, 1, 30, 1, 2], [2, 2, 2, 2], [5, 1, 4, 1, 3, 1, 2, 1]):
            assert err(run_schedule(rig, t, cuts), ref) < TOL["float32"]


def test_close_router_scores_choose_by_score_not_by_weight():
    """scores close to saturation: sigmoid scores of about 1 differ little, but the choice follows their order and the weights
    their values"""
    cfg = config([att(moe(6, 3, 2.0, 16))])
    w = bo.random_weights(cfg, 68)
    w["l0.mlp.router"] = (w["l0.mlp.router"] * 6).to(torch.bfloat16).float()
    t = toks(100, seed=69)
    with Rig(cfg, "float32", weights=w) as rig:
        ref = rig.oracle(t)
        assert err(run_schedule(rig, t, [100]), ref) < TOL["float32"]
        assert err(run_schedule(rig, t, [40, 2]), ref) < TOL["float32"]


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
        if k.endswith((".r1", ".r2")):
            t = 0.2 + 0.3 * t.abs()
        elif "norm" in k:
            t = 0.2 * t
        elif len(s) == 2 and not k.endswith("conv") and k not in ("embed", "pos"):
            t = t * s[-1] ** -0.5
        out[k] = t.to(torch.bfloat16).float()
    return out


def rms1p(x, w, eps):
    return bo.unit_rms(x, eps) * (1 + w)


def test_distance_bias_under_a_softmax_with_a_sink_and_parallel_gated_experts():
    """softmax attention takes the distance bias too (beside a sink); the side-by-side layer takes one-plus RMS norms, softmax
    router scores with a correction, identity experts, a gated shared expert and the gelu-gated feed-forward"""
    cls = made_up("TestBiasSoftmax", {"norm": "rms", "parallel_ff": True, "qk_norm": False, "mask": "window", "dist_bias": True, "sink": True,
                                      "router": "scored", "expert_act": "swiglu", "shared_gate": True})
    H, G, dk, dv, size, E, ident, top = 4, 2, 16, 24, 30, 3, 1, 2
    mx = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": 0.3, "mask": {"size": size}}
    cfg = {"architecture": "TestBiasSoftmax", "vocab": 64, "width": 48, "norm": {"eps": 1e-5}, "residual_mult": 0.6,
           "layers": [{"type": "attention", "mixer": mx, "mlp": {"kind": "moe", "router": {"experts": E, "top": top, "identity": ident, "scale": 1.5},
                                                                  "expert": {"ff": 20}, "shared": {"ff": 28}}},
                      {"type": "attention", "mixer": mx, "mlp": {"kind": "dense", "ff": 40}}]}
    w = random_for(cls, cfg, 501)
    t = toks(130, vocab=64, seed=502)

    def silu(z):
        return z / (1 + torch.exp(-z))

    def gelu(z):
        return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))

    d = {k: v.double() for k, v in w.items()}
    x = d["embed"][t]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms1p(x, d[p + "norm1"], 1e-5)
        q, k, v = (h @ d[p + "mix." + c].T for c in "qkv")
        q, k, v = q.view(-1, H, dk), k.view(-1, G, dk), v.view(-1, G, dv)
        rows = []
        for j in range(len(t)):
            js = bo.visible(j, size)
            of = [a // (H // G) for a in range(H)]
            s = torch.einsum("hd,nhd->hn", q[j], k[js][:, of]) * 0.3
            s = s - bo.distance_bias(torch.tensor([float(j - a) for a in js], dtype=torch.float64), d[p + "mix.r1"], d[p + "mix.r2"])
            a = torch.softmax(torch.cat([s, d[p + "sink"][:, None]], 1), 1)[:, :-1]
            rows.append(torch.einsum("hn,nhd->hd", a, v[js][:, of]).reshape(-1))
        y = torch.stack(rows) @ d[p + "mix.o"].T
        if L["mlp"]["kind"] == "dense":
            f = (gelu(h @ d[p + "mlp.gate"].T) * (h @ d[p + "mlp.up"].T)) @ d[p + "mlp.down"].T
        else:
            s = torch.softmax(h @ d[p + "router"].T, 1)
            f = torch.sigmoid(h @ d[p + "shared.sg"].T) * ((silu(h @ d[p + "shared.gate"].T) * (h @ d[p + "shared.up"].T)) @ d[p + "shared.down"].T)
            for n in range(len(t)):
                c = torch.topk(s[n] + d[p + "router.corr"], top).indices.tolist()
                tot = float(s[n, c].sum())
                for e in c:
                    o = h[n] if e >= E else (silu(d[f"{p}mlp.e{e}.gate"] @ h[n]) * (d[f"{p}mlp.e{e}.up"] @ h[n])) @ d[f"{p}mlp.e{e}.down"].T
                    f[n] += float(s[n, e]) / tot * 1.5 * o
        x = x + 0.6 * (y + f)
    ref = rms1p(x, d["final.norm"], 1e-5) @ d["head"].T
    for dtype in ("float32", "bfloat16"):
        with Rig(cfg, dtype, weights=w) as rig:
            assert off(dtype)(run_schedule(rig, t, [130]), ref) < TOL[dtype]
            assert off(dtype)(run_schedule(rig, t, [50, 2, 40]), ref) < TOL[dtype]


def test_sigmoid_weights_in_sequential_layers_with_capped_scores_and_gated_heads():
    """sigmoid weights under a block mask, capped scores, gated heads, q / k norms over the whole projection; scalar norms
    before each of two sublayers; the residual factor where each joins; learned positions beside a scaled embedding"""
    cls = made_up("TestSigmoidSeq", {"norm": "rms_scalar", "qk_norm": True, "mask": "block", "attn_weight": "sigmoid", "head_gate": True, "ff_act": "relu2"})
    H, G, dk, dv, chunk = 4, 1, 16, 8, 24
    mx = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": 1.0, "softcap": 3.0, "conv": 2, "mask": {"size": chunk}}
    cfg = {"architecture": "TestSigmoidSeq", "vocab": 64, "width": 48, "norm": {"eps": 1e-5}, "residual_mult": 0.7, "max_positions": 140,
           "embedding": {"scale": 1.5}, "layers": [{"type": "attention", "mixer": mx, "mlp": {"kind": "dense", "ff": 40}}] * 2}
    w = random_for(cls, cfg, 503)
    t = toks(130, vocab=64, seed=504)
    d = {k: v.double() for k, v in w.items()}
    x = 1.5 * d["embed"][t] + d["pos"][:len(t)]
    for i in range(2):
        p = f"l{i}."
        h = bo.scalar_rms_norm(x, d[p + "norm1"], 1e-5)
        q, k, v = (bo.short_convolution(h @ d[f"{p}mix.{c}"].T, d[f"{p}mix.{c}.conv"]) for c in "qkv")
        q, k = bo.unit_rms(q, 1e-5) * d[p + "mix.q.norm"], bo.unit_rms(k, 1e-5) * d[p + "mix.k.norm"]
        q = q.view(-1, H, dk)
        gate = torch.sigmoid(h @ d[p + "head_gate"].T)
        rows = []
        for j in range(len(t)):
            js = list(range(j // chunk * chunk, j + 1))
            s = torch.einsum("hd,nd->hn", q[j], k[js])
            a = bo.key_weights(3.0 * torch.tanh(s / 3.0), d[p + "mix.pb"])
            rows.append((gate[j][:, None] * (a @ v[js])).reshape(-1))
        x = x + 0.7 * torch.stack(rows) @ d[p + "mix.o"].T
        h = bo.scalar_rms_norm(x, d[p + "norm2"], 1e-5)
        x = x + 0.7 * (bo.squared_relu(h @ d[p + "mlp.up"].T + d[p + "mlp.up.b"]) @ d[p + "mlp.down"].T + d[p + "mlp.down.b"])
    ref = bo.scalar_rms_norm(x, d["final.norm"], 1e-5) @ d["head"].T
    for dtype in ("float32", "bfloat16"):
        with Rig(cfg, dtype, weights=w) as rig:
            assert off(dtype)(run_schedule(rig, t, [130]), ref) < TOL[dtype]
            assert off(dtype)(run_schedule(rig, t, [50, 2, 40]), ref) < TOL[dtype]


# -- the token loop, the command lines, the runtime ----------------------------------------------------------------------------
def greedy_agrees(cfg, w, prompt, got, margin=1e-3):
    seq = list(prompt)
    for tok in got:
        lg = bo.forward(cfg, w, seq)[-1]
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


def test_generation_up_to_the_last_position():
    from dnet_b200.shard.batching import GenRequest

    cfg = config([att(DENSE)], positions=40)
    with Rig(cfg, "float32", max_tokens=128) as rig:
        r = GenRequest("g", toks(35, seed=106), max_new_tokens=6)        # feeds the positions 0 .. 39
        greedy_agrees(cfg, rig.w, r.prompt, rig.eng.generate([r])["g"])
        with pytest.raises(ValueError, match="40 positions"):
            rig.eng.generate([GenRequest("h", toks(35, seed=106), max_new_tokens=7)])
        assert rig.model.free_slots == 4


def test_command_lines_on_a_checkpoint_folder(tmp_path):
    """bin/trace_run and bin/generate on a folder with config.json and model.safetensors: the class is picked by the
    config's architecture; norms are scalars in the file"""
    import json
    import os
    import struct
    import subprocess
    import sys

    import numpy as np

    cfg = config([att(DENSE), att(moe())])
    w = bo.random_weights(cfg, 110)
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
    ref = bo.forward(cfg, w, t)
    got = [torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"]) for i in range(3)]
    assert err(got[0], ref[[49]]) < TOL["float32"]
    assert err(got[1], torch.cat([ref[[50, 51]], bo.forward(cfg, w, t[:9])[[8]]])) < TOL["float32"]
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

    w = bo.random_weights(FULL, 21)
    n = len(FULL["layers"])
    rt = ShardRuntime(shard_id="s0", queue_size=64)
    rt.kv_cache_config.max_tokens = 256
    src = HostDictSource({k: v.to(torch.bfloat16) for k, v in w.items()}, FULL)
    rt.load_model_core(ShardLoadModelRequest(model_path=src, total_layers=n, layers=list(range(n)), window_size=n, residency_size=n, kv_bits="fp16"))
    try:
        assert isinstance(rt.policy, BatchedStepPolicy)
        a, b = toks(45, seed=180), toks(70, seed=181)
        out_a = [t for t, _, _ in ring_generate([rt], "na", a, 5)]
        greedy_agrees(FULL, w, a, out_a, margin=5e-2 * float(bo.forward(FULL, w, a)[-1].std()))
        for part in (b[:30], b[30:64]):
            rt.policy.process(token_message(rt, "nb", part, more=True))
            with pytest.raises(queue.Empty):
                rt.activation_send_queue.get_nowait()
        out_b = [t for t, _, _ in ring_generate([rt], "nb", b[64:], 4)]
        greedy_agrees(FULL, w, b, out_b, margin=5e-2 * float(bo.forward(FULL, w, b)[-1].std()))
        rt.release_nonce("na")
        rt.release_nonce_deferred("nb")
        assert rt.model.free_pages == rt.model.pool_pages
    finally:
        assert rt.unload_model_core().success
