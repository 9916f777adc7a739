"""bench_bokenex.py -- `bench.py --config bokenex`: prefill and decode throughput of the Bokenex family (windowed GQA
attention with short convolutions, sigmoid weights and a logarithmic distance bias; mixer and feed-forward side by side on
one scalar RMS norm; a dense relu-squared feed-forward or sigmoid-routed experts) beside Moputar, the closest family of
this framework (same library, same ragged-batch step, GQA attention with short convolutions and q / k norms, a dense
feed-forward), at equal width, heads, layers and feed-forward width -- and beside Lutesun, whose routed experts and
relu-squared feed-forward are the like kernels of Bokenex's.  Random weights, synthetic tokens, one GPU.

Per size: prefill (one P-token prompt in one step), decode of one and of four sequences at the end of a P-token
context, and the device time of every phase of the step (the library's phase timers) with its algorithmic FLOPs or
bytes and the fraction of the measured peak, for the three families.
"""
from __future__ import annotations

from bench_lutesun import _run_lutesun, lutesun_algorithmic
from bench_seqmix import HD, SIZES, VOCAB, _Flusher, _rand, _roofline, _run_moputar, _timed, moputar_algorithmic

WINDOW, CONV, EXPERTS, TOP = 1024, 4, 16, 4


def bokenex_config(sz: dict, P: int) -> dict:
    """6 layers, the dense and the routed feed-forward in turn; heads of 128 under a window of 1,024 positions; the active
    width of the routed layers (top x expert width) equals the dense width of the size"""
    W, H, G, ff = sz["width"], sz["heads"], sz["kv_heads"], sz["ff"]
    mx = {"heads": H, "kv_heads": G, "dim": HD, "vdim": HD, "conv": CONV, "scale": HD ** -0.5, "mask": {"size": WINDOW}}
    dense = {"type": "attention", "mixer": mx, "mlp": {"kind": "dense", "ff": ff}}
    moe = {"type": "attention", "mixer": mx, "mlp": {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP, "scale": 2.0}, "expert": {"ff": ff // TOP}}}
    return {"architecture": "Bokenex", "vocab": VOCAB, "width": W, "norm": {"eps": 1e-5}, "residual_mult": 0.4, "max_positions": 2 * P + 1024,
            "layers": [dense, moe] * 3}


def bokenex_weights(model, g, dev):
    import torch

    items = []
    for name, shape in model.expected_tensors().items():
        leaf = name.split(".", 1)[-1]
        if leaf in ("norm1", "mix.q.norm", "mix.k.norm") or name == "final.norm":
            t = torch.ones(shape, dtype=torch.bfloat16, device=dev)
        elif leaf in ("mix.r1", "mix.r2"):
            t = _rand(shape, g, 0.3, dev).abs()
        elif leaf == "mix.pb":
            t = _rand(shape, g, 0.5, dev) - 5.0
        elif leaf.endswith(".conv"):
            t = _rand(shape, g, 0.5, dev)
        elif name in ("embed", "pos"):
            t = _rand(shape, g, 1.0 if name == "embed" else 0.3, dev)
        else:
            t = _rand(shape, g, shape[-1] ** -0.5, dev)
        items.append((name, t))
    return items


def bokenex_algorithmic(cfg: dict, N: int, ctx0: int, n_seqs: int) -> dict:
    """FLOPs and the bytes that must move per phase, for a step of n_seqs entries x (N / n_seqs) tokens whose
    sequences already hold ctx0 tokens each; summed over the layers.  In steps of up to 8 tokens a dense layer's up (down)
    product runs in the projections' (output product's) launch."""
    W = cfg["width"]
    f = {k: 0.0 for k in ("proj", "attn_prep", "attn", "out_proj", "ff_up", "ff_down", "moe_up", "moe_down", "write_back")}
    by = dict(f)
    per = N // n_seqs
    for L in cfg["layers"]:
        mx, mlp = L["mixer"], L.get("mlp")
        H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        cols, co, win = H * dk + G * (dk + dv), H * dv, mx["mask"]["size"]
        f["proj"] += 2.0 * N * W * cols
        by["proj"] += 2.0 * W * cols
        by["attn_prep"] += 4.0 * N * cols + 2.0 * mx["conv"] * cols
        vis = sum(min(p + 1, win) for p in range(ctx0, ctx0 + per)) * n_seqs
        f["attn"] += 2.0 * (dk + dv) * H * vis
        by["attn"] += 2.0 * n_seqs * min(ctx0 + per, win + per - 1) * G * (dk + dv) + 2.0 * N * (H * dk + co)
        f["out_proj"] += 2.0 * N * co * W
        by["out_proj"] += 2.0 * co * W
        by["write_back"] += N * W * (8.0 + 4.0 + 2.0)
        if not mlp:
            continue
        if mlp["kind"] == "dense":
            by["write_back"] += 4.0 * N * W
            for a, b in (("ff_up", "proj"), ("ff_down", "out_proj")):
                k = b if N <= 8 else a
                f[k] += 2.0 * N * W * mlp["ff"]
                by[k] += 2.0 * W * mlp["ff"]
            continue
        E, top, ef = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
        by["write_back"] += 4.0 * top * N * W
        hit = E * (1.0 - (1.0 - top / E) ** N)      # experts that N tokens reach, on average
        for k in ("moe_up", "moe_down"):
            f[k] += 2.0 * N * top * W * ef
            by[k] += 2.0 * hit * W * ef
    return {"flops": f, "bytes": by}


def moputar_small_phases(alg: dict, cfg: dict, N: int) -> dict:
    """adds the bytes of Moputar's prep and write-back phases, counted as Bokenex's are"""
    W, S = cfg["width"], max(1, cfg.get("streams", 0))
    a = w = 0.0
    for L in cfg["layers"]:
        mx = L["mixer"]
        w += (2 if L.get("mlp") else 1) * N * W * (8.0 * S + 4.0)
        if L["type"] == "attention":
            cols = mx["heads"] * mx["dim"] + (0 if "kv_from" in mx else mx["kv_heads"] * (mx["dim"] + mx["vdim"]))
            a += 4.0 * N * cols + 2.0 * mx["conv"] * cols
    for k, v in (("attn_prep", a), ("write_back", w)):
        alg["flops"][k], alg["bytes"][k] = 0.0, v
    return alg


def _run_bokenex(sz: dict, args, P: int, flush, dev) -> dict:
    import torch

    from dnet_b200.core.models import get_ring_model

    cfg = bokenex_config(sz, P)
    pages = 4 * ((P + 64 + 63) // 64)
    model = get_ring_model("bokenex", cfg, assigned_layers=list(range(len(cfg["layers"]))), dtype="bfloat16", kv_pool_pages=pages,
                           max_seqs=4, max_batch_tokens=max(P, 64))
    g = torch.Generator(device=dev).manual_seed(7)
    model.load_weights(bokenex_weights(model, g, dev), strict=True)
    assert not model.missing_tensors()
    prompt = torch.randint(0, VOCAB, (P,), generator=torch.Generator().manual_seed(11)).tolist()
    K, Wm = args.steps, args.warmup
    live = []
    st = torch.cuda.current_stream()

    def fresh(n):
        for h in live:
            h.free()
        live.clear()
        live.extend(model.make_cache(stream=st) for _ in range(n))

    res = {"config": {"layers": [l["mlp"]["kind"] for l in cfg["layers"]], "window": WINDOW, "conv": CONV, "experts": EXPERTS, "top": TOP}}
    t = _timed(lambda: model.step([(live[0], prompt)], [P - 1], stream=st), lambda: fresh(1), K, Wm, flush)
    res["prefill"] = {"ms": t, "tok_s": P / t * 1e3}
    fresh(1)
    model.profile(True)
    model.step([(live[0], prompt)], [P - 1], stream=st)
    res["prefill"]["phases_ms"] = model.profile_read(reset=True)
    model.profile(False)
    for n_seq in (1, 4):
        ctx = (P if n_seq == 1 else P // 4) - 1
        fresh(n_seq)
        model.step([(h, prompt[:ctx]) for h in live], [], stream=st)
        toks = [[int(prompt[(i * 7 + 3) % P])] for i in range(n_seq)]
        want = list(range(n_seq))
        t = _timed(lambda: model.step([(h, toks[i]) for i, h in enumerate(live)], want, stream=st), lambda: None, K, Wm, flush)
        key = "decode_bs%d" % n_seq
        res[key] = {"ms": t, "tok_s": n_seq / t * 1e3, "context": ctx}
        model.profile(True)
        for _ in range(4):
            flush()
            model.step([(h, toks[i]) for i, h in enumerate(live)], want, stream=st)
        ph = model.profile_read(reset=True)
        model.profile(False)
        res[key]["phases_ms"] = {k: v / 4 for k, v in ph.items()}
    model.check(st)
    fresh(0)
    launches = int(model._lib.dn_seq_launch_count())
    model.destroy()
    res["cfg"] = cfg
    res["launches"] = launches
    return res


def run_bokenex(args, rank: int, local_rank: int, world: int) -> None:
    import time

    import torch

    import bench as B
    import bench_seqmix as BS
    from bench import ClockSampler, log

    if world != 1:
        raise SystemExit("--config bokenex runs on one GPU")
    dev = torch.device("cuda", local_rank)
    P = int(args.seqmix_prompt)
    gbs, peak_src = B.peaks()
    tf = B.tensor_peak_tf()
    props = torch.cuda.get_device_properties(dev)
    f32_tf = props.multi_processor_count * 128 * 2 * 1.965e9 / 1e12
    flush = _Flusher(dev)
    side = torch.cuda.Stream(device=dev)
    sampler = ClockSampler(local_rank)
    sampler.start()
    tw0 = time.perf_counter()
    BS.FP32_PHASES = ("recur", "delta_rule")
    sizes, launches = {}, 0
    for name in args.seqmix_sizes.split(","):
        sz = SIZES[name]
        with torch.cuda.stream(side):
            bk = _run_bokenex(sz, args, P, flush, dev)
            mo = _run_moputar(sz, args, P, flush, dev)
            lu = _run_lutesun(sz, args, P, flush, dev)
        side.synchronize()
        launches += bk.pop("launches") + mo.pop("launches") + lu.pop("launches")
        bcfg, mcfg, lcfg = bk.pop("cfg"), mo.pop("cfg"), lu.pop("cfg")
        for key in ("prefill", "decode_bs1", "decode_bs4"):
            n_seq = 4 if key.endswith("4") else 1
            N, ctx0 = (P, 0) if key == "prefill" else (n_seq, bk[key]["context"])
            bk[key]["roofline"] = _roofline(bk[key]["phases_ms"], bokenex_algorithmic(bcfg, N, ctx0, n_seq), tf, gbs, f32_tf)
            mo[key]["roofline"] = _roofline(mo[key]["phases_ms"], moputar_small_phases(moputar_algorithmic(mcfg, N, ctx0, n_seq), mcfg, N), tf, gbs, f32_tf)
            lu[key]["roofline"] = _roofline(lu[key]["phases_ms"], lutesun_algorithmic(lcfg, N, ctx0, n_seq), tf, gbs, f32_tf)
            bk[key]["vs_moputar"] = round(bk[key]["tok_s"] / mo[key]["tok_s"], 4)
            log(f"{name} {key}: bokenex {bk[key]['ms']:.3f} ms ({bk[key]['tok_s']:,.0f} tok/s), moputar {mo[key]['ms']:.3f} ms ({mo[key]['tok_s']:,.0f} tok/s), "
                f"lutesun {lu[key]['ms']:.3f} ms ({lu[key]['tok_s']:,.0f} tok/s)")
            for fam, r in (("bokenex", bk), ("moputar", mo), ("lutesun", lu)):
                log(f"   {fam} " + ", ".join(f"{k} {v['ms']:.3f}ms/{v['frac']:.3f}" for k, v in r[key]["roofline"].items()))
            log("   bokenex phases " + ", ".join(f"{k} {v:.3f}" for k, v in bk[key]["phases_ms"].items() if v > 0))
            log("   moputar phases " + ", ".join(f"{k} {v:.3f}" for k, v in mo[key]["phases_ms"].items() if v > 0))
            log("   lutesun phases " + ", ".join(f"{k} {v:.3f}" for k, v in lu[key]["phases_ms"].items() if v > 0))
        sizes[name] = {"dims": sz, "bokenex": bk, "moputar": mo, "lutesun": lu}
    tw1 = time.perf_counter()
    head = sizes[args.seqmix_sizes.split(",")[-1]]
    out = {"metric": "prefill tok/s Bokenex (layer-list family) beside Moputar at equal size, one prompt in one step",
           "value": head["bokenex"]["prefill"]["tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
           "ms_per_step": head["bokenex"]["prefill"]["ms"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
           "data": "synthetic",
           "config": {"model": "Bokenex, random weights", "prompt_len": P, "sizes": args.seqmix_sizes,
                      "timing": "CUDA events around each step, a 256 MB buffer written between steps (L2 flush)",
                      "peaks": {"bf16_tflops": tf, "hbm_gbs": gbs, "source": peak_src, "fp32_tflops_nominal": round(f32_tf, 1)}},
           "gpu_launches": launches, "sizes": sizes, "clocks": sampler.summary(tw0, tw1)}
    sampler.stop()
    B.emit(out)
