"""bench_tuguvik.py -- `bench.py --config tuguvik`: prefill and decode throughput of the Tuguvik family (latent attention with
sinks, gated heads and borrowed rows beside differential attention under a window that keeps the first tokens; dynamic-tanh
norms, channel scales, a silu-gated feed-forward and a gated token row per layer) beside the families of this framework whose
kernels are like its own, at equal width, heads, layers and feed-forward width: Moputar (GQA softmax attention, a gated dense
feed-forward, the residual joined by a kernel of its own) and Lutesun (latent attention over a cached row of the same size).
Random weights, synthetic tokens, one GPU.

Per size: prefill (one P-token prompt in one step), decode of one and of four sequences at the end of a P-token context, and
the device time of every phase of the step (the library's phase timers) with its algorithmic FLOPs or bytes and the fraction
of the measured peak.  Three Tuguvik models are run: the two layer types in turn, and each type alone, so that an attention
phase can be held against the like phase of the family that has only that kind.
"""
from __future__ import annotations

from bench_bokenex import moputar_small_phases
from bench_lutesun import KV_RANK, ROT, WINDOW, _run_lutesun, lutesun_algorithmic
from bench_seqmix import HD, SIZES, VOCAB, _Flusher, _rand, _roofline, _run_moputar, _timed, moputar_algorithmic

KEEP, SIDE, MAP_DIM = 4, 256, 64


def tuguvik_config(sz: dict, kind: str) -> dict:
    """6 layers.  Differential layers: two maps of 64 per head over values of 128 (projections as wide as plain heads of 128);
    latent layers as the Lutesun workload's (128 unrotated + 64 rotated dims over a latent of 512), every third one reading the
    rows of the latent layer before it.  Both under a window of 1,024 positions."""
    W, H, G, ff = sz["width"], sz["heads"], sz["kv_heads"], sz["ff"]
    dense = {"kind": "dense", "ff": ff}
    dif = {"type": "attention", "mlp": dense,
           "mixer": {"heads": H, "kv_heads": G, "dim": MAP_DIM, "vdim": HD, "scale": MAP_DIM ** -0.5, "diff": 0.4, "mask": {"size": WINDOW, "keep_first": KEEP},
                     "rot": {"base": 500000.0, "dims": MAP_DIM, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}}
    mx = {"heads": H, "dim": HD, "rot_dim": ROT, "vdim": HD, "kv_rank": KV_RANK, "q_rank": max(256, W // 2), "scale": (HD + ROT) ** -0.5, "mask": {"size": WINDOW},
          "rot": {"base": 10000.0, "dims": ROT, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    lat = lambda src=None: {"type": "latent_attention", "mlp": dense, "mixer": mx if src is None else {**mx, "kv_from": src}}
    layers = {"mixed": [lat(), dif, dif, lat(0), dif, lat()], "latent": [lat(), lat(), lat(1), lat(), lat(), lat(4)], "differential": [dif] * 6}[kind]
    return {"architecture": "Tuguvik", "vocab": VOCAB, "width": W, "norm": {"eps": 1e-5}, "token_side": {"dim": SIDE}, "layers": layers}


def tuguvik_weights(model, g, dev):
    import torch

    items = []
    for name, shape in model.expected_tensors().items():
        leaf = name.split(".", 1)[-1]
        if leaf in ("norm1", "norm2", "side.norm") or leaf.endswith(("dq.norm", "dkv.norm")) or name == "final.norm":
            t = torch.ones(shape, dtype=torch.bfloat16, device=dev)
        elif leaf.endswith("alpha"):
            t = torch.full(shape, 0.6, dtype=torch.bfloat16, device=dev)
        elif leaf in ("ls1", "ls2"):
            t = torch.full(shape, 0.5, dtype=torch.bfloat16, device=dev)
        elif len(shape) == 1:
            t = _rand(shape, g, 0.1, dev)
        elif name in ("embed", "side.embed"):
            t = _rand(shape, g, 1.0, dev)
        else:
            t = _rand(shape, g, shape[-1] ** -0.5, dev)
        items.append((name, t))
    return items


def tuguvik_algorithmic(cfg: dict, N: int, ctx0: int, n_seqs: int) -> dict:
    """FLOPs and the bytes that must move per phase, for a step of n_seqs entries x (N / n_seqs) tokens whose sequences already
    hold ctx0 tokens each; summed over the layers.  Latent attention is counted as in lutesun_algorithmic; a differential head as
    two score rows and two weighted sums over its value.  The output and down products include the residual that they read and
    write, fp32, and the normed row that they leave."""
    W = cfg["width"]
    side = cfg["token_side"]["dim"]
    f = {k: 0.0 for k in ("proj", "attn_prep", "latent_in", "attn", "latent_out", "out_proj", "ff_up", "ff_down", "side")}
    by = dict(f)
    per = N // n_seqs
    for L in cfg["layers"]:
        mx = L["mixer"]
        H, dv, win = mx["heads"], mx["vdim"], mx["mask"]["size"]
        vis = sum(min(p + 1, win) for p in range(ctx0, ctx0 + per)) * n_seqs
        keys = n_seqs * min(ctx0 + per, win + per - 1)
        if L["type"] == "attention":
            G, dk = mx["kv_heads"], mx["dim"]
            cols = 2 * H * dk + G * (2 * dk + dv)
            f["proj"] += 2.0 * N * W * cols
            by["proj"] += 2.0 * W * cols
            by["attn_prep"] += 4.0 * N * cols
            f["attn"] += 2.0 * 2 * (dk + dv) * H * vis
            by["attn"] += 2.0 * keys * G * (2 * dk + dv) + 2.0 * N * H * (2 * dk + dv)
        else:
            dn, dr, R, qr = mx["dim"], mx["rot_dim"], mx["kv_rank"], mx["q_rank"]
            own = 0 if "kv_from" in mx else R + dr
            cq = H * (dn + dr)
            wq = W * qr + qr * cq + W * (own + H)
            f["proj"] += 2.0 * N * wq
            by["proj"] += 2.0 * wq
            f["latent_in"] += 2.0 * N * H * dn * R
            by["latent_in"] += 2.0 * H * dn * R + 2.0 * N * (cq + H * (R + dr))
            f["attn"] += 2.0 * (2 * R + dr) * H * vis
            by["attn"] += 2.0 * keys * (R + dr) + 2.0 * N * H * (2 * R + dr)
            f["latent_out"] += 2.0 * N * H * dv * R
            by["latent_out"] += 2.0 * H * dv * R + 2.0 * N * H * (R + dv)
        f["out_proj"] += 2.0 * N * W * H * dv
        by["out_proj"] += 2.0 * W * H * dv + 10.0 * N * W
        ff = L["mlp"]["ff"]
        f["ff_up"] += 4.0 * N * W * ff
        by["ff_up"] += 4.0 * W * ff
        f["ff_down"] += 2.0 * N * W * ff
        by["ff_down"] += 2.0 * W * ff + 10.0 * N * W
        f["side"] += 4.0 * N * W * side
        by["side"] += 4.0 * W * side + N * (W * (2.0 + 8.0 + 8.0 + 2.0) + 6.0 * side)
    return {"flops": f, "bytes": by}


def _run_tuguvik(sz: dict, kind: str, args, P: int, flush, dev) -> dict:
    import torch

    from dnet_b200.core.models import get_ring_model

    cfg = tuguvik_config(sz, kind)
    pages = 4 * ((P + 64 + 63) // 64)
    model = get_ring_model("tuguvik", cfg, assigned_layers=list(range(len(cfg["layers"]))), dtype="bfloat16", kv_pool_pages=pages,
                           max_seqs=4, max_batch_tokens=max(P, 64))
    g = torch.Generator(device=dev).manual_seed(7)
    model.load_weights(tuguvik_weights(model, g, dev), strict=True)
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

    res = {"config": {"layers": [l["type"] + ("(borrowed rows)" if "kv_from" in l["mixer"] else "") for l in cfg["layers"]], "window": WINDOW, "keep_first": KEEP,
                      "side": SIDE, "map_dim": MAP_DIM, "kv_rank": KV_RANK}}
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


def run_tuguvik(args, rank: int, local_rank: int, world: int) -> None:
    import time

    import torch

    import bench as B
    import bench_seqmix as BS
    from bench import ClockSampler, log

    if world != 1:
        raise SystemExit("--config tuguvik runs on one GPU")
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
            runs = {"tuguvik": _run_tuguvik(sz, "mixed", args, P, flush, dev), "tuguvik_latent": _run_tuguvik(sz, "latent", args, P, flush, dev),
                    "tuguvik_differential": _run_tuguvik(sz, "differential", args, P, flush, dev), "moputar": _run_moputar(sz, args, P, flush, dev),
                    "lutesun": _run_lutesun(sz, args, P, flush, dev)}
        side.synchronize()
        cfgs = {k: r.pop("cfg") for k, r in runs.items()}
        launches += sum(r.pop("launches") for r in runs.values())
        for key in ("prefill", "decode_bs1", "decode_bs4"):
            n_seq = 4 if key.endswith("4") else 1
            N, ctx0 = (P, 0) if key == "prefill" else (n_seq, runs["tuguvik"][key]["context"])
            for fam, r in runs.items():
                c = cfgs[fam]
                alg = moputar_small_phases(moputar_algorithmic(c, N, ctx0, n_seq), c, N) if fam == "moputar" else \
                    lutesun_algorithmic(c, N, ctx0, n_seq) if fam == "lutesun" else tuguvik_algorithmic(c, N, ctx0, n_seq)
                r[key]["roofline"] = _roofline(r[key]["phases_ms"], alg, tf, gbs, f32_tf)
                log(f"{name} {key} {fam}: {r[key]['ms']:.3f} ms ({r[key]['tok_s']:,.0f} tok/s)  " +
                    ", ".join(f"{k} {v['ms']:.3f}ms/{v['frac']:.3f}" for k, v in r[key]["roofline"].items()))
                log("      phases " + ", ".join(f"{k} {v:.3f}" for k, v in r[key]["phases_ms"].items() if v > 0))
            for other in ("moputar", "lutesun"):
                runs["tuguvik"][key]["vs_" + other] = round(runs["tuguvik"][key]["tok_s"] / runs[other][key]["tok_s"], 4)
        sizes[name] = {"dims": sz, **runs}
    tw1 = time.perf_counter()
    head = sizes[args.seqmix_sizes.split(",")[-1]]
    out = {"metric": "prefill tok/s Tuguvik (layer-list family) beside Moputar and Lutesun at equal size, one prompt in one step",
           "value": head["tuguvik"]["prefill"]["tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
           "ms_per_step": head["tuguvik"]["prefill"]["ms"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16",
           "data": "synthetic",
           "config": {"model": "Tuguvik, random weights", "prompt_len": P, "sizes": args.seqmix_sizes,
                      "timing": "CUDA events around each step, a 256 MB buffer written between steps (L2 flush)",
                      "peaks": {"bf16_tflops": tf, "hbm_gbs": gbs, "source": peak_src, "fp32_tflops_nominal": round(f32_tf, 1)}},
           "gpu_launches": launches, "sizes": sizes, "clocks": sampler.summary(tw0, tw1)}
    sampler.stop()
    B.emit(out)
