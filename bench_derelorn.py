"""`bench.py --workload derelorn`: prefill and decode throughput of the Derelorn design at sizes that resemble a real model's
layers (random weights), beside the Sefevik model of equal width, depth and parameter count, and each kernel's time against
its roofline beside the like kernel of that model.

Decode: one captured step (device-side bookkeeping, embedding, layers, head, arg-max, the token fed back) of `batch`
sequences.  Prefill: `prompts` prompts of `prompt_len` tokens in one forward, logits of the last tokens, arg-max.  The
end-to-end figure goes through Engine.step: host token ids in, logits' arg-max back, every step.
"""
from __future__ import annotations

import json
import time

import numpy as np
import torch

import bench_hybrid as bh
from bench_hybrid import captured, contiguous_tables, peaks, prompt_meta, timed

# (mlstm, parallel, mlstm, delta) repeated; mlstm heads x (dim, vdim), attention heads / kv, Mamba-2 heads x (state, vdim), delta heads / kv
SIZES = {
    "0.3B": dict(width=1024, depth=12, ff=2816, vocab=32768, mlstm=(4, 128, 256), attn=(16, 4, 64, 512), mamba=(32, 64, 64, 1), delta=(8, 4, 128, 128)),
    "1.4B": dict(width=2048, depth=24, ff=5632, vocab=32768, mlstm=(8, 128, 256), attn=(16, 4, 128, 1024), mamba=(64, 64, 128, 1), delta=(16, 8, 128, 128)),
    "4B": dict(width=4096, depth=16, ff=11264, vocab=65536, mlstm=(16, 128, 256), attn=(32, 8, 128, 1024), mamba=(128, 64, 128, 1), delta=(32, 16, 128, 128)),
}
TAPS = 4


def derelorn_config(s: dict) -> dict:
    layers = []
    for i in range(s["depth"]):
        kind = ("mlstm", "parallel", "mlstm", "delta")[i % 4]
        if kind == "mlstm":
            m = dict(zip(("heads", "dim", "vdim"), s["mlstm"]), gate_cap=15.0)
        elif kind == "delta":
            m = dict(zip(("heads", "kv_heads", "dim", "vdim"), s["delta"]), conv=TAPS)
        else:
            h, g, d, w = s["attn"]
            mh, v, n, groups = s["mamba"]
            m = {"left": {"heads": h, "kv_heads": g, "dim": d, "vdim": d, "scale": d ** -0.5, "mask": {"size": w}},
                 "right": {"heads": mh, "vdim": v, "state": n, "groups": groups, "conv": TAPS, "norm_groups": 1}}
        layers.append({"type": kind, "mixer": m, "mlp": {"kind": "dense", "ff": s["ff"]}})
    return {"architecture": "Derelorn", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "layers": layers}


def closest_shape(s: dict, params: int) -> dict:
    """The Sefevik size of the same width and depth whose feed-forward makes the parameter counts meet."""
    base = next(z for z in bh.SIZES.values() if z["width"] == s["width"])
    W, heads = s["width"], base["heads"]
    gru = 4 * W * base["gru"]
    att = W * (heads * (base["dim"] + base["rot"]) + base["rank"] + base["rot"]) + heads * base["rank"] * (base["dim"] + base["vdim"]) + heads * base["vdim"] * W
    n_att = sum(i % 3 == 2 for i in range(s["depth"]))
    rest = params - s["vocab"] * W - (s["depth"] - n_att) * gru - n_att * att
    return {**base, "depth": s["depth"], "vocab": s["vocab"], "ff": max(128, int(round(rest / (2 * W * s["depth"]) / 128)) * 128)}


def build(s: dict, pages: int, batch: int):
    from mini_sgl_integer_b200.kvcache.hybrid_pool import HybridCache
    from mini_sgl_integer_b200.models.config import DerelornConfig
    from mini_sgl_integer_b200.models.derelorn import DerelornForCausalLM, random_weights
    cfg = DerelornConfig.from_dict(derelorn_config(s))
    sd = random_weights(cfg, 3, device="cuda")
    params = sum(v.numel() for k, v in sd.items() if k != "embed")
    model = DerelornForCausalLM(cfg, torch.bfloat16, "cuda")
    model.load_state_dict(sd)
    cache = HybridCache(cfg, pages, batch, torch.bfloat16, "cuda")
    for i, m in enumerate(cfg.memory):
        if m.planes:
            cache.k_cache(i).normal_()
            cache.v_cache(i).normal_()
        for name, _ in m.state:
            cache.state(i, name).normal_().mul_(0.1)
    return cfg, model, cache, params


def decode(s: dict, cfg, model, cache, table, lens, max_len: int, steps: int, warmup: int, weights: int) -> dict:
    from mini_sgl_integer_b200 import _lib
    from mini_sgl_integer_b200.attention.hybrid_backend import HybridMetadata
    from mini_sgl_integer_b200.kernel.float_ops import argmax_f32
    from mini_sgl_integer_b200.kvcache.hybrid_pool import HybridCache
    from mini_sgl_integer_b200.models import DecodeBatch
    B = len(lens)
    state = DecodeBatch(table, torch.from_numpy(lens).cuda(), max_len)
    slots = torch.arange(B, dtype=torch.int32, device="cuda")
    cur = torch.zeros(B, dtype=torch.int32, device="cuda")

    def step():
        b = state.advance()
        md = HybridMetadata(b.positions, b.out_loc, b.page_table, b.kv_lens, slots, None, None, 1, max_len)
        cur.copy_(argmax_f32(model.forward_tokens(cur, md, cache)))
    g = captured(step, 1)
    c0 = _lib.CALLS
    step()
    calls = _lib.CALLS - c0
    ms = timed(g.replay, steps, warmup)
    model.check_status()
    window = cfg.max_window
    kv = float(np.minimum(lens, window).sum()) * sum(h * n * 2 for m in cfg.memory for h, n in m.planes)
    st = 2.0 * B * HybridCache.slot_bytes(cfg)
    gbs = (2.0 * weights + kv + st) / ms / 1e6
    return {"ms": ms, "tok_s": B / ms * 1e3, "weight_bytes": 2 * weights, "kv_bytes": kv, "state_bytes": st, "GBs": gbs, "frac": gbs / peaks()["hbm_gbs"],
            "launches": calls}


# ----------------------------------------------------------------------------- kernels one by one
def kernel_table(s: dict, c: dict, B: int, prompts: int, n: int, ctx: int) -> dict:
    """name -> {us, frac of the roofline, like: {name, us, frac}}.  Inputs and outputs of prompts exceed L2 together; decode
    kernels rotate over copies of what they stream (states, caches)."""
    from mini_sgl_integer_b200.kernel import float_ops as fo
    pk, out, bf = peaks(), {}, torch.bfloat16
    T = prompts * n
    rnd = lambda *sh: torch.randn(sh, device="cuda").to(bf)
    f32 = lambda *sh: torch.randn(sh, device="cuda")

    def frac(ms, bytes_, flops=0.0):
        return max(bytes_ / pk["hbm_gbs"] / 1e6, flops / pk["bf16_tflops"] / 1e9) / ms

    def device_ms(fn, calls=8, reps=4):
        def many():
            for _ in range(calls):
                fn()
        return timed(captured(many, 1).replay, reps) / calls

    def entry(name, ms, bytes_, flops=0.0, like=None):
        out[name] = {"us": ms * 1e3, "frac": frac(ms, bytes_, flops)}
        if like:
            out[name]["like"] = {**like, "ratio": out[name]["frac"] / like["frac"]}
    pos, loc, seq, start, plens = prompt_meta(prompts, n, contiguous_tables(prompts, n)[0])
    one, sl, spr = (torch.ones(B, dtype=torch.int32, device="cuda"), torch.arange(B, dtype=torch.int32, device="cuda"),
                    torch.arange(prompts, dtype=torch.int32, device="cuda"))

    # like kernels of the closest model
    W, gru, rank, rot, H = c["width"], c["gru"], c["rank"], c["rot"], c["heads"]
    like = {}
    for M, prompt in ((B, False), (T, True)):
        zug, bz, y = torch.randn(1, M, 3 * gru, device="cuda"), f32(gru), fo.rows(M, gru, bf, "cuda")
        st = torch.zeros(max(B, prompts), gru, device="cuda")
        ms = device_ms(lambda: fo.mingru(zug, bz, bz, st, spr if prompt else sl, pos if prompt else one, start if prompt else None, prompts if prompt else B, y))
        by = (14.0 if prompt else 22.0) * M * gru
        like["scan", M] = {"name": "minGRU " + ("scan" if prompt else "step"), "us": ms * 1e3, "frac": frac(ms, by)}
        yy, x, nw, xo, xt = f32(1, M, W), f32(M, W), f32(W), f32(M, W), fo.rows(M, W, bf, "cuda")
        ms = device_ms(lambda: fo.sublayer_end(yy, x, nw, 1e-6, xo, xt, bf))
        like["rows", M] = {"name": "sublayer end", "us": ms * 1e3, "frac": frac(ms, 14.0 * M * W)}
        lat, nq = rank + rot, H * (c["dim"] + rot) + rank + rot
        qd, pool, rope = f32(1, M, nq), torch.zeros(M // 16 + 1, 16, lat, dtype=bf, device="cuda"), f32(max(n, 2), rot)
        qn, ql, dn = torch.empty(M, H, c["dim"], dtype=bf, device="cuda"), torch.empty(M, H, lat, dtype=bf, device="cuda"), torch.ones(rank, device="cuda")
        pp, ll = torch.zeros(M, dtype=torch.int32, device="cuda"), torch.arange(M, dtype=torch.int32, device="cuda")
        ms = device_ms(lambda: fo.latent_prepare(qd, pp, ll, rope, dn, 1e-6, qn, ql, pool, H, c["dim"], rot, rank))
        like["prepare", M] = {"name": "latent prepare", "us": ms * 1e3, "frac": frac(ms, M * (4.0 * nq + 2.0 * H * (c["dim"] + rot) + 2.0 * lat))}
        del zug, y, st, yy, x, xo, xt, qd, pool, qn, ql
    table, pages = contiguous_tables(B, -(-ctx // 16) * 16)
    lens = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    lat, sink = rank + rot, torch.zeros(H, device="cuda")
    lc, ql, lo = rnd(pages, 16, lat), rnd(B, H, lat), torch.empty(B, H, rank, dtype=bf, device="cuda")
    seen = min(ctx, c["window"])
    ms = device_ms(lambda: fo.latent_attention(ql, lc, table, lens, None, sink, lo, rank, rot, c["window"], 0.1, 1, ctx))
    like["attn", B] = {"name": "latent attention, decode", "us": ms * 1e3, "frac": frac(ms, 2.0 * B * seen * lat + 2.0 * B * H * (lat + rank), 2.0 * B * seen * H * (lat + rank))}
    ql, lo, tb = rnd(T, H, lat), torch.empty(T, H, rank, dtype=bf, device="cuda"), table[:prompts].contiguous()
    pairs = lambda w: prompts * (min(n, w) * (min(n, w) + 1) / 2 + (n - min(n, w)) * w)
    ms = device_ms(lambda: fo.latent_attention(ql, lc, tb, plens, start, sink, lo, rank, rot, c["window"], 0.1, n, n), calls=4)
    like["attn", T] = {"name": "latent attention, prompts", "us": ms * 1e3,
                       "frac": frac(ms, 2.0 * T * lat + 2.0 * T * H * (lat + rank), 2.0 * pairs(c["window"]) * H * (lat + rank))}
    del lc, ql, lo
    torch.cuda.empty_cache()

    # matrix memories
    mh, md, mv = s["mlstm"]
    dh, dg, dd, dv = s["delta"]
    sh, sv, sn, sg = s["mamba"]
    kinds = {"mLSTM": (fo.MEMORY_EXP, mh, mh, md, mv, 0, fo.GATE_SIGMOID_AFTER), "Mamba-2": (fo.MEMORY_SSD, sh, sg, sn, sv, TAPS, fo.GATE_SILU_BEFORE),
             "gated delta": (fo.MEMORY_DELTA, dh, dg, dd, dv, TAPS, fo.GATE_SILU_AFTER)}
    for name, (kind, h, g, d, v, taps, gate) in kinds.items():
        exp, qk, width = kind == fo.MEMORY_EXP, g * d, 2 * g * d + h * v
        seg = [(qk, d), (qk, d), (h * v, v)]
        cols = -(-(width + 2 * h + h * v) // 8) * 8
        cw, zero, nw = (f32(width, taps) if taps else None), torch.zeros(h, device="cuda"), f32(h * v)
        for M, prompt in ((B, False), (T, True)):
            slots, p_, st_, ids, count = (spr, pos, start, seq, prompts) if prompt else (sl, one, None, None, B)
            parts = 1 if prompt else fo.query("b200f_gemm_splits", M, cols, W, 1, 1)
            y, rows, gates = f32(parts, M, cols), fo.rows(M, width, bf, "cuda"), torch.empty(M, h, 4, device="cuda")
            cs, ns = torch.zeros(count, max(taps - 1, 0), width, device="cuda"), torch.zeros(count, h, d + 1, device="cuda")
            run = lambda: fo.memory_prepare(y, 0, seg, cw, None, cs if taps else None, slots, p_, st_, ids, rows, kind, h, (width, width + h), zero, zero, gates, 15.0,
                                            ns if exp else None)
            by = M * (4.0 * parts * (width + 2 * h) + 2.0 * width + 16.0 * h) + count * 8.0 * max(taps - 1, 0) * width
            entry(f"{name} prepare M={M}", device_ms(run), by, like=like["prepare", M])
            states = [torch.zeros(count, h, d, v, device="cuda") for _ in range(1 if prompt else 2)]
            gates[..., 0] = -0.01
            gates[..., 1] = 0.5
            o, den, k = torch.empty(M, h * v, device="cuda"), torch.empty(M, h, device="cuda"), [0]

            def scan():
                k[0] = (k[0] + 1) % len(states)
                fo.memory_scan(rows, (0, qk, 2 * qk), g, h, d, v, kind, gates, 0.1, None, states[k[0]], ns if exp else None, slots, p_, st_, o, den if exp else None,
                               n if prompt else 1)
            by = M * (2.0 * width + 16.0 * h + 4.0 * h * v) + count * 8.0 * h * d * v
            entry(f"{name} {'scan' if prompt else 'step'} M={M}", device_ms(scan), by, 4.0 * M * h * d * v, like=like["scan", M])
            group = h * v if gate == fo.GATE_SILU_BEFORE else v
            ob = fo.rows(M, h * v, bf, "cuda")
            w_ = nw if gate != fo.GATE_SILU_AFTER else nw[:v].contiguous()
            run = lambda: fo.memory_output(o, den if exp else None, h, v, group, y, width + 2 * h, gate, w_, 1e-6, ob)
            o.normal_()
            den.fill_(1.0)
            entry(f"{name} output M={M}", device_ms(run), M * h * v * (6.0 + 4.0 * parts), like=like["rows", M])
            del y, rows, gates, cs, ns, states, o, den, ob
            torch.cuda.empty_cache()

    # grouped attention
    h, g, d, window = s["attn"]
    for M, prompt in ((B, False), (T, True)):
        parts = 1 if prompt else fo.query("b200f_gemm_splits", M, (h + 2 * g) * d, W, 1, 1)
        y, qw, kw = f32(parts, M, (h + 2 * g) * d), f32(h * d), f32(g * d)
        q = torch.empty(M, h, d, dtype=bf, device="cuda")
        kc, vc = rnd(max(pages, M // 16 + 1), 16, g * d), rnd(max(pages, M // 16 + 1), 16, g * d)
        ll = torch.arange(M, dtype=torch.int32, device="cuda")
        ms = device_ms(lambda: fo.grouped_prepare(y, (0, h * d, (h + g) * d), qw, kw, 1e-6, ll, q, kc, vc, h, g, d, d))
        entry(f"grouped prepare M={M}", ms, M * (h + 2 * g) * d * (4.0 * parts + 2.0), like=like["prepare", M])
        q.normal_()
        o = fo.rows(M, h * d, bf, "cuda")
        if prompt:
            ms = device_ms(lambda: fo.grouped_attention(q, kc, vc, tb, plens, start, o, g, d, d, window, 0.1, n, n), calls=4)
            entry("grouped attention, prompts", ms, 2.0 * T * d * (2 * h + 2 * g), 4.0 * pairs(window) * h * d, like=like["attn", T])
        else:
            ms = device_ms(lambda: fo.grouped_attention(q, kc, vc, table, lens, None, o, g, d, d, window, 0.1, 1, ctx))
            seen = min(ctx, window)
            entry("grouped attention, decode", ms, 4.0 * B * seen * g * d + 4.0 * B * h * d, 4.0 * B * seen * h * d, like=like["attn", B])
        del y, q, kc, vc, o
        torch.cuda.empty_cache()

    # ends of the two-sided layer, gated feed-forward beside the xIELU one of equal width
    from mini_sgl_integer_b200.layers.float_linear import GatedSiluMLP, XieluMLP
    for M in (B, T):
        y, y2, x, xt = f32(1, M, W), f32(1, M, W), f32(M, W), fo.rows(M, W, bf, "cuda")
        w = [f32(W) for _ in range(4)]
        ms = device_ms(lambda: fo.sublayer_end(y, x, w[0], 1e-6, x, xt, bf, mean_with=(w[1], y2, w[2]), final_w=w[3]))
        entry(f"sublayer end of two mixers M={M}", ms, 18.0 * M * W, like=like["rows", M])
        ff = s["ff"]
        gm, xm = GatedSiluMLP(W, ff, bf, "cuda"), XieluMLP(W, ff, bf, "cuda")
        gm.load_state_dict({"gate": rnd(ff, W), "up": rnd(ff, W), "down": rnd(W, ff)})
        xm.load_state_dict({"up": rnd(ff, W), "down": rnd(W, ff), "act": torch.zeros(2, dtype=bf)})
        hx = rnd(M, W) * 0.1
        lms = device_ms(lambda: xm.forward(hx))
        l = {"name": "xIELU feed-forward", "us": lms * 1e3, "frac": frac(lms, 4.0 * ff * W + 2.0 * M * W + 4.0 * M * W, 4.0 * M * ff * W)}
        entry(f"gated feed-forward M={M}", device_ms(lambda: gm.forward(hx)), 6.0 * ff * W + 2.0 * M * W + 4.0 * M * W, 6.0 * M * ff * W, like=l)
        del y, y2, x, xt, gm, xm, hx
        torch.cuda.empty_cache()
    return out


def engine_e2e(s: dict, B: int, n: int, steps: int) -> dict:
    """Decode through Engine.step: host ids in, arg-max ids out, every step."""
    from mini_sgl_integer_b200.engine import Engine
    from mini_sgl_integer_b200.engine.sample import greedy
    from mini_sgl_integer_b200.models.config import DerelornConfig
    from mini_sgl_integer_b200.models.derelorn import random_weights
    d = derelorn_config(s)
    e = Engine(config=d, weights=random_weights(DerelornConfig.from_dict(d), 3, device="cuda"), max_tokens=B * (n + steps + 32), max_reqs=B,
               max_len=n + steps + 32, max_portion=8192)
    rng = np.random.default_rng(0)
    reqs = [e.open() for _ in range(B)]
    t0 = time.perf_counter()
    per = max(1, 8192 // n)
    for i in range(0, B, per):
        greedy(e.step(reqs[i:i + per], [rng.integers(0, s["vocab"], n).tolist() for _ in reqs[i:i + per]]))
    torch.cuda.synchronize()
    pre = time.perf_counter() - t0
    cur = rng.integers(0, s["vocab"], B).tolist()
    for _ in range(3):
        cur = greedy(e.step(reqs, [[t] for t in cur])).tolist()
    t0 = time.perf_counter()
    for _ in range(steps):
        cur = greedy(e.step(reqs, [[t] for t in cur])).tolist()
    dec = (time.perf_counter() - t0) / steps
    e.check_status()
    return {"decode_tok_s": B / dec, "decode_ms_per_step": dec * 1e3, "prefill_tok_s": B * n / pre, "h2d_bytes_per_step": B * 4 * 6 + 4, "d2h_bytes_per_step": 4 * B}


def run(args) -> None:
    from bench import ClockSampler
    torch.cuda.set_device(0)
    sampler = ClockSampler(0)
    t0 = time.perf_counter()
    B, prompts, n = min(args.batch, 256), 8, 1024
    names = args.sizes.split(",") if args.sizes else list(SIZES)
    res, launches = {}, 0
    for name in names:
        s, steps = SIZES[name], args.steps
        lens = np.random.default_rng(21).integers(100, 2049, B).astype(np.int32)
        max_len = -(-(2048 + 4 * steps + 64) // 16) * 16
        table, pages = contiguous_tables(B, max_len)
        cfg, model, cache, params = build(s, pages, B)
        rec = {"shape": s, "params": params, "decode": decode(s, cfg, model, cache, table, lens, max_len, steps, args.warmup, params)}
        launches += rec["decode"]["launches"] * steps
        rec["prefill"] = bh.sefevik_prefill(cfg, model, cache, table, prompts, n, max(3, steps // 4), params)
        del model, cache
        torch.cuda.empty_cache()
        c = closest_shape(s, params)
        ccfg, cmodel, ccache, cparams = bh.build_sefevik(c, max_len, pages, B)
        rec["closest"] = {"shape": c, "params": cparams, "decode": bh.sefevik_decode(c, ccfg, cmodel, ccache, table, lens, max_len, steps, args.warmup),
                          "prefill": bh.sefevik_prefill(ccfg, cmodel, ccache, table, prompts, n, max(3, steps // 4), cparams)}
        del cmodel, ccache
        torch.cuda.empty_cache()
        if not args.no_kernels:
            rec["kernels"] = kernel_table(s, c, B, prompts, n, 1100)
        torch.cuda.empty_cache()
        res[name] = rec
    e2e_name = names[min(1, len(names) - 1)]
    e2e = engine_e2e(SIZES[e2e_name], B, 512, args.steps)
    clocks = sampler.stop(t0, time.perf_counter())
    main = res[e2e_name]
    print(json.dumps({
        "metric": f"decode tokens/s, Derelorn {e2e_name}, bf16 (random weights)", "value": main["decode"]["tok_s"], "unit": "tokens/s", "n_gpus": 1,
        "steps": args.steps, "warmup": args.warmup, "ms_per_step": main["decode"]["ms"], "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic (seeded random weights and ids)",
        "config": {"workload": f"Derelorn at {', '.join(names)} parameters: decode batch {B}, contexts U[100,2048]; prefill {prompts} x {n} tokens",
                   "global_batch": B, "parallelism": "none", "l2": "weights, caches and states of a step exceed L2 (0.3B: 0.6 GB); kernels stream more than L2 or rotate over copies"},
        "e2e": {"value": e2e["decode_tok_s"], "unit": "tokens/s", "h2d_bytes_per_step": e2e["h2d_bytes_per_step"], "d2h_bytes_per_step": e2e["d2h_bytes_per_step"], **e2e},
        "gpu_launches": launches, "peaks": peaks(), "sizes": res, "clocks": clocks}))
