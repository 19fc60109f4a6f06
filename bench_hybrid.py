"""`bench.py --workload sefevik`: prefill and decode throughput of the Sefevik design at sizes that resemble a real model's
layers (random weights), beside the integer Qwen3-shaped model of equal width, depth and about equal parameter count, and
each kernel's time against its roofline beside the like kernel of that model.

Decode: one captured step (device-side bookkeeping, embedding, layers, head, arg-max, the token fed back) of `batch`
sequences.  Prefill: `prompts` prompts of `prompt_len` tokens in one forward, logits of the last tokens, arg-max.  The
end-to-end figure goes through Engine.step: host token ids in, logits' arg-max back, every step.
"""
from __future__ import annotations

import json
import os
import time

import numpy as np
import torch

ROOT = os.path.dirname(os.path.abspath(__file__))

# (gru, gru, attention, gru, gru, attention with kv_from) repeated
SIZES = {
    "0.3B": dict(width=1024, depth=12, gru=1536, ff=4096, heads=16, dim=64, rot=32, vdim=64, rank=256, window=512, vocab=32768),
    "1.4B": dict(width=2048, depth=24, gru=3072, ff=8192, heads=16, dim=128, rot=64, vdim=128, rank=512, window=1024, vocab=32768),
    "4B": dict(width=4096, depth=18, gru=6144, ff=16384, heads=32, dim=128, rot=64, vdim=128, rank=512, window=1024, vocab=65536),
}
YARN = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}


def sefevik_config(s: dict) -> dict:
    layers = []
    for i in range(s["depth"]):
        mlp = {"kind": "dense", "ff": s["ff"]}
        if i % 3 != 2:
            layers.append({"type": "mingru", "mixer": {"width": s["gru"]}, "mlp": mlp})
            continue
        m = {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot"], "vdim": s["vdim"], "kv_rank": s["rank"],
             "scale": (s["dim"] + s["rot"]) ** -0.5, "mask": {"size": s["window"]},
             "rot": {"dims": s["rot"], "base": 1e6, "scaling": YARN}}
        if i % 6 == 5:
            m["kv_from"] = i - 3
        layers.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
    return {"architecture": "Sefevik", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "layers": layers,
            "embedding": {"bigram": {"buckets": 65521, "mul_prev": 1_000_003, "mul_cur": 8191}}}


def peaks() -> dict:
    p = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        p = {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
    except Exception:
        pass
    p["int8_tops"] = 4500.0          # nominal: no measured int8 figure exists
    return p


def timed(fn, reps: int, warmup: int = 3) -> float:
    """Mean milliseconds of `fn` over `reps` back-to-back calls."""
    for _ in range(max(3, warmup)):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(reps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / reps


def captured(step, warm: int = 2):
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for _ in range(warm):
            step()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        step()
    return g


def contiguous_tables(batch: int, max_len: int):
    pitch = -(-max_len // 16)
    perm = np.random.default_rng(1).permutation(batch * pitch).astype(np.int32).reshape(batch, pitch)
    return torch.from_numpy(perm).cuda(), batch * pitch


def prompt_meta(prompts: int, n: int, table):
    pos = np.tile(np.arange(n, dtype=np.int32), prompts)
    seq = np.repeat(np.arange(prompts, dtype=np.int32), n)
    t = table.cpu().numpy()
    loc = (t[seq, pos // 16] * 16 + pos % 16).astype(np.int32)
    d = lambda a: torch.from_numpy(np.ascontiguousarray(a)).cuda()
    return d(pos), d(loc), d(seq), d((np.arange(prompts + 1) * n).astype(np.int32)), d(np.full(prompts, n, dtype=np.int32))


# ----------------------------------------------------------------------------- the design
def build_sefevik(s: dict, max_len: int, pages: int, batch: int):
    from mini_sgl_integer_b200.kvcache.hybrid_pool import HybridCache
    from mini_sgl_integer_b200.models.config import SefevikConfig
    from mini_sgl_integer_b200.models.sefevik import SefevikForCausalLM, random_weights
    cfg = SefevikConfig.from_dict(sefevik_config(s))
    sd = random_weights(cfg, 3, device="cuda")
    params = sum(v.numel() for k, v in sd.items() if k not in ("embed", "bigram"))
    model = SefevikForCausalLM(cfg, torch.bfloat16, "cuda", max_position=max_len)
    model.load_state_dict(sd)
    cache = HybridCache(cfg, pages, batch, torch.bfloat16, "cuda")
    for i in cfg.cache_layers:
        cache.k_cache(i).normal_()
    for i in cfg.recurrent_layers:
        cache.state(i).normal_()
    return cfg, model, cache, params


def sefevik_decode(s: dict, cfg, model, cache, table, lens, max_len: int, steps: int, warmup: int) -> dict:
    from mini_sgl_integer_b200 import _lib
    from mini_sgl_integer_b200.attention.hybrid_backend import HybridMetadata
    from mini_sgl_integer_b200.kernel.float_ops import argmax_f32
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
    weights = sum(l.numel() for l in _weights(model)) * 2
    kv = sum(float(np.minimum(lens, m.window).sum()) * (m.kv_rank + m.rot_dim) * 2 for m in (cfg.layers[i].mixer for i in cfg.attention_layers))
    st = len(cfg.recurrent_layers) * B * s["gru"] * 8.0
    gbs = (weights + kv + st) / ms / 1e6
    return {"ms": ms, "tok_s": B / ms * 1e3, "weight_bytes": weights, "kv_bytes": kv, "state_bytes": st, "GBs": gbs, "frac": gbs / peaks()["hbm_gbs"],
            "launches": calls}


def _weights(model):
    for l in model.layers.op_list:
        m = l.mix
        yield from (x.weight for x in ((m.zug, m.o) if hasattr(m, "zug") else (m.qd, m.o)))
        if hasattr(m, "uk"):
            yield m.uk
            yield m.uv
        if l.mlp is not None:
            yield l.mlp.up.weight
            yield l.mlp.down.weight
    yield model.head.weight


def sefevik_prefill(cfg, model, cache, table, prompts: int, n: int, steps: int, params: int) -> dict:
    from mini_sgl_integer_b200.attention.hybrid_backend import HybridMetadata
    from mini_sgl_integer_b200.kernel.float_ops import argmax_f32
    pos, loc, seq, start, lens = prompt_meta(prompts, n, table)
    md = HybridMetadata(pos, loc, table[:prompts].contiguous(), lens, torch.arange(prompts, dtype=torch.int32, device="cuda"), start, seq, n, n)
    ids = torch.randint(0, cfg.vocab_size, (prompts * n,), dtype=torch.int32, device="cuda")
    last = (start[1:] - 1).to(torch.int64)
    ms = timed(lambda: argmax_f32(model.forward_tokens(ids, md, cache, last)), steps)
    model.check_status()
    flops = 2.0 * (params - cfg.vocab_size * cfg.hidden_size) * prompts * n
    return {"ms": ms, "tok_s": prompts * n / ms * 1e3, "linear_TFLOPs": flops / ms / 1e9, "frac": flops / ms / 1e9 / peaks()["bf16_tflops"]}


# ----------------------------------------------------------------------------- the closest existing model
def qwen_shape(s: dict, params: int) -> dict:
    heads, kv = s["width"] // 128, max(1, s["width"] // 512)
    attn = (2 * heads + 2 * kv) * 128 * s["width"]
    per = (params - s["vocab"] * s["width"]) / s["depth"]
    inter = max(128, int(round((per - attn) / (3 * s["width"]) / 128)) * 128)
    return dict(width=s["width"], depth=s["depth"], heads=heads, kv=kv, inter=inter, vocab=s["vocab"])


def qwen_run(q: dict, table, pages: int, lens, max_len: int, prompts: int, n: int, steps: int, warmup: int) -> dict:
    from mini_sgl_integer_b200.attention import Int8PagedKVCache
    from mini_sgl_integer_b200.layers.decoder_layer import AttnBatch
    from mini_sgl_integer_b200.models import DecodeBatch, Qwen3ForCausalLMInteger, Qwen3IntegerConfig, check_device_status, random_weights
    from bench import fill_pool_random
    cfg = Qwen3IntegerConfig(q["depth"], q["width"], q["heads"], q["kv"], q["inter"], q["vocab"], max_pos=max_len)
    w = random_weights(cfg, seed=4, device="cuda", generate_on_device=True)
    pool = Int8PagedKVCache(q["kv"], q["depth"], 128, pages, "cuda")
    fill_pool_random(pool, q["depth"], torch.Generator(device="cuda").manual_seed(5), v_shift=(36, 40))
    lm = Qwen3ForCausalLMInteger(cfg, w, pool)
    pos, loc, _, start, plens = prompt_meta(prompts, n, table)
    ab = AttnBatch(pos, loc, table[:prompts].contiguous(), plens, plens, max_len)
    ids = torch.randint(0, q["vocab"], (prompts * n,), dtype=torch.int32, device="cuda")
    pre = timed(lambda: lm.greedy(ids, ab, start[1:] - 1), max(3, steps // 4))
    state = DecodeBatch(table, torch.from_numpy(lens).cuda(), max_len, first_wave_rows=max(1, 296 // q["kv"]))
    cur = torch.zeros(len(lens), dtype=torch.int32, device="cuda")

    def step():
        cur.copy_(lm.greedy(cur, state.advance()))
    dec = timed(captured(step, 1).replay, steps, warmup)
    check_device_status()
    per = (2 * q["heads"] + 2 * q["kv"]) * 128 * q["width"] + 3 * q["inter"] * q["width"]
    weights = q["depth"] * per + q["vocab"] * q["width"]
    kv = float(lens.sum()) * q["kv"] * 266 * q["depth"]
    pk = peaks()
    flops = 2.0 * q["depth"] * per * prompts * n
    return {"shape": q, "params": weights,
            "decode": {"ms": dec, "tok_s": len(lens) / dec * 1e3, "weight_bytes": weights, "kv_bytes": kv, "GBs": (weights + kv) / dec / 1e6,
                       "frac": (weights + kv) / dec / 1e6 / pk["hbm_gbs"]},
            "prefill": {"ms": pre, "tok_s": prompts * n / pre * 1e3, "linear_TOPs": flops / pre / 1e9, "frac": flops / pre / 1e9 / pk["int8_tops"]}}


# ----------------------------------------------------------------------------- kernels one by one
def kernel_table(s: dict, q: dict, B: int, prompts: int, n: int, ctx: int) -> dict:
    """name -> {ms, frac of the roofline, like: {name, ms, frac}}.  Inputs rotate over copies that exceed L2 together."""
    from mini_sgl_integer_b200.kernel import float_ops as fo
    pk, out = peaks(), {}
    bf = torch.bfloat16
    T = prompts * n
    rnd = lambda *sh: torch.randn(sh, device="cuda").to(bf)

    def entry(name, ms, bytes_=None, flops=None, like=None):
        best = max((bytes_ or 0) / pk["hbm_gbs"] / 1e6, (flops or 0) / pk["bf16_tflops"] / 1e9)
        out[name] = {"us": ms * 1e3, "bound": "hbm" if (bytes_ or 0) / pk["hbm_gbs"] / 1e6 >= best else "tensor", "frac": best / ms}
        if like:
            lname, lms, lbytes, lflops = like
            lbest = max((lbytes or 0) / pk["hbm_gbs"] / 1e6, (lflops or 0) / pk["int8_tops"] / 1e9)
            out[name]["like"] = {"name": lname, "us": lms * 1e3, "frac": lbest / lms}

    def device_ms(fn, calls=16, reps=5):
        """Per call, from a captured graph of `calls` calls: small kernels would otherwise be timed at the host's launch rate."""
        def many():
            for _ in range(calls):
                fn()
        return timed(captured(many, 1).replay, reps) / calls

    def rotating(make, fn, bytes_each):
        copies = [make() for _ in range(max(1, min(16, int(3e8 // max(bytes_each, 1)) + 1)))]
        k = [0]

        def run():
            k[0] = (k[0] + 1) % len(copies)
            fn(copies[k[0]])
        return device_ms(run)

    # linears, and the int8 linear of the same (M, N, K)
    from mini_sgl_integer_b200.layers.w8a8_int8 import int8_gemm_q15
    W = s["width"]
    shapes = {"zug": (3 * s["gru"], W), "mingru o": (W, s["gru"]), "up": (s["ff"], W), "down": (W, s["ff"]),
              "qd": (s["heads"] * (s["dim"] + s["rot"]) + s["rank"] + s["rot"], W), "head": (s["vocab"], W)}
    for M in (B, T):
        for name, (N, K) in shapes.items():
            if name == "head" and M == T:
                continue
            x = rnd(M, K)
            ms = rotating(lambda: rnd(N, K), lambda w: fo.linear_parts(x, w), 2 * N * K)
            x8 = torch.randint(-127, 128, (M, K), dtype=torch.int8, device="cuda")
            am = torch.randint(1, 2 ** 22, (M,), dtype=torch.int32, device="cuda")
            mul = torch.randint(2 ** 29, 2 ** 30, (N,), dtype=torch.int32, device="cuda")
            k8 = K - K % 16
            lms = rotating(lambda: torch.randint(-127, 128, (N, k8), dtype=torch.int8, device="cuda"),
                           lambda w: int8_gemm_q15(x8[:, :k8].contiguous() if k8 != K else x8, None, None, w, mul, None, x_absmax=am), N * K)
            entry(f"linear {name} M={M}", ms, 2 * N * K + 2 * M * K + 4 * M * N, 2.0 * M * N * K,
                  ("gemm_w8a8 of the same shape", lms, N * K + M * K + 4 * M * N, 2.0 * M * N * K))
            del x, x8
    for M in (B, T):
        H, r, d = s["heads"], s["rank"], s["dim"]
        x, o = rnd(M, H, d), torch.empty(M, H, fo.pad8(r + s["rot"]), dtype=bf, device="cuda")
        ms = rotating(lambda: rnd(H, r, d), lambda w: fo.head_linear(x, w, o[..., :r]), 2 * H * r * d)
        entry(f"head linear uk M={M}", ms, 2 * H * r * d + 2 * M * H * (d + r), 2.0 * M * H * r * d)
        x2, o2 = rnd(M, H, r), torch.empty(M, H, s["vdim"], dtype=bf, device="cuda")
        ms = rotating(lambda: rnd(H, s["vdim"], r), lambda w: fo.head_linear(x2, w, o2), 2 * H * r * d)
        entry(f"head linear uv M={M}", ms, 2 * H * r * d + 2 * M * H * (d + r), 2.0 * M * H * r * s["vdim"])
        del x, o, x2, o2

    # attention
    from mini_sgl_integer_b200.attention import Int8PagedKVCache, decode_attention_int8_paged, prefill_attention_int8_paged
    from bench import fill_pool_random
    H, lat = s["heads"], s["rank"] + s["rot"]
    max_len = -(-ctx // 16) * 16
    table, pages = contiguous_tables(B, max_len)
    lens = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    sink = torch.zeros(H, device="cuda")
    ql, o = rnd(B, H, lat), torch.empty(B, H, s["rank"], dtype=bf, device="cuda")
    seen = min(ctx, s["window"])
    ms = rotating(lambda: rnd(pages, 16, lat), lambda c: fo.latent_attention(ql, c, table, lens, None, sink, o, s["rank"], s["rot"], s["window"], 0.1, 1, ctx),
                  2 * B * seen * lat)
    pool = Int8PagedKVCache(q["kv"], 4, 128, pages, "cuda")
    fill_pool_random(pool, 4, torch.Generator(device="cuda").manual_seed(5), v_shift=(36, 40))
    q8 = torch.randint(-127, 128, (B, q["heads"], 128), dtype=torch.int8, device="cuda")
    qm = torch.randint(2 ** 30, 2 ** 31, (B, q["heads"]), dtype=torch.int64, device="cuda").to(torch.int32)
    qs = torch.full((B, q["heads"]), 44, dtype=torch.int32, device="cuda")
    rot = [0]

    def like_decode():
        rot[0] = (rot[0] + 1) % 4
        decode_attention_int8_paged(q8, qm, qs, pool, rot[0], table, lens, max_len)
    lms = device_ms(like_decode)
    entry("latent attention, decode", ms, 2.0 * B * seen * lat + 2.0 * B * H * (lat + s["rank"]), 2.0 * B * seen * H * (lat + s["rank"]),
          ("attn_decode (int8)", lms, float(B * ctx * q["kv"] * 266), 4.0 * B * ctx * q["heads"] * 128))
    pos, loc, seq, start, plens = prompt_meta(prompts, n, table)
    ql2, o2 = rnd(T, H, lat), torch.empty(T, H, s["rank"], dtype=bf, device="cuda")
    c = rnd(pages, 16, lat)
    tb = table[:prompts].contiguous()
    ms = device_ms(lambda: fo.latent_attention(ql2, c, tb, plens, start, sink, o2, s["rank"], s["rot"], s["window"], 0.1, n, n))
    w = min(n, s["window"])
    pairs = prompts * (w * (w + 1) / 2 + (n - w) * w)
    q8p = torch.randint(-127, 128, (T, q["heads"], 128), dtype=torch.int8, device="cuda")
    qmp = torch.randint(2 ** 30, 2 ** 31, (T, q["heads"]), dtype=torch.int64, device="cuda").to(torch.int32)
    qsp = torch.full((T, q["heads"]), 44, dtype=torch.int32, device="cuda")
    lms = device_ms(lambda: prefill_attention_int8_paged(q8p, qmp, qsp, pool, 0, tb, plens, plens, n, n))
    entry("latent attention, prompts", ms, 2.0 * T * lat + 2.0 * T * H * (lat + s["rank"]), 2.0 * pairs * H * (lat + s["rank"]),
          ("attn_prefill (int8)", lms, None, 4.0 * prompts * n * (n + 1) / 2 * q["heads"] * 128))
    del pool, q8p, qmp, qsp, ql2, o2, c
    torch.cuda.empty_cache()

    # row kernels
    from mini_sgl_integer_b200.kernel import fixed_point as fp
    for M in (B, T):
        y, x, nw = torch.randn(1, M, W, device="cuda"), torch.randn(M, W, device="cuda"), torch.randn(W, device="cuda")
        xo, xt = torch.empty_like(x), fo.rows(M, W, bf, "cuda")
        planes = s["depth"] // 2
        xi, ri, wi = (torch.randint(-2 ** 18, 2 ** 18, sh, dtype=torch.int32, device="cuda") for sh in ((M, W), (M, W), (W,)))
        lms = device_ms(lambda: fp.fused_add_rmsnorm_quant(xi, ri, wi))
        like = ("add + RMSNorm + quant rows (int)", lms, 13.0 * M * W, None)
        entry(f"sublayer end M={M}", device_ms(lambda: fo.sublayer_end(y, x, nw, 1e-6, xo, xt, bf)), 14.0 * M * W, None, like)
        h, coef = torch.randn(planes + 1, M, W, device="cuda"), torch.randn(planes + 1, device="cuda")
        entry(f"sublayer end + depth average over {planes + 1} M={M}",
              device_ms(lambda: fo.sublayer_end(y, x, nw, 1e-6, xo, xt, bf, hist=h, planes=planes, coef=coef, hist_out=h[planes])),
              (18.0 + 4.0 * planes) * M * W, None, like)
        del h, y, x, xo, xt, xi, ri
        gru = s["gru"]
        zug, bz = torch.randn(1, M, 3 * gru, device="cuda"), torch.randn(gru, device="cuda")
        state, yo = torch.zeros(max(B, prompts), gru, device="cuda"), fo.rows(M, gru, bf, "cuda")
        gu = torch.randint(-2 ** 18, 2 ** 18, (M, 2 * (gru - gru % 128)), dtype=torch.int32, device="cuda")
        lms = device_ms(lambda: fp.silu_mul_fwht_quant(gu, 128))
        like = ("SiLU * up + rotation + quant rows (int)", lms, 9.0 * M * (gru - gru % 128), None)
        if M == B:
            sl, p1 = torch.arange(B, dtype=torch.int32, device="cuda"), torch.ones(B, dtype=torch.int32, device="cuda")
            entry(f"minGRU step M={M}", device_ms(lambda: fo.mingru(zug, bz, bz, state, sl, p1, None, B, yo)), 22.0 * M * gru, None, like)
        else:
            sl = torch.arange(prompts, dtype=torch.int32, device="cuda")
            entry(f"minGRU scan M={M}", device_ms(lambda: fo.mingru(zug, bz, bz, state, sl, pos, start, prompts, yo)), 14.0 * M * gru, None, like)
        del zug, gu, yo
        nq = H * (s["dim"] + s["rot"]) + lat
        qd, cache = torch.randn(1, M, nq, device="cuda"), torch.zeros(pages, 16, lat, dtype=bf, device="cuda")
        rope = torch.randn(max(n, 2), s["rot"], device="cuda")
        qn, qq = torch.empty(M, H, s["dim"], dtype=bf, device="cuda"), torch.empty(M, H, lat, dtype=bf, device="cuda")
        pp = torch.zeros(M, dtype=torch.int32, device="cuda")
        ll = torch.arange(M, dtype=torch.int32, device="cuda")
        from mini_sgl_integer_b200.attention import qkv_rope_quant_store
        from mini_sgl_integer_b200.models import rope_cache_q15
        pool = Int8PagedKVCache(q["kv"], 1, 128, M // 16 + 1, "cuda")
        qkv = torch.randint(-2 ** 18, 2 ** 18, (M, (q["heads"] + 2 * q["kv"]) * 128), dtype=torch.int32, device="cuda")
        cs = rope_cache_q15(16).cuda()
        nwq = torch.randint(2 ** 11, 2 ** 13, (128,), dtype=torch.int32, device="cuda")
        lms = device_ms(lambda: qkv_rope_quant_store(pp, qkv, q["heads"], pool, 0, ll, cs, nwq, nwq))
        lb = M * ((q["heads"] + 2 * q["kv"]) * 512.0 + q["heads"] * 136.0 + q["kv"] * 266.0)
        dn = torch.ones(s["rank"], device="cuda")
        ms = device_ms(lambda: fo.latent_prepare(qd, pp, ll, rope, dn, 1e-6, qn, qq, cache, H, s["dim"], s["rot"], s["rank"]))
        entry(f"latent prepare M={M}", ms, M * (4.0 * nq + 2.0 * H * (s["dim"] + s["rot"]) + 2.0 * lat), None, ("qkv_prepare rows (int)", lms, lb, None))
        del qd, cache, qn, qq, pool, qkv
        torch.cuda.empty_cache()
    return out


def engine_e2e(s: dict, B: int, n: int, steps: int) -> dict:
    """Decode through Engine.step: host ids in, arg-max ids out, every step."""
    from mini_sgl_integer_b200.engine import Engine
    from mini_sgl_integer_b200.engine.sample import greedy
    from mini_sgl_integer_b200.models.config import SefevikConfig
    from mini_sgl_integer_b200.models.sefevik import random_weights
    d = sefevik_config(s)
    e = Engine(config=d, weights=random_weights(SefevikConfig.from_dict(d), 3, device="cuda"), max_tokens=B * (n + steps + 32), max_reqs=B,
               max_len=n + steps + 32, max_portion=8192)
    rng = np.random.default_rng(0)
    reqs = [e.open() for _ in range(B)]
    t0 = time.perf_counter()
    per = max(1, 8192 // n)
    for i in range(0, B, per):
        ids = greedy(e.step(reqs[i:i + per], [rng.integers(0, s["vocab"], n).tolist() for _ in reqs[i:i + per]]))
    torch.cuda.synchronize()
    pre = time.perf_counter() - t0
    cur = rng.integers(0, s["vocab"], B).tolist()
    for _ in range(3):
        cur = greedy(e.step(reqs, [[c] for c in cur])).tolist()
    t0 = time.perf_counter()
    for _ in range(steps):
        cur = greedy(e.step(reqs, [[c] for c in cur])).tolist()
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
        s = SIZES[name]
        steps = args.steps
        lens = np.random.default_rng(21).integers(100, 2049, B).astype(np.int32)
        max_len = -(-(2048 + 4 * steps + 64) // 16) * 16
        table, pages = contiguous_tables(B, max_len)
        cfg, model, cache, params = build_sefevik(s, max_len, pages, B)
        rec = {"shape": s, "params": params, "decode": sefevik_decode(s, cfg, model, cache, table, lens, max_len, steps, args.warmup)}
        launches += rec["decode"]["launches"] * steps
        rec["prefill"] = sefevik_prefill(cfg, model, cache, table, prompts, n, max(3, steps // 4), params)
        del model, cache
        torch.cuda.empty_cache()
        rec["closest"] = qwen_run(qwen_shape(s, params), table, pages, lens, max_len, prompts, n, steps, args.warmup)
        torch.cuda.empty_cache()
        if not args.no_kernels:
            rec["kernels"] = kernel_table(s, rec["closest"]["shape"], B, prompts, n, 1100)
        torch.cuda.empty_cache()
        res[name] = rec
    e2e_name = names[min(1, len(names) - 1)]
    e2e = engine_e2e(SIZES[e2e_name], B, 512, args.steps)
    clocks = sampler.stop(t0, time.perf_counter())
    main = res[e2e_name]
    print(json.dumps({
        "metric": f"decode tokens/s, Sefevik {e2e_name}, bf16 (random weights)", "value": main["decode"]["tok_s"], "unit": "tokens/s", "n_gpus": 1,
        "steps": args.steps, "warmup": args.warmup, "ms_per_step": main["decode"]["ms"], "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic (seeded random weights and ids)",
        "config": {"workload": f"Sefevik at {', '.join(names)} parameters: decode batch {B}, contexts U[100,2048]; prefill {prompts} x {n} tokens",
                   "global_batch": B, "parallelism": "none", "l2": "weights + cache per step exceed L2 (0.3B: 0.5 GB); kernel inputs rotate over copies larger than L2 where they are smaller"},
        "e2e": {"value": e2e["decode_tok_s"], "unit": "tokens/s", "h2d_bytes_per_step": e2e["h2d_bytes_per_step"], "d2h_bytes_per_step": e2e["d2h_bytes_per_step"], **e2e},
        "gpu_launches": launches, "peaks": peaks(), "sizes": res, "clocks": clocks}))
