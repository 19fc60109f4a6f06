"""The floating-point kernels one by one against plain references: the numpy functions of oracle/sefevik.py, or a float64
matrix product.  bf16 cases feed the reference the rounded operands, so only accumulation order and the final rounding
differ."""
from __future__ import annotations

import numpy as np
import pytest
import torch

from mini_sgl_integer_b200.kernel import float_ops as fo
from mini_sgl_integer_b200.layers.float_linear import padded_rows
from oracle import sefevik as S

pytestmark = pytest.mark.gpu
DT = [torch.float32, torch.bfloat16]


def dev(a, dtype=torch.float32):
    return torch.as_tensor(np.ascontiguousarray(a)).to(dtype).cuda()


def i32(a):
    return torch.as_tensor(np.asarray(a, dtype=np.int32)).cuda()


def host(t):
    return t.detach().double().cpu().numpy()


def close(got, want, dtype, f32_tol=2e-5, bf_tol=8e-3):
    """Largest error relative to the reference's root mean square (bf16: half an ulp of the largest values allowed)."""
    got, want = host(got) if isinstance(got, torch.Tensor) else got, np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    scale = np.sqrt(np.mean(want ** 2)) + 1e-30
    err = np.abs(got - want) / (scale + np.abs(want))
    assert err.max() <= (f32_tol if dtype == torch.float32 else bf_tol), err.max()


def rows_of(g, n, k, dtype):
    return padded_rows(torch.randn(n, k, generator=g), dtype, "cuda")


# ----------------------------------------------------------------------------- linears
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("m,n,k", [(1, 40, 24), (3, 129, 200), (17, 384, 520), (33, 56, 64), (64, 1000, 72), (100, 300, 1032), (130, 260, 136),
                                   (256, 700, 2048), (257, 520, 320), (700, 333, 96), (1500, 2600, 130)])
def test_linear(dtype, m, n, k):
    g = torch.Generator().manual_seed(m + n)
    x, w = rows_of(g, m, k, dtype), rows_of(g, n, k, dtype)
    want = host(x) @ host(w).T
    close(fo.linear(x, w, out_f32=True), want, torch.float32)
    close(fo.linear(x, w), want, dtype)
    parts = fo.linear_parts(x, w)
    close(parts.sum(0), want, torch.float32)
    assert parts.shape[0] == 1 or (dtype == torch.bfloat16 and m <= 256)
    a, b = 0.7, 1.1
    z = want / np.sqrt(k)
    xs = padded_rows((x.float() / np.sqrt(k)).cpu(), dtype, "cuda")
    z = host(xs) @ host(w).T
    close(fo.linear(xs, w, act=fo.ACT_XIELU, act_a=a, act_b=b), np.where(z > 0, a * z * z + z / 2, b * (np.expm1(np.minimum(z, 0)) - np.minimum(z, 0)) + z / 2), dtype)
    fo.check_status()


def test_linear_splits_k_for_few_rows():
    g = torch.Generator().manual_seed(5)
    x, w = rows_of(g, 4, 4096, torch.bfloat16), rows_of(g, 256, 4096, torch.bfloat16)
    parts = fo.linear_parts(x, w)
    assert parts.shape[0] > 1
    close(parts.sum(0), host(x) @ host(w).T, torch.float32)
    assert torch.equal(parts, fo.linear_parts(x, w))           # no atomics: the same bits every time


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T,H,n,k", [(1, 3, 24, 40), (5, 7, 200, 24), (70, 2, 40, 136), (300, 5, 136, 72), (3, 4, 1, 9)])
def test_head_linear(dtype, T, H, n, k):
    g = torch.Generator().manual_seed(T)
    kp, npad = fo.pad8(k), fo.pad8(n) + 16
    x = torch.randn(T, H, kp, generator=g).to(dtype).cuda()[..., :k]
    w = padded_rows(torch.randn(H, n, k, generator=g), dtype, "cuda")
    out = torch.full((T, H, npad), 7.0, dtype=dtype, device="cuda")
    fo.head_linear(x, w, out[..., :n])
    close(out[..., :n], np.einsum("thk,hnk->thn", host(x), host(w)), dtype)
    assert bool((out[..., n:] == 7.0).all())                   # nothing outside the view is touched


# ----------------------------------------------------------------------------- embedding
@pytest.mark.parametrize("dtype", DT)
def test_embedding_with_bigram_rows_over_portions(dtype):
    rng = np.random.default_rng(3)
    V, W, buckets, mp, mc = 90, 52, 37, 1_000_003, 90_001
    w = {"embed": rng.standard_normal((V, W)), "bigram": rng.standard_normal((buckets + 1, W))}
    t, b = dev(w["embed"], dtype), dev(w["bigram"], dtype)
    cfg = {"embedding": {"bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}}
    seqs = [rng.integers(0, V, n) for n in (9, 1, 14)]
    want = [S.embed(s, cfg, {"embed": host(t), "bigram": host(b)}) for s in seqs]
    slots, prev = [4, 0, 2], torch.full((6,), 55, dtype=torch.int32, device="cuda")
    at = [0, 0, 0]

    def run(counts):
        who = [i for i, c in enumerate(counts) if c]
        ids = np.concatenate([seqs[i][at[i]:at[i] + counts[i]] for i in who])
        pos = np.concatenate([np.arange(at[i], at[i] + counts[i]) for i in who])
        start = np.concatenate([[0], np.cumsum([counts[i] for i in who])])
        seq = np.repeat(np.arange(len(who)), [counts[i] for i in who])
        out, out_t = torch.empty(len(ids), W, device="cuda"), fo.rows(len(ids), W, dtype, "cuda")
        decode = all(counts[i] == 1 for i in who)
        fo.embed_bigram(t, b, i32(ids), i32(pos), None if decode else i32(seq), None if decode else i32(start), i32([slots[i] for i in who]),
                        prev, buckets, mp, mc, out, out_t)
        ref = np.concatenate([want[i][at[i]:at[i] + counts[i]] for i in who])
        close(out, ref, torch.float32, 1e-6)
        close(out_t, ref, dtype)
        for i in who:
            at[i] += counts[i]
    run([4, 1, 6]); run([1, 0, 1]); run([3, 0, 5]); run([1, 0, 2])
    assert prev[4] == int(seqs[0][-1]) and prev[0] == int(seqs[1][-1]) and prev[1] == 55


def test_embedding_without_bigram_table():
    t = torch.randn(20, 24, device="cuda").to(torch.bfloat16)
    ids = i32([3, 19, 0])
    out = torch.empty(3, 24, device="cuda")
    fo.embed_bigram(t, None, ids, i32([0, 1, 2]), i32([0, 0, 0]), i32([0, 3]), i32([0]), torch.zeros(1, dtype=torch.int32, device="cuda"), 0, 0, 0, out, None)
    assert torch.equal(out, t[ids.long()].float())


# ----------------------------------------------------------------------------- row kernels
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("width", [24, 90, 257, 1024, 5000, 12288])
@pytest.mark.parametrize("parts", [1, 3])
def test_sublayer_end(dtype, width, parts):
    rng = np.random.default_rng(width)
    T, eps, L = 5, 1e-3, 6
    y, x, w, fw = rng.standard_normal((parts, T, width)) * 0.01, rng.standard_normal((T, width)), rng.standard_normal(width), rng.standard_normal(width)
    if width % 4 and parts > 1:
        pytest.skip("parts are as wide as the row: covered by the aligned widths")
    hist, coef = rng.standard_normal((L, T, width)), rng.standard_normal(L + 1)
    r = x + S.rms_norm(y.sum(0), w, eps)
    xo, xt = torch.empty(T, width, device="cuda"), fo.rows(T, width, dtype, "cuda")
    fo.sublayer_end(dev(y), dev(x), dev(w), eps, xo, xt, dtype)
    close(xo, r, torch.float32); close(xt, r, dtype)
    for planes in (0, 1, 4, 5):
        c = coef[:planes + 1]
        want = S.depth_average(list(hist[:planes]) + [r], c)
        h = dev(hist)
        fo.sublayer_end(dev(y), dev(x), dev(w), eps, xo, xt, dtype, hist=h, planes=planes, coef=dev(c), hist_out=h[planes])
        close(xo, want, torch.float32); close(xt, want, dtype); close(h[planes], r, torch.float32)
        fo.sublayer_end(dev(y), dev(x), dev(w), eps, None, xt, dtype, hist=h, planes=planes, coef=dev(c), final_w=dev(fw))
        close(xt, S.rms_norm(want, fw, eps), dtype)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("n", [40, 133, 2052])
def test_xielu(dtype, n):
    rng = np.random.default_rng(n)
    p, q = 0.3, -0.8
    y = rng.standard_normal((2, 4, n)) * np.array([1e-4, 1.0, 6.0, 30.0])[None, :, None]
    out = fo.rows(4, n, dtype, "cuda")
    fo.xielu(dev(y), out, float(S.softplus(p)), float(0.5 + S.softplus(q)))
    for r in range(4):                                          # row by row: tiny inputs have their own scale
        close(out[r], S.xielu(y.sum(0)[r], p, q), dtype)


def test_argmax_takes_the_lowest_index_on_ties():
    x = torch.randn(5, 1003, device="cuda")
    x[0, [7, 900]] = 50.0
    x[1] = -3.0
    x[2, 1002] = 60.0
    x[3, 4], x[3, 2] = 0.0, -0.0
    x[3][x[3] > 0] = -1.0
    x[4, 11] = float("nan")
    got = fo.argmax_f32(x).tolist()
    assert got[:4] == [7, 0, 1002, 2]
    assert got[4] == int(torch.nan_to_num(x[4], nan=-1e9).argmax())


# ----------------------------------------------------------------------------- recurrence
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("width", [40, 161, 512])
def test_mingru_prompts_portions_and_steps(dtype, width):
    rng = np.random.default_rng(width)
    lens, slots = [300, 1, 129, 17], [5, 2, 0, 3]
    bz, bu = rng.standard_normal(width) - 3.0, rng.standard_normal(width)     # small z: the state remembers far back
    pre = [rng.standard_normal((n, 3 * width)) for n in lens]
    states = [S.mingru_scan(p[:, :width] + bz, p[:, width:2 * width] + bu) for p in pre]
    want = [s * S.silu(p[:, 2 * width:]) for s, p in zip(states, pre)]
    state = torch.full((7, width), 123.0, device="cuda")                       # left by an earlier request
    at = [0] * len(lens)

    def run(counts, parts=1):
        who = [i for i, c in enumerate(counts) if c]
        x = np.concatenate([pre[i][at[i]:at[i] + counts[i]] for i in who])
        T = len(x)
        zug = np.zeros((parts, T, 3 * width))
        zug[:] = x / parts
        start = np.concatenate([[0], np.cumsum([counts[i] for i in who])])
        pos = np.concatenate([np.arange(at[i], at[i] + counts[i]) for i in who])
        out = fo.rows(T, width, dtype, "cuda")
        decode = all(counts[i] == 1 for i in who)
        fo.mingru(dev(zug), dev(bz), dev(bu), state, i32([slots[i] for i in who]), i32(pos), None if decode else i32(start), len(who), out)
        close(out, np.concatenate([want[i][at[i]:at[i] + counts[i]] for i in who]), dtype)
        for i in who:
            at[i] += counts[i]
            close(state[slots[i]], states[i][at[i] - 1], torch.float32)
    run([150, 1, 128, 2]); run([2, 0, 1, 8], parts=3); run([1, 0, 0, 1], parts=2); run([127, 0, 0, 6])
    assert bool((state[[1, 4, 6]] == 123.0).all())


# ----------------------------------------------------------------------------- latent attention
ROT = {"dims": 12, "base": 5000.0, "scaling": {"factor": 3.0, "original": 96, "fast": 8.0, "slow": 1.0}}


def test_rotary_table_against_the_oracle():
    from mini_sgl_integer_b200.layers.rotary_float import rotary_frequencies, rotary_table
    from mini_sgl_integer_b200.models.config import RotarySpec, YarnScaling
    for dims, base, sc in [(12, 5000.0, ROT["scaling"]), (64, 1e6, {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                           (2, 100.0, {"factor": 2.0, "original": 8, "fast": 4.0, "slow": 2.0}), (8, 10000.0, None)]:
        spec = RotarySpec(dims, base, None if sc is None else YarnScaling(sc["factor"], sc["original"], sc["fast"], sc["slow"]))
        f, m = rotary_frequencies(spec)
        fw, mw = S.rotary_frequencies({"dims": dims, "base": base, "scaling": sc})
        np.testing.assert_allclose(f.numpy(), fw, rtol=1e-14); assert abs(m - mw) < 1e-14
        table = rotary_table(spec, 50, "cuda").double().cpu().numpy()
        ang = np.arange(50)[:, None] * fw
        np.testing.assert_allclose(table, np.concatenate([np.cos(ang) * mw, np.sin(ang) * mw], 1), atol=3e-7)


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("own", [True, False])
def test_latent_prepare(dtype, own):
    from mini_sgl_integer_b200.layers.rotary_float import rotary_table
    from mini_sgl_integer_b200.models.config import RotarySpec, YarnScaling
    rng = np.random.default_rng(1)
    T, H, dim, rot, rank, parts, eps = 9, 3, 20, 14, 35, 2, 1e-2
    sc = ROT["scaling"]
    rope = rotary_table(RotarySpec(12, 5000.0, YarnScaling(sc["factor"], sc["original"], sc["fast"], sc["slow"])), 300, "cuda")
    n = H * (dim + rot) + (rank + rot if own else 0)
    qd = rng.standard_normal((parts, T, n)) * 0.3
    pos = rng.integers(0, 300, T)
    loc = rng.permutation(5 * 16)[:T]
    w = rng.standard_normal(rank)
    full = qd.sum(0)
    lat = fo.pad8(rank + rot)
    qn = torch.zeros(T, H, fo.pad8(dim), dtype=dtype, device="cuda")
    ql = torch.full((T, H, lat), 9.0, dtype=dtype, device="cuda")
    cache = torch.zeros(5, 16, lat, dtype=dtype, device="cuda")
    fo.latent_prepare(dev(qd), i32(pos), i32(loc), rope, dev(w) if own else None, eps, qn, ql, cache if own else None, H, dim, rot, rank)
    q = full[:, :H * (dim + rot)].reshape(T, H, dim + rot)
    close(qn[..., :dim], q[..., :dim], dtype)
    close(ql[..., rank:rank + rot], S.rotate(q[..., dim:], pos, ROT), dtype)
    assert bool((ql[..., :rank] == 9.0).all()) and bool((ql[..., rank + rot:] == 0.0).all())
    rows = cache.view(-1, lat)[loc.tolist()]
    if own:
        d = full[:, H * (dim + rot):]
        close(rows[:, :rank], S.rms_norm(d[:, :rank], w, eps), dtype)
        close(rows[:, rank:rank + rot], S.rotate(d[:, rank:], pos, ROT), dtype)
        assert int((cache.view(-1, lat).abs().sum(1) > 0).sum()) == T
    else:
        assert bool((cache == 0).all())


def attention_case(rng, kv_lens, q_lens, heads, rank, rot, dtype, spike=True):
    """Latent rows in shuffled pages, queries, and a spike: one key far back that a head attends to almost alone."""
    lat, pages = fo.pad8(rank + rot), [-(-n // 16) for n in kv_lens]
    total = sum(pages)
    table = np.full((len(kv_lens), max(pages) + 1), total, dtype=np.int64)     # unused entries name a page of NaNs
    perm = rng.permutation(total)
    cache = torch.full((total + 1, 16, lat), float("nan"), dtype=dtype, device="cuda")
    keys, qs, at = [], [], 0
    for b, (n, ql) in enumerate(zip(kv_lens, q_lens)):
        table[b, :pages[b]] = perm[at:at + pages[b]]
        at += pages[b]
        k = rng.standard_normal((n, rank + rot))
        q = rng.standard_normal((ql, heads, rank + rot))
        if spike and n > 3:
            for h in range(0, heads, 2):
                q[-1, h] = 3.0 * k[int(rng.integers(0, n))]
        k, q = host(dev(k, dtype)), host(dev(q, dtype))
        rows = cache[torch.as_tensor(table[b, :pages[b]]).cuda()].view(-1, lat)
        rows[:n] = 0
        rows[:n, :rank + rot] = dev(k, dtype)
        cache[torch.as_tensor(table[b, :pages[b]]).cuda()] = rows.view(-1, 16, lat)
        keys.append(k); qs.append(q)
    q_lat = torch.zeros(sum(q_lens), heads, lat, dtype=dtype, device="cuda")
    q_lat[..., :rank + rot] = dev(np.concatenate(qs), dtype)
    return cache, i32(table), keys, qs, q_lat


def attention_reference(keys, qs, kv_lens, q_lens, heads, rank, window, scale, sink):
    out = []
    for k, q, n, ql in zip(keys, qs, kv_lens, q_lens):
        s = np.einsum("thd,jd->htj", q, k) * scale
        mask = S.window_mask(n, window)[n - ql:]
        s = np.where(mask[None], s, -np.inf)
        p = np.stack([S.sink_softmax(s[h], sink[h]) for h in range(heads)])
        out.append(np.einsum("htj,jd->thd", p, k[:, :rank]))
    return np.concatenate(out)


@pytest.mark.parametrize("dtype,simple", [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("heads,rank,rot,window", [(1, 24, 8, 5), (3, 40, 16, 31), (5, 72, 24, 33), (16, 128, 32, 100), (20, 256, 64, None), (33, 512, 64, 65),
                                                   (70, 64, 16, 1), (6, 520, 40, 200), (4, 35, 14, 48)])
def test_latent_attention_prompts_portions_and_decode(dtype, simple, heads, rank, rot, window):
    rng = np.random.default_rng(heads * 1000 + rank)
    for kv_lens, q_lens in [([70, 1, 33], [70, 1, 33]), ([260, 64, 97], [37, 2, 1]), ([301, 16, 17, 65], [1, 1, 1, 1])]:
        cache, table, keys, qs, q_lat = attention_case(rng, kv_lens, q_lens, heads, rank, rot, dtype)
        sink = rng.standard_normal(heads) * 2
        sink[0] = 9.0
        scale = (rank + rot) ** -0.5
        want = attention_reference(keys, qs, kv_lens, q_lens, heads, rank, window, scale, sink)
        decode = all(n == 1 for n in q_lens)
        out = torch.full((sum(q_lens), heads, fo.pad8(rank)), 5.0, dtype=dtype, device="cuda")
        fo.latent_attention(q_lat, cache, table, i32(kv_lens), None if decode else i32(np.concatenate([[0], np.cumsum(q_lens)])), dev(sink), out,
                            rank, rot, window or 0, scale, max(q_lens), max(kv_lens), simple=simple)
        close(out[..., :rank], want, dtype, 3e-5, 1.5e-2)


@pytest.mark.parametrize("heads,rank,rot", [(8, 64, 16), (40, 128, 32)])
@pytest.mark.parametrize("splits", [2, 5, 11])
def test_latent_attention_with_split_keys(heads, rank, rot, splits):
    rng = np.random.default_rng(splits)
    kv_lens, q_lens, dtype = [700, 3, 128], [1, 1, 1], torch.bfloat16
    cache, table, keys, qs, q_lat = attention_case(rng, kv_lens, q_lens, heads, rank, rot, dtype)
    sink, scale = rng.standard_normal(heads), 0.1
    for window in (None, 130):
        out = torch.empty(3, heads, rank, dtype=dtype, device="cuda")
        fo.latent_attention(q_lat, cache, table, i32(kv_lens), None, dev(sink), out, rank, rot, window or 0, scale, 1, 700, key_splits=splits)
        close(out, attention_reference(keys, qs, kv_lens, q_lens, heads, rank, window, scale, sink), dtype, 0, 1.5e-2)


def test_window_edge_key_decides():
    """A key exactly at the window's edge holds all the weight; one token further it must be gone."""
    rank, rot, heads, window = 32, 16, 2, 24
    for dtype, simple in [(torch.float32, True), (torch.bfloat16, False)]:
        for n in (24, 25, 40, 41, 64, 65, 100):
            k = np.zeros((n, rank + rot))
            k[:, 0] = 1.0
            for inside in (True, False):
                j = n - window - (0 if inside else 1)          # the oldest visible key, or the one before it
                if j < 0:
                    continue
                kk = k.copy()
                kk[j, 1], kk[j, 2] = 40.0, 8.0
                pages = -(-n // 16)
                cache = torch.zeros(pages + 1, 16, 48, dtype=dtype, device="cuda")
                cache.view(-1, 48)[:n] = dev(kk, dtype)
                q = torch.zeros(1, heads, 48, dtype=dtype, device="cuda")
                q[..., 1] = 1.0
                out = torch.empty(1, heads, rank, dtype=dtype, device="cuda")
                fo.latent_attention(q, cache, i32([list(range(pages))]), i32([n]), None, dev([-3.0, -3.0]), out, rank, rot, window, 1.0, 1, n, simple=simple)
                assert (float(out[0, 0, 2]) > 7.9) == inside
