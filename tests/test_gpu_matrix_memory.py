"""The kernels behind matrix memories and grouped attention one by one, against the numpy functions of oracle/derelorn.py.
bf16 cases feed the reference the rounded operands, so only accumulation order and the final rounding differ."""
from __future__ import annotations

import numpy as np
import pytest
import torch

from mini_sgl_integer_b200.kernel import float_ops as fo
from mini_sgl_integer_b200.layers.float_linear import padded_rows
from oracle import derelorn as D
from oracle import sefevik as S
from tests.test_gpu_float_ops import close, dev, host, i32

pytestmark = pytest.mark.gpu
DT = [torch.float32, torch.bfloat16]
KINDS = {"mlstm": fo.MEMORY_EXP, "mamba": fo.MEMORY_SSD, "delta": fo.MEMORY_DELTA}


class Feeder:
    """Cuts several sequences into steps of unequal portions and describes each step to the kernels."""

    def __init__(self, lens, slots):
        self.lens, self.slots, self.at = lens, slots, [0] * len(lens)

    def step(self, counts):
        who = [i for i, c in enumerate(counts) if c]
        span = [(i, self.at[i], self.at[i] + counts[i]) for i in who]
        for i in who:
            self.at[i] += counts[i]
            assert self.at[i] <= self.lens[i]
        pos = np.concatenate([np.arange(a, b) for _, a, b in span])
        start = np.concatenate([[0], np.cumsum([b - a for _, a, b in span])])
        decode = all(b - a == 1 for _, a, b in span)
        meta = dict(slots=i32([self.slots[i] for i in who]), positions=i32(pos), seq_start=None if decode else i32(start),
                    seq_ids=None if decode else i32(np.repeat(np.arange(len(who)), np.diff(start))))
        return span, meta


def pick(arrays, span):
    return np.concatenate([arrays[i][a:b] for i, a, b in span])


# ----------------------------------------------------------------------------- the scan
def scan_case(kind, rng, lens, H, G, dim, vdim, dtype, strong=True):
    """Operands per sequence."""
    cases = []
    for n in lens:
        q, k, v = rng.standard_normal((n, G, dim)), rng.standard_normal((n, G, dim)), rng.standard_normal((n, H, vdim))
        if strong and n > 40:                                     # the last token asks for one far back
            k[5] *= 6.0
            q[-1] = 6.0 * k[5]
        q, k, v = (host(dev(a, dtype)) for a in (q, k, v))
        if kind == "mlstm":
            g = np.stack([-0.02 * rng.random((n, H)) - 0.4 * (rng.random((n, H)) < 0.05), 3.0 * rng.standard_normal((n, H))], -1)   # log gates f, i
        else:
            g = np.stack([np.exp(-0.02 * rng.random((n, H))), rng.random((n, H))], -1)
        cases.append((q, k, v, host(dev(g))))
    return cases


def scan_oracle(kind, case, H, G, dim, skip):
    """Read-outs, and for mlstm (whose read-outs are not divided yet) the normalisers."""
    q, k, v, g = case
    share = np.arange(H) // (H // G)
    q, k = q[:, share], k[:, share]
    if kind == "mlstm":
        gates, _ = running_max_gates(g, np.zeros(H))
        scan = lambda x: D.ssd_scan(x, k, q * dim ** -0.5, gates[..., 1], gates[..., 0], np.zeros(H))
        num, den = scan(v), np.maximum(np.abs(scan(np.ones((*v.shape[:2], 1)))[..., 0]), gates[..., 2]) + 1e-6
        quotient = D.mlstm_scan(q * dim ** -0.5, k, v, g[..., 1], g[..., 0])
        assert np.abs(num / den[..., None] - quotient).max() < 1e-8 * np.abs(quotient).max()
        return num, den
    if kind == "mamba":
        return D.ssd_scan(v, k, q, g[..., 1], g[..., 0], skip), None
    return D.delta_scan(D.unit(q) * dim ** -0.5, D.unit(k), v, g[..., 1], g[..., 0]), None


def running_max_gates(g, m0):
    """(decay, write, exp(-m)) of log gates [n, H, 2] and the maximum behind them."""
    out, m = [], m0
    for f, i in zip(g[..., 0], g[..., 1]):
        new = np.maximum(f + m, i)
        out.append(np.stack([np.exp(f + m - new), np.exp(i - new), np.exp(-new)], -1))
        m = new
    return np.stack(out), m


@pytest.mark.parametrize("dtype,simple", [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("kind", list(KINDS))
@pytest.mark.parametrize("H,G,dim,vdim", [(2, 1, 8, 8), (3, 3, 20, 37), (4, 2, 32, 64), (2, 2, 64, 40), (2, 1, 72, 136), (3, 1, 128, 24), (1, 1, 200, 72),
                                          (2, 1, 260, 20)])
def test_scan_over_portions_and_steps(dtype, simple, kind, H, G, dim, vdim):
    if kind == "mlstm":
        G = H
    rng = np.random.default_rng(dim + vdim)
    lens, slots = [290, 1, 153, 18], [5, 2, 0, 3]
    cases = scan_case(kind, rng, lens, H, G, dim, vdim, dtype)
    skip = rng.standard_normal(H) if kind == "mamba" else None
    want = [scan_oracle(kind, c, H, G, dim, skip) for c in cases]
    vp, hp = fo.pad8(vdim), fo.pad8(dim)
    state = torch.full((7, H, dim, vp), 123.0, device="cuda")                  # left by earlier requests
    n_state = torch.full((7, H, dim + 1), 55.0, device="cuda")
    m = [np.zeros(H) for _ in lens]
    limit = 3e-5 if simple else 2e-4                              # operands as two bf16 numbers: 16 bits of fraction
    f, scale = Feeder(lens, slots), dim ** -0.5 if kind != "mamba" else 1.0
    for counts in ([40, 1, 16, 2], [2, 0, 1, 3], [1, 0, 1, 1], [133, 0, 64, 1], [1, 0, 0, 1], [113, 0, 71, 10]):
        span, md = f.step(counts)
        T = sum(b - a for _, a, b in span)
        rows = torch.full((T, 2 * G * hp + H * vp), float("nan"), dtype=dtype, device="cuda")
        for off, which, heads, size, pad in ((0, 0, G, dim, hp), (G * hp, 1, G, dim, hp), (2 * G * hp, 2, H, vdim, vp)):
            rows[:, off:off + heads * pad].view(T, heads, pad)[..., :size] = dev(pick([c[which] for c in cases], span), dtype)
        if kind == "mlstm":
            gates = []
            for i, a, b in span:
                g, m[i] = running_max_gates(cases[i][3][a:b], m[i])
                gates.append(g)
            gates = np.concatenate(gates)
        else:
            gates = pick([c[3] for c in cases], span)
        g4 = torch.zeros(T, H, 4, device="cuda")
        g4[..., :gates.shape[-1]] = dev(np.concatenate([np.log(gates[..., :1]), gates[..., 1:]], -1))
        out, den = torch.empty(T, H * vdim, device="cuda"), torch.empty(T, H, device="cuda")
        fo.memory_scan(rows, (0, G * hp, 2 * G * hp), G, H, dim, vdim, KINDS[kind], g4, scale, None if skip is None else dev(skip), state,
                       n_state if kind == "mlstm" else None, md["slots"], md["positions"], md["seq_start"], out, den if kind == "mlstm" else None,
                       max(counts), simple=simple)
        close(out.view(T, H, vdim), pick([w[0] for w in want], span), torch.float32, limit)
        if kind == "mlstm":
            close(den, pick([w[1] for w in want], span), torch.float32, limit)
    assert bool((state[[1, 4, 6]] == 123.0).all()) and bool((n_state[[1, 4, 6]] == 55.0).all())


def test_scan_does_not_depend_on_how_a_prompt_is_cut():
    """Token by token in the same order: the same bits whatever the portions (two tokens or more), batch and slot are."""
    rng = np.random.default_rng(1)
    H, dim, vdim, n = 2, 64, 48, 70
    q = torch.randn(n, 2 * H * dim + H * vdim, device="cuda").to(torch.bfloat16)
    g4 = torch.rand(n, H, 4, device="cuda")
    g4[..., 0] *= -0.1
    res = []
    for cuts in ([], [2, 33, 49, 66], [16, 32, 48, 64]):
        state, out = torch.zeros(4, H, dim, vdim, device="cuda"), torch.empty(n, H * vdim, device="cuda")
        slot = int(rng.integers(0, 4))
        for a, b in zip([0] + cuts, cuts + [n]):
            o = torch.empty(b - a, H * vdim, device="cuda")
            fo.memory_scan(q[a:b], (0, H * dim, 2 * H * dim), H, H, dim, vdim, fo.MEMORY_DELTA, g4[a:b].contiguous(), 0.125, None, state, None,
                           i32([slot]), i32(np.arange(a, b)), i32([0, b - a]), o, None, b - a, simple=True)
            out[a:b] = o
        res.append(out)
    assert torch.equal(res[0], res[1]) and torch.equal(res[0], res[2])


# ----------------------------------------------------------------------------- preparation
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("parts", [1, 3])
@pytest.mark.parametrize("kind,taps,H,G,dim,vdim", [("mlstm", 0, 4, 4, 24, 16), ("mlstm", 0, 3, 3, 7, 9), ("mamba", 3, 6, 2, 16, 8), ("mamba", 5, 5, 1, 10, 6),
                                                    ("mamba", 1, 4, 2, 12, 8), ("delta", 4, 4, 2, 16, 24), ("delta", 2, 3, 1, 11, 13)])
def test_prepare_over_portions_and_steps(dtype, parts, kind, taps, H, G, dim, vdim):
    rng = np.random.default_rng(taps * 100 + dim)
    order = "vkq" if kind == "mamba" else "qkv"
    seg = [(H * vdim, vdim) if c == "v" else (G * dim, dim) for c in order]
    width, first = sum(w for w, _ in seg), 8 if kind == "mamba" else 3
    n = -(-(first + width + 2 * H) // 8) * 8
    col_a, col_b = first + width, first + width + H
    lens, slots = [61, 1, 40, 9], [1, 4, 0, 3]
    pre = [host(dev(rng.standard_normal((m, n)) * 2)) for m in lens]
    cw = rng.standard_normal((width, taps)) if taps else None
    cb = rng.standard_normal(width) if kind == "mamba" else None
    ga, gb, cap = rng.standard_normal(H), rng.standard_normal(H), 3.5
    want_rows, want_gates = [], []
    for x in pre:
        c = x[:, first:first + width]
        want_rows.append(S.silu(D.causal_conv(c, cw, cb)) if taps else c)
        a, b = x[:, col_a:col_a + H], x[:, col_b:col_b + H]
        if kind == "mlstm":
            soft = lambda z: cap * np.tanh(z / cap)
            f, i = -S.softplus(-soft(a + ga)), soft(b + gb)
            g = running_max_gates(np.stack([f, i], -1), np.zeros(H))[0]
            want_gates.append(np.concatenate([np.log(g[..., :1]), g[..., 1:]], -1))
        else:
            dt = S.softplus(a + gb)
            want_gates.append(np.stack([-np.exp(ga) * dt, dt if kind == "mamba" else S.sigmoid(b)], -1))
    conv_state = torch.full((6, max(taps - 1, 0), width), 77.0, device="cuda")
    n_state = torch.full((6, H, dim + 1), 55.0, device="cuda")
    padded = sum(w // h * fo.pad8(h) for w, h in seg)
    f = Feeder(lens, slots)
    for counts in ([20, 1, 1, 2], [1, 0, 3, 1], [1, 0, 1, 1], [2, 0, 1, 0], [1, 0, 0, 1], [36, 0, 34, 4]):
        span, md = f.step(counts)
        x = pick(pre, span)
        T = len(x)
        split = rng.standard_normal((parts, T, n))
        split[-1] = x - split[:-1].sum(0)
        y = dev(split)
        out = torch.full((T, padded), 9.0, dtype=dtype, device="cuda")
        gates = torch.empty(T, H, 4, device="cuda")
        fo.memory_prepare(y, first, seg, None if cw is None else dev(cw), None if cb is None else dev(cb), conv_state if taps else None, md["slots"],
                          md["positions"], md["seq_start"], md["seq_ids"], out, KINDS[kind], H, (col_a, col_b if kind != "mamba" else col_a), dev(ga), dev(gb),
                          gates, cap, n_state if kind == "mlstm" else None)
        at_p = at = 0
        ref = pick(want_rows, span)
        for w, h in seg:
            got = out[:, at_p:at_p + w // h * fo.pad8(h)].view(T, w // h, -1)
            close(got[..., :h].reshape(T, w), ref[:, at:at + w], dtype, 5e-5)
            assert bool((got[..., h:] == 9.0).all())
            at_p, at = at_p + w // h * fo.pad8(h), at + w
        wg = pick(want_gates, span)
        close(gates[..., :wg.shape[-1]], wg, torch.float32, 5e-5)
        if kind == "mlstm":
            assert bool((n_state[..., :dim] == 55.0).all())
    assert bool((conv_state[[2, 5]] == 77.0).all()) and bool((n_state[[2, 5]] == 55.0).all())


@pytest.mark.parametrize("dtype", DT)
def test_prepare_of_a_long_prompt(dtype):
    """Several token blocks per sequence, whose first taps reach into the block before or into the stored inputs."""
    rng = np.random.default_rng(4)
    H, G, dim, vdim, taps = 8, 4, 64, 64, 4
    seg = [(G * dim, dim), (G * dim, dim), (H * vdim, vdim)]
    width = sum(w for w, _ in seg)
    lens = [3000, 2100]
    pre = [host(dev(rng.standard_normal((m, width + 2 * H)))) for m in lens]
    cw = rng.standard_normal((width, taps))
    want = [S.silu(D.causal_conv(x[:, :width], cw)) for x in pre]
    conv = torch.full((2, taps - 1, width), 9.0, device="cuda")
    f = Feeder(lens, [1, 0])
    for counts in ([1700, 901], [1299, 1199], [1, 0]):
        span, md = f.step(counts)
        x = pick(pre, span)
        out, gates = torch.empty(len(x), width, dtype=dtype, device="cuda"), torch.empty(len(x), H, 4, device="cuda")
        fo.memory_prepare(dev(x[None]), 0, seg, dev(cw), None, conv, md["slots"], md["positions"], md["seq_start"], md["seq_ids"], out, fo.MEMORY_DELTA, H,
                          (width, width + H), dev(np.zeros(H)), dev(np.zeros(H)), gates)
        close(out, pick(want, span), dtype, 5e-5)


# ----------------------------------------------------------------------------- output
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,V,group", [(1, 8, 8), (4, 24, 24), (6, 16, 32), (5, 6, 15), (3, 40, 120), (32, 128, 128), (32, 64, 2048), (2, 9, 9), (3, 64, 64), (2, 1024, 1024)])
def test_memory_output(dtype, H, V, group):
    rng = np.random.default_rng(H * V)
    T, n, eps, parts = 5, H * V, 1e-3, 2
    col = 12 if V % 4 == 0 else 11
    o, den = rng.standard_normal((T, n)) * 0.1, 0.5 + rng.random((T, H))
    y = rng.standard_normal((parts, T, col + n + 4))
    z, w = y.sum(0)[:, col:col + n], rng.standard_normal(n)
    norm = lambda x: S.rms_norm(x.reshape(T, -1, group), 1.0, eps).reshape(T, n)
    out = fo.rows(T, n, dtype, "cuda")
    if group == V:
        scaled = (o.reshape(T, H, V) / den[..., None]).reshape(T, n)
        fo.memory_output(dev(o), dev(den), H, V, group, dev(y), col, fo.GATE_SIGMOID_AFTER, dev(w), eps, out)
        close(out, norm(scaled) * w * S.sigmoid(z), dtype, 5e-5)
    fo.memory_output(dev(o), None, H, V, group, dev(y), col, fo.GATE_SILU_AFTER, dev(w[:group]), eps, out)
    close(out, norm(o) * np.tile(w[:group], n // group) * S.silu(z), dtype, 5e-5)
    fo.memory_output(dev(o), None, H, V, group, dev(y), col, fo.GATE_SILU_BEFORE, dev(w), eps, out)
    close(out, norm(o * S.silu(z)) * w, dtype, 5e-5)


@pytest.mark.parametrize("H,V,rows", [(4, 24, 2501), (2, 256, 4801), (1, 100, 2369)])
def test_memory_output_of_many_short_rows(H, V, rows):
    """Several rows per CTA, the last one with fewer."""
    rng = np.random.default_rng(rows)
    n, eps = H * V, 1e-4
    o, y, w = rng.standard_normal((rows, n)), rng.standard_normal((1, rows, 2 * n)), rng.standard_normal(n)
    out = fo.rows(rows, n, torch.bfloat16, "cuda")
    fo.memory_output(dev(o), None, H, V, V, dev(y), n, fo.GATE_SIGMOID_AFTER, dev(w), eps, out)
    close(out, S.rms_norm(o.reshape(rows, H, V), 1.0, eps).reshape(rows, n) * w * S.sigmoid(y[0, :, n:]), torch.bfloat16)


# ----------------------------------------------------------------------------- gated feed-forward, ends of a sublayer
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("T,ff,width", [(1, 16, 24), (3, 37, 50), (70, 200, 64), (200, 4096, 128), (300, 130, 72), (1100, 5000, 96), (4, 5000, 2048)])
def test_gated_mlp(dtype, T, ff, width):
    from mini_sgl_integer_b200.layers.float_linear import GatedSiluMLP
    g = torch.Generator().manual_seed(T + ff)
    w = {k: (torch.randn(*s, generator=g) * s[1] ** -0.5).to(dtype) for k, s in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))}
    x = padded_rows(torch.randn(T, width, generator=g) * 2, dtype, "cuda")
    m = GatedSiluMLP(width, ff, dtype, "cuda")
    m.load_state_dict(dict(w))
    act = S.silu(host(x) @ host(w["gate"]).T) * (host(x) @ host(w["up"]).T)
    if dtype == torch.bfloat16:
        act = host(dev(act, dtype))
    got = m.forward(x).sum(0)
    close(got, act @ host(w["down"]).T, dtype, 2e-5, 8e-3)
    fo.check_status()


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("width", [24, 90, 1024, 5000])
def test_sublayer_end_of_two_mixers_and_of_a_pass(dtype, width):
    rng = np.random.default_rng(width)
    T, eps, parts = 4, 1e-3, 1 if width % 4 else 3
    y, y2, x = rng.standard_normal((parts, T, width)) * 0.02, rng.standard_normal((1, T, width)) * 5, rng.standard_normal((T, width))
    w, w1, w2, add, fw = (rng.standard_normal(width) for _ in range(5))
    xs, xt = dev(x), fo.rows(T, width, dtype, "cuda")
    mean = 0.5 * (S.rms_norm(y.sum(0), w1, eps) + S.rms_norm(y2[0], w2, eps))
    want = x + S.rms_norm(mean, w, eps) + add
    fo.sublayer_end(dev(y), xs, dev(w), eps, xs, xt, dtype, mean_with=(dev(w1), dev(y2), dev(w2)), add=dev(add), final_w=dev(fw))
    close(xs, want, torch.float32)
    close(xt, S.rms_norm(want, fw, eps), dtype)
    fo.sublayer_end(dev(y), None, dev(w), eps, xs, xt, dtype, final_w=dev(fw))
    want = S.rms_norm(y.sum(0), w, eps)
    close(xs, want, torch.float32)
    close(xt, S.rms_norm(want, fw, eps), dtype)
    fo.sublayer_end(None, xs, None, eps, xs, xt, dtype, add=dev(add), final_w=dev(fw))
    close(xs, want + add, torch.float32)
    close(xt, S.rms_norm(want + add, fw, eps), dtype)


# ----------------------------------------------------------------------------- grouped attention
@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("H,G,dim,vdim,normed", [(4, 2, 16, 24, True), (3, 1, 9, 7, True), (32, 8, 128, 128, True), (2, 2, 8, 8, False)])
def test_grouped_prepare(dtype, H, G, dim, vdim, normed):
    rng = np.random.default_rng(dim)
    T, parts, eps, col = 7, 2, 1e-2, 5
    n = col + (H + G) * dim + G * vdim
    y = rng.standard_normal((parts, T, n)) * 0.4
    qw, kw = rng.standard_normal(H * dim), rng.standard_normal(G * dim)
    x, loc = y.sum(0)[:, col:], rng.permutation(4 * 16)[:T]
    q, k, v = np.split(x, [H * dim, (H + G) * dim], axis=1)
    if normed:
        q, k = S.rms_norm(q, qw, eps), S.rms_norm(k, kw, eps)
    dp, vp = fo.pad8(dim), fo.pad8(vdim)
    qo = torch.full((T, H, dp), 9.0, dtype=dtype, device="cuda")
    kc, vc = torch.full((4, 16, G * dp), 3.0, dtype=dtype, device="cuda"), torch.full((4, 16, G * vp), 3.0, dtype=dtype, device="cuda")
    fo.grouped_prepare(dev(y), (col, col + H * dim, col + (H + G) * dim), dev(qw) if normed else None, dev(kw) if normed else None, eps, i32(loc), qo, kc, vc,
                       H, G, dim, vdim)
    close(qo[..., :dim], q.reshape(T, H, dim), dtype)
    at = torch.as_tensor(loc).cuda()
    close(kc.view(-1, G, dp)[at][..., :dim], k.reshape(T, G, dim), dtype)
    close(vc.view(-1, G, vp)[at][..., :vdim], v.reshape(T, G, vdim), dtype)
    assert bool((qo[..., dim:] == 0).all()) and bool((kc.view(-1, G, dp)[at][..., dim:] == 0).all())
    rest = torch.ones(64, dtype=torch.bool, device="cuda")
    rest[at] = False
    assert bool((kc.view(-1, G * dp)[rest] == 3.0).all()) and bool((vc.view(-1, G * vp)[rest] == 3.0).all())


def paged_case(rng, kv_lens, q_lens, H, G, dim, vdim, window, dtype):
    """Keys and values in shuffled pages; pages behind the window and unused ones hold NaN, every other head's last query
    looks for one key."""
    dp, vp, pages = fo.pad8(dim), fo.pad8(vdim), [-(-n // 16) for n in kv_lens]
    total = sum(pages)
    table = np.full((len(kv_lens), max(pages) + 1), total, dtype=np.int64)
    perm = rng.permutation(total)
    kc = torch.full((total + 1, 16, G, dp), float("nan"), dtype=dtype, device="cuda")
    vc = torch.full((total + 1, 16, G, vp), float("nan"), dtype=dtype, device="cuda")
    qs, ks, vs, at = [], [], [], 0
    for b, (n, ql) in enumerate(zip(kv_lens, q_lens)):
        table[b, :pages[b]] = perm[at:at + pages[b]]
        at += pages[b]
        k, v, q = rng.standard_normal((n, G, dim)), rng.standard_normal((n, G, vdim)), rng.standard_normal((ql, H, dim))
        for h in range(0, H, 2):
            q[-1, h] = 4.0 * k[int(rng.integers(max(0, n - (window or n)), n)), h // (H // G)]
        q, k, v = (host(dev(a, dtype)) for a in (q, k, v))
        first = max(0, n - ql - (window or n) + 1) // 16 * 16
        for pos in range(first, n):
            pg, off = int(table[b, pos // 16]), pos % 16
            kc[pg, off] = 0
            vc[pg, off] = 0
            kc[pg, off, :, :dim], vc[pg, off, :, :vdim] = dev(k[pos], dtype), dev(v[pos], dtype)
        table[b, :first // 16] = total
        qs.append(q); ks.append(k); vs.append(v)
    q = torch.zeros(sum(q_lens), H, dp, dtype=dtype, device="cuda")
    q[..., :dim] = dev(np.concatenate(qs), dtype)
    return q, kc.view(total + 1, 16, -1), vc.view(total + 1, 16, -1), i32(table), qs, ks, vs


def grouped_reference(qs, ks, vs, window, scale):
    out = []
    for q, k, v in zip(qs, ks, vs):
        n, ql = len(k), len(q)
        full = np.concatenate([np.zeros((n - ql, *q.shape[1:])), q])
        out.append(D.grouped_attention(full, k, v, window, scale)[n - ql:])
    return np.concatenate(out)


@pytest.mark.parametrize("dtype,simple", [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("H,G,dim,vdim,window", [(1, 1, 8, 8, 5), (4, 2, 24, 40, 31), (6, 2, 64, 64, 64), (8, 1, 128, 96, 100), (40, 2, 72, 200, 33),
                                                 (5, 5, 256, 16, None), (70, 1, 16, 128, 1), (3, 3, 9, 7, 48), (32, 8, 128, 128, 80)])
def test_grouped_attention_prompts_portions_and_decode(dtype, simple, H, G, dim, vdim, window):
    rng = np.random.default_rng(H * 1000 + dim)
    for kv_lens, q_lens in [([70, 1, 33], [70, 1, 33]), ([260, 64, 97], [37, 2, 1]), ([301, 16, 17, 65], [1, 1, 1, 1])]:
        q, kc, vc, table, qs, ks, vs = paged_case(rng, kv_lens, q_lens, H, G, dim, vdim, window, dtype)
        scale = 1.5 * dim ** -0.5
        want = grouped_reference(qs, ks, vs, window, scale).reshape(sum(q_lens), -1)
        decode = all(n == 1 for n in q_lens)
        out = fo.rows(sum(q_lens), H * vdim, dtype, "cuda")
        fo.grouped_attention(q, kc, vc, table, i32(kv_lens), None if decode else i32(np.concatenate([[0], np.cumsum(q_lens)])), out, G, dim, vdim,
                             window or 0, scale, max(q_lens), max(kv_lens), simple=simple)
        close(out, want, dtype, 3e-5, 1.5e-2)


@pytest.mark.parametrize("H,G", [(8, 2), (40, 2)])
@pytest.mark.parametrize("splits", [2, 3, 7])
def test_grouped_attention_with_split_keys(H, G, splits):
    rng = np.random.default_rng(splits)
    kv_lens, dtype, dim, vdim = [700, 3, 128], torch.bfloat16, 64, 40
    for window in (None, 130):
        q, kc, vc, table, qs, ks, vs = paged_case(rng, kv_lens, [1, 1, 1], H, G, dim, vdim, window, dtype)
        out = fo.rows(3, H * vdim, dtype, "cuda")
        fo.grouped_attention(q, kc, vc, table, i32(kv_lens), None, out, G, dim, vdim, window or 0, 0.2, 1, 700, key_splits=splits)
        close(out, grouped_reference(qs, ks, vs, window, 0.2).reshape(3, -1), dtype, 0, 1.5e-2)


def test_window_edge_key_decides():
    """A key exactly at the window's edge holds all the weight; one token further it must be gone."""
    H, G, dim, vdim, window = 4, 2, 16, 24, 24
    for dtype in DT:
        for decode in (True, False):
            for n in (24, 25, 40, 41, 64, 65, 88, 100):
                for inside in (True, False):
                    j = n - window - (0 if inside else 1)                       # the oldest visible key, or the one before it
                    if j < 0:
                        continue
                    pages = -(-n // 16)
                    kc, vc = torch.zeros(pages, 16, G * dim, dtype=dtype, device="cuda"), torch.zeros(pages, 16, G * vdim, dtype=dtype, device="cuda")
                    kc.view(-1, G, dim)[j, :, 1] = 40.0
                    vc.view(-1, G, vdim)[j, :, 2] = 8.0
                    ql = 1 if decode else 5
                    q = torch.zeros(ql, H, dim, dtype=dtype, device="cuda")
                    q[..., 1] = 1.0
                    out = fo.rows(ql, H * vdim, dtype, "cuda")
                    fo.grouped_attention(q, kc, vc, i32([list(range(pages))]), i32([n]), None if decode else i32([0, ql]), out, G, dim, vdim, window, 1.0, ql, n)
                    last = out[-1].view(H, vdim)[:, 2].float()
                    assert bool(((last > 7.9) == inside).all()), (n, inside, decode)
