"""Derelorn without a GPU: configuration, the C ABI's argument checks, and that the tests' own models would show a fault
(mistakes planted in the oracle)."""
from __future__ import annotations

import copy
import ctypes

import numpy as np
import pytest

from mini_sgl_integer_b200 import _lib
from mini_sgl_integer_b200.models import SUPPORTED_MODELS
from mini_sgl_integer_b200.models.config import DerelornConfig, RunMemory
from mini_sgl_integer_b200.models.weight import architecture_of, load_checkpoint, load_config_dict
from oracle import derelorn as D
from oracle import sefevik as S
from tests.derelorn_util import CONFIGS, attn, delta, float_weights, logit_error, make_weights, mamba, mlstm, model, parallel, write_model


# ----------------------------------------------------------------------------- configuration
def test_configuration_is_read_from_the_file(tmp_path):
    cfg = CONFIGS["mixed"]
    write_model(str(tmp_path), cfg, make_weights(cfg, 1))
    d = load_config_dict(str(tmp_path))
    entry = SUPPORTED_MODELS[architecture_of(d)]()
    c = entry.parse_config(d)
    assert (c.vocab_size, c.hidden_size, c.num_layers) == (123, 80, 4)
    assert [(r.layer, r.begins) for r in c.runs] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert c.cache_layers == (0,) and c.max_window == 21 and entry.window(c) == 21 and entry.needs_pages(c)
    assert c.memory[0].planes == ((2, 16), (2, 24)) and dict(c.memory[0].state) == {"S": (6, 24, 16), "conv": (3, 192)}
    assert c.memory[1] == RunMemory(state=(("S", (3, 24, 16)), ("n", (3, 25))))
    assert dict(c.memory[2].state)["conv"] == (2, 2 * 2 * 24 + 6 * 16)
    assert set(load_checkpoint(str(tmp_path))) == set(make_weights(cfg, 1))


def test_every_pass_of_a_loop_has_its_own_cache():
    c = DerelornConfig.from_dict(CONFIGS["loop over everything"])
    assert len(c.runs) == len(c.memory) == 4 and c.cache_layers == (0, 2) and [r.begins for r in c.runs] == [0, None, 1, None]
    assert DerelornConfig.from_dict(CONFIGS["one layer"]).max_window == 0
    assert DerelornConfig.from_dict(CONFIGS["wide heads"]).max_window is None          # one of its windows is unbounded
    for name, cfg in CONFIGS.items():
        assert [(r.layer, r.begins) for r in DerelornConfig.from_dict(cfg).runs] == D.schedule(cfg), name


@pytest.mark.parametrize("change", [
    lambda c: c["loop"].update(stop=5), lambda c: c["loop"].update(start=3), lambda c: c["loop"].update(times=0),
    lambda c: c["layers"][2]["mixer"].update(kv_heads=4), lambda c: c["layers"][2]["mixer"].update(conv=0), lambda c: c["layers"][1].update(type="other"),
    lambda c: c["layers"][1].update(type="mingru", mixer={"width": 8}), lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=5),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), lambda c: c["layers"][0]["mixer"]["right"].update(groups=4),
    lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=7), lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0),
    lambda c: c["layers"][1]["mlp"].update(kind="sparse"), lambda c: c.update(architecture="Other")])
def test_configurations_that_make_no_sense_are_refused(change):
    c = copy.deepcopy(CONFIGS["mixed"])
    change(c)
    with pytest.raises(ValueError):
        DerelornConfig.from_dict(c)


# ----------------------------------------------------------------------------- C ABI
def test_entry_points_reject_bad_arguments_before_launch():
    one = ctypes.c_void_p(16)

    def code(name, *args):
        with pytest.raises(_lib.B200Error) as e:
            _lib.call(name, *args)
        return e.value.code

    def segments(*v):
        return ctypes.cast((ctypes.c_int32 * 6)(*v), ctypes.c_void_p)
    prepare = lambda seg, pitch=64, kind=2, taps=2, conv=one, start=None, ids=None: (
        "b200f_memory_prepare", one, 1, 0, pitch, 0, seg, conv, None, taps, one, one, one, start, ids, one, 64, 1, kind, 2, 48, 50, one, one, 0.0, one, None, 0,
        3, 3, None)
    ok = segments(16, 8, 16, 8, 16, 8)
    assert code(*prepare(segments(16, 8, 15, 8, 16, 8))) == -2
    assert code(*prepare(ok, pitch=51)) == -2                      # the gates' columns do not fit
    assert code(*prepare(ok, kind=5)) == -4
    assert code(*prepare(ok, conv=None)) == -1
    assert code(*prepare(ok, start=one)) == -1                     # sequence bounds without sequence ids
    assert code(*prepare(ok, kind=0)) == -2                        # exponential gates without their state
    scan = lambda dim=8, heads=2, qk=2, q_off=0, pitch=48, den=None, kind=1, dtype=1: (
        "b200f_memory_scan", one, dtype, pitch, q_off, 16, 32, qk, heads, dim, 8, kind, one, 1.0, None, one, None, one, one, None, one, den, 3, 3, 1, None, 0, None)
    assert code(*scan(qk=3)) == -2
    assert code(*scan(pitch=40)) == -2
    assert code(*scan(dim=600)) == -4
    assert code(*scan(q_off=4)) == -3
    assert code(*scan(kind=0)) == -1
    assert code(*scan(dtype=9)) == -4
    out = lambda group=8, gate=1, norm=16: ("b200f_memory_output", one, None, 2, 8, group, one, 1, 0, 32, 0, gate, one, norm, 1e-5, one, 16, 1, 3, None)
    assert code(*out(group=5)) == -2 and code(*out(norm=3)) == -2 and code(*out(gate=3)) == -4
    assert code("b200f_gated_silu", one, 1, 0, 32, one, 1, 2, 17, 24, None) == -2
    assert code("b200f_grouped_prepare", one, 1, 0, 64, 0, 32, 48, one, one, 1e-5, one, one, one, one, 1, 2, 4, 3, 8, 8, 8, 8, 32, None) == -2
    attention = lambda kv=2, max_q=1, splits=1, ws=None, pitch=32: ("b200f_grouped_attn", one, one, one, one, 4, one, None, one, 1, 2, 2, max_q, 4, kv, 8, 8, 8, 8,
                                                                   pitch, 0, 1.0, splits, ws, 0, None)
    assert code(*attention(kv=3)) == -2 and code(*attention(max_q=2)) == -2 and code(*attention(pitch=31)) == -2 and code(*attention(splits=2)) == -1
    gemm = ("b200f_gemm", one, one, one, 1, 0, 4, 40, 8, 1, 8, 0, 8, 0, 24, 0, 1, 0, 2, 0.0, 0.0, None)
    assert code(*gemm) == -4                                       # gated columns come in blocks of 32


# ----------------------------------------------------------------------------- the oracle's mechanisms against their definitions
def test_running_maximum_changes_nothing_but_the_range():
    """Without the maximum the recurrence is S_t = e^f S + e^i k v^T, divided by max(|n . q|, 1)."""
    rng = np.random.default_rng(0)
    T, H, dim, vdim = 30, 2, 6, 5
    q, k, v = (rng.standard_normal((T, H, n)) for n in (dim, dim, vdim))
    i, f = rng.standard_normal((T, H)), -rng.random((T, H))
    got = D.mlstm_scan(q, k, v, i, f)
    for h in range(H):
        for t in (0, 7, 29):
            w = np.array([np.exp(i[s, h] + f[s + 1:t + 1, h].sum()) * (k[s, h] @ q[t, h]) for s in range(t + 1)])
            np.testing.assert_allclose(got[t, h], (w @ v[:t + 1, h]) / max(abs(w.sum()), 1.0), rtol=2e-5)
    assert np.isfinite(D.mlstm_scan(q, k, v, i + 800.0, f)).all()


def test_delta_rule_replaces_what_the_memory_returns():
    rng = np.random.default_rng(1)
    k = D.unit(rng.standard_normal((2, 1, 8)))
    k[1] = k[0]
    v = rng.standard_normal((2, 1, 4))
    one = np.ones((2, 1))
    np.testing.assert_allclose(D.delta_scan(k, k, v, one, one)[1, 0], v[1, 0], rtol=1e-5, atol=1e-6)       # the old value is gone
    np.testing.assert_allclose(D.delta_scan(k, k, v, 0.5 * one, one)[1, 0], 0.25 * v[0, 0] + 0.5 * v[1, 0], rtol=1e-5, atol=1e-6)


def test_convolution_is_causal_and_its_last_tap_is_the_current_token():
    x = np.zeros((6, 1))
    x[2] = 1.0
    np.testing.assert_array_equal(D.causal_conv(x, np.array([[5.0, 3.0, 2.0]]))[:, 0], [0, 0, 2, 3, 5, 0])


# ----------------------------------------------------------------------------- the tests' models show faults
def _probe():
    cfg = model(50, 40, [parallel(attn(4, 2, 8, 8, 20, 1.0), mamba(4, 8, 12, 2, 3, 2), 32), mlstm(2, 12, 16, 24, cap=6.0), delta(4, 2, 12, 8, 4, 24)], loop=(1, 3, 2))
    return cfg, float_weights(make_weights(cfg, 9)), np.random.default_rng(2).integers(0, 50, 90)


FAULTS = ["window + 1", "window - 1", "norm per head", "key head by remainder", "scale of the head", "one group of B and C", "one norm group", "gate behind the norm",
          "skip left out", "convolution bias", "taps reversed", "clamped dt", "maximum from minus infinity", "normaliser left out", "gate cap", "shared state of the passes",
          "step vectors left out", "step vector of the first pass", "state lost", "convolution lost", "read before write", "beta left out", "decay inside the write",
          "unit vectors left out", "sum instead of mean", "output norms of the sides", "no output norm", "eps", "embedding norm"]


@pytest.mark.parametrize("fault", FAULTS)
def test_planted_mistakes_show(fault, monkeypatch):
    cfg, w, ids = _probe()
    want = D.forward(ids, cfg, w)
    bad, wb = copy.deepcopy(cfg), dict(w)
    left, right = bad["layers"][0]["mixer"]["left"], bad["layers"][0]["mixer"]["right"]
    swap = lambda name, fn: monkeypatch.setattr(D, name, fn)
    keep = {n: getattr(D, n) for n in ("rms_norm", "grouped_attention", "ssd_scan", "mlstm_scan", "delta_scan", "causal_conv", "unit", "softplus", "silu", "schedule", "parallel")}

    def cut(fn, seq, at=60):
        """A recurrence that starts anew at token 60."""
        return lambda *a: np.concatenate([fn(*[x[:at] if i in seq else x for i, x in enumerate(a)]), fn(*[x[at:] if i in seq else x for i, x in enumerate(a)])])
    if fault.startswith("window"):
        left["mask"]["size"] += 1 if "+" in fault else -1
    elif fault == "norm per head":
        def attention(q, k, v, *a):
            unit = lambda x: x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True))
            return keep["grouped_attention"](unit(q), unit(k), v, *a)
        swap("grouped_attention", attention)
    elif fault == "key head by remainder":
        swap("grouped_attention", lambda q, k, v, *a: keep["grouped_attention"](q, np.concatenate([k, k], 1)[:, ::1], np.concatenate([v, v], 1), *a))
    elif fault == "scale of the head":
        left["scale"] = left["dim"] ** -0.5
    elif fault == "one group of B and C":
        swap("ssd_scan", lambda x, B, C, *a: keep["ssd_scan"](x, np.repeat(B[:, :1], 4, 1), np.repeat(C[:, :1], 4, 1), *a))
    elif fault == "one norm group":
        right["norm_groups"] = 1
    elif fault == "gate behind the norm":
        def mamba_behind(h, mix, weights, pre, eps):
            z = S.silu((h @ weights[pre + "in"].T)[:, :mix["heads"] * mix["vdim"]])
            other = dict(weights)
            other[pre + "o"] = np.eye(z.shape[1])
            monkeypatch.setattr(D, "silu", lambda v: np.ones_like(v) if v.shape == z.shape else keep["silu"](v))
            y = mamba2(h, mix, other, pre, eps)
            monkeypatch.setattr(D, "silu", keep["silu"])
            return (y * z) @ weights[pre + "o"].T
        mamba2 = D.mamba2
        swap("mamba2", mamba_behind)
    elif fault == "skip left out":
        wb["l0.mix.right.D"] = 0 * w["l0.mix.right.D"]
    elif fault == "convolution bias":
        wb["l0.mix.right.conv.b"] = 0 * w["l0.mix.right.conv.b"]
    elif fault == "taps reversed":
        for k in w:
            if k.endswith(".conv"):
                wb[k] = w[k][:, ::-1]
    elif fault == "clamped dt":
        swap("softplus", lambda v: np.clip(keep["softplus"](v), 0.05, None))
    elif fault == "maximum from minus infinity":
        def scan(q, k, v, i, f):
            first = i.copy()
            shift = np.minimum(first[0], 0.0)                      # the maximum of a sequence that begins with i[0] < 0
            return keep["mlstm_scan"](q, k, v, i - shift, f)
        swap("mlstm_scan", scan)
    elif fault == "normaliser left out":
        swap("mlstm_scan", lambda q, k, v, i, f: keep["ssd_scan"](v, k, q, np.exp(i), np.exp(f), np.zeros(q.shape[1])) + 1.0)
    elif fault == "gate cap":
        bad["layers"][1]["mixer"]["gate_cap"] = 60.0
    elif fault == "shared state of the passes":
        bad["loop"]["times"] = 1
    elif fault == "step vectors left out":
        wb["loop.step"] = 0 * w["loop.step"]
    elif fault == "step vector of the first pass":
        wb["loop.step"] = w["loop.step"][[0, 0]]
    elif fault == "state lost":
        swap("delta_scan", cut(keep["delta_scan"], range(5)))
    elif fault == "convolution lost":
        swap("causal_conv", cut(keep["causal_conv"], (0,)))
    elif fault == "read before write":
        def delta_before(q, k, v, beta, g):
            own = np.einsum("thd,thd->th", q, k)[..., None]
            out = keep["delta_scan"](q, k, v, beta, g)
            return out - 0.5 * own * v * beta[..., None]
        swap("delta_scan", delta_before)
    elif fault == "beta left out":
        swap("delta_scan", lambda q, k, v, beta, g: keep["delta_scan"](q, k, v, np.ones_like(beta), g))
    elif fault == "decay inside the write":
        swap("delta_scan", lambda q, k, v, beta, g: keep["delta_scan"](q, k, v * g[..., None], beta, g))
    elif fault == "unit vectors left out":
        swap("unit", lambda x: x)
    elif fault == "sum instead of mean":
        for k in ("left.out", "right.out"):
            wb["l0.mix." + k] = w["l0.mix." + k] * (2.0 if k == "left.out" else 1.0)
    elif fault == "output norms of the sides":
        wb["l0.mix.left.out"], wb["l0.mix.right.out"] = w["l0.mix.right.out"], w["l0.mix.left.out"]
    elif fault == "no output norm":
        wb["l1.norm1b"] = np.ones_like(w["l1.norm1b"])
    elif fault == "eps":
        bad["norm"]["eps"] = 1e-2
    else:
        wb["embed.norm"] = np.ones_like(w["embed.norm"])
    err = logit_error(D.forward(ids, bad, wb), want)
    assert err.max() > 2e-3, err.max()                            # the 32-bit tests allow 1e-4
    if fault.startswith("window"):
        assert err[:19].max() < 1e-12                             # nothing has fallen out of the window before
    if fault in ("state lost", "convolution lost"):
        assert err[:60].max() < 1e-12 and err[60:].max() > 2e-3
