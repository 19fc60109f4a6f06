"""Sefevik without a GPU: configuration and checkpoint reading, the page and slot allocator, the C ABI's argument checks,
and that the tests' own models would show a fault (mistakes planted in the oracle)."""
from __future__ import annotations

import copy
import ctypes
import os
import re

import numpy as np
import pytest
import torch

from mini_sgl_integer_b200 import _lib
from mini_sgl_integer_b200.kvcache.manager import CacheManager, OutOfPages
from mini_sgl_integer_b200.models import SUPPORTED_MODELS
from mini_sgl_integer_b200.models.config import SefevikConfig
from mini_sgl_integer_b200.models.weight import architecture_of, load_checkpoint, load_config_dict
from oracle import sefevik as S
from tests.sefevik_util import CONFIGS, gru, logit_error, make_weights, mla, model, numpy_weights, write_model

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ----------------------------------------------------------------------------- configuration and weights
def test_configuration_is_read_from_the_file(tmp_path):
    cfg = CONFIGS["mixed"]
    sd = make_weights(cfg, 1)
    write_model(str(tmp_path), cfg, sd)
    d = load_config_dict(str(tmp_path))
    entry = SUPPORTED_MODELS[architecture_of(d)]()
    c = entry.parse_config(d)
    assert (c.vocab_size, c.hidden_size, c.num_layers) == (131, 72, 6)
    assert c.cache_layers == (1, 4) and c.attention_layers == (1, 3, 4) and c.recurrent_layers == (0, 2, 5)
    assert c.max_window == 70 and c.layers[2].mlp is None and c.layers[3].mixer.kv_from == 1
    assert c.layers[1].mixer.rot.scaling.factor == 4.0
    back = load_checkpoint(str(tmp_path))
    assert set(back) == set(sd) and all(torch.equal(back[k], sd[k]) for k in sd)


def test_configurations_without_windows_or_attention():
    assert SefevikConfig.from_dict(CONFIGS["attention only, no bigram, full and single-token windows"]).max_window is None
    c = SefevikConfig.from_dict(CONFIGS["recurrence only"])
    assert c.max_window == 0 and not SUPPORTED_MODELS["Sefevik"]().needs_pages(c)


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][3]["mixer"].update(kv_from=4), lambda c: c["layers"][3]["mixer"].update(kv_from=0),
    lambda c: c["layers"][4]["mixer"].update(kv_from=3), lambda c: c["layers"][3]["mixer"].update(kv_rank=8),
    lambda c: c["layers"][3]["mixer"]["rot"].update(base=77.0), lambda c: c["layers"][1].update(type="other"),
    lambda c: c["layers"][1]["mlp"].update(kind="sparse"), lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
    lambda c: c.update(architecture="Other")])
def test_configurations_that_make_no_sense_are_refused(change):
    c = copy.deepcopy(CONFIGS["mixed"])
    change(c)
    with pytest.raises(ValueError):
        SefevikConfig.from_dict(c)


def test_registry_names():
    assert {"Sefevik", "Qwen3ForCausalLM"} <= set(SUPPORTED_MODELS.supported_names())
    with pytest.raises(KeyError):
        SUPPORTED_MODELS["NoSuchModel"]
    assert architecture_of({"architectures": ["Qwen3ForCausalLM"]}) == "Qwen3ForCausalLM"
    with pytest.raises(ValueError):
        architecture_of({})


def test_broken_checkpoint_is_refused(tmp_path):
    cfg = CONFIGS["one layer"]
    write_model(str(tmp_path), cfg, make_weights(cfg, 1))
    p = tmp_path / "model.safetensors"
    raw = p.read_bytes()
    p.write_bytes(raw[:-10])
    with pytest.raises(ValueError):
        load_checkpoint(str(tmp_path))
    p.write_bytes(raw[:4])
    with pytest.raises(ValueError):
        load_checkpoint(str(tmp_path))


# ----------------------------------------------------------------------------- pages and slots
def test_manager_gives_pages_back_behind_the_window():
    m = CacheManager(num_pages=8, num_slots=2, max_len=1000, window=33, device="cpu", spare_page=8)
    s = m.allocate()
    used = []
    for n in range(1, 900):
        m.extend(s, n - 1, n)
        m.sync()
        first = max(0, n - 1 - 32)                                # oldest key the new token sees
        pages = [int(m.page_table[s, k // 16]) for k in range(first, n)]
        assert len(set(pages)) == n // 16 - first // 16 + (1 if n % 16 else 0)      # no page serves two places
        used.append(m.num_pages - m.free_pages)
        m.trim(s, n)
    assert max(used) <= m.pages_for(900, 1) <= 5
    m.free(s)
    assert m.free_pages == 8 and m.free_slots == 2
    assert bool((m.page_table[2] == 8).all())


def test_manager_never_hands_a_page_out_twice():
    rng = np.random.default_rng(0)
    m = CacheManager(num_pages=40, num_slots=5, max_len=200, window=None, device="cpu", spare_page=40)
    live: dict = {}
    for _ in range(600):
        if live and (rng.random() < 0.2 or not m.free_slots):
            s = int(rng.choice(list(live)))
            m.free(s)
            del live[s]
            continue
        s = m.allocate() if m.free_slots and rng.random() < 0.3 else (int(rng.choice(list(live))) if live else m.allocate())
        n = live.setdefault(s, 0)
        k = min(int(rng.integers(1, 30)), 200 - n)
        before = m.free_pages
        try:
            m.extend(s, n, n + k)
            live[s] = n + k
        except OutOfPages:
            assert m.free_pages == before                          # all or nothing
        m.sync()
        held = [int(p) for t, n in live.items() for p in m.page_table[t, :-(-n // 16)]]
        assert len(held) == len(set(held)) and len(held) + m.free_pages == 40
    with pytest.raises(ValueError):
        s = next(iter(live))
        m.extend(s, live[s], 300)


def test_manager_without_pages():
    m = CacheManager(num_pages=1, num_slots=1, max_len=100, window=0, device="cpu", spare_page=1, pages_needed=False)
    s = m.allocate()
    m.extend(s, 0, 100)
    m.trim(s, 100)
    assert m.free_pages == 1 and m.pages_for(100, 50) == 0
    with pytest.raises(OutOfPages):
        m.allocate()


# ----------------------------------------------------------------------------- C ABI
def test_float_library_exports_its_header():
    text = open(os.path.join(ROOT, "include", "b200float.h")).read()
    names = sorted(set(re.findall(r"B200_API\s+[\w\s\*]+?\b(b200f_\w+)\s*\(", text)))
    lib = _lib.load("float")
    assert names == sorted(_lib.FLOAT_SIGNATURES) and all(hasattr(lib, n) for n in names)
    assert hasattr(lib, "b200_decode_prepare")


def test_float_entry_points_reject_bad_arguments_before_launch():
    one = ctypes.c_void_p(16)

    def code(name, *args):
        with pytest.raises(_lib.B200Error) as e:
            _lib.call(name, *args)
        return e.value.code
    gemm = lambda x=one, dtype=1, m=4, n=8, k=8, xp=8, splits=1, act=0: ("b200f_gemm", x, one, one, dtype, 1, m, n, k, 1, xp, 0, 8, 0, 8, 0, splits, 0, act, 0.0, 0.0, None)
    assert code(*gemm(x=None)) == -1
    assert code(*gemm(dtype=7)) == -4
    assert code(*gemm(n=0)) == -2
    assert code(*gemm(k=16)) == -2                                # pitch shorter than the row
    assert code(*gemm(xp=12)) == -3                               # pitch not a multiple of 8 values
    assert code(*gemm(x=ctypes.c_void_p(24))) == -3
    assert code(*gemm(splits=2, act=1)) == -4
    assert code("b200f_mingru", one, 1, 0, one, one, one, one, one, None, one, 1, 3, 2, 8, 8, None) == -2
    assert code("b200f_latent_attn", one, one, one, 4, one, None, one, one, 1, 2, 2, 1, 4, 16, 8, 16, 16, 0, 1.0, 1, None, 0, None) == -2
    assert code("b200f_latent_attn", one, one, one, 4, one, None, one, one, 1, 2, 2, 1, 4, 16, 8, 24, 16, 0, 1.0, 2, None, 0, None) == -1
    assert code("b200f_latent_prepare", one, 1, 0, 64, one, one, one, 3, 9, None, 1e-5, one, one, None, 1, 2, 2, 4, 4, 8, 8, 8, 16, 0, None) == -2
    assert code("b200f_sublayer_end", one, 0, 0, None, 1, 0, None, None, one, one, None, one, None, None, 0, 0, None, None, None, 1, 2, 8, 8, 1e-5, None) == -2
    assert code("b200f_argmax", one, 2, 8, 4, one, None) == -2


def test_float_ops_refuse_cpu_tensors():
    from mini_sgl_integer_b200.kernel import float_ops as fo
    with pytest.raises(RuntimeError, match="no CPU fallback"):
        fo.linear(torch.zeros(2, 8), torch.zeros(4, 8))
    with pytest.raises(TypeError):
        fo.dtype_code(torch.float16)


# ----------------------------------------------------------------------------- the tests' models show faults
def _probe():
    cfg = model(50, 40, [gru(48, 32), mla(4, 16, 8, 16, 24, 20, 0.9, ff=32), mla(3, 16, 8, 16, 24, 44, 0.9, kv_from=1), gru(32)])
    return cfg, numpy_weights(make_weights(cfg, 9)), np.random.default_rng(2).integers(0, 50, 90)


@pytest.mark.parametrize("fault", ["window + 1", "window - 1", "no sink", "no rotation scaling", "scaled unrotated part", "own cache", "state lost",
                                   "no bigram", "first bigram row", "candidate", "depth average", "eps", "negative xielu branch"])
def test_planted_mistakes_show(fault, monkeypatch):
    cfg, w, ids = _probe()
    want = S.forward(ids, cfg, w)
    bad, wb = copy.deepcopy(cfg), dict(w)
    if fault.startswith("window"):
        bad["layers"][2]["mixer"]["mask"]["size"] += 1 if "+" in fault else -1
    elif fault == "no sink":
        wb["l1.mix.sink"] = w["l1.mix.sink"] - 1e3
    elif fault == "no rotation scaling":
        for i in (1, 2):
            del bad["layers"][i]["mixer"]["rot"]["scaling"]
    elif fault == "scaled unrotated part":
        bad["layers"][1]["mixer"]["scale"] *= 0.1 * np.log(4.0) + 1
    elif fault == "own cache":
        del bad["layers"][2]["mixer"]["kv_from"]
        wb["l2.mix.dkv"], wb["l2.mix.dkv.norm"] = w["l1.mix.dkv"], w["l1.mix.dkv.norm"]
    elif fault == "state lost":
        scan = S.mingru_scan
        monkeypatch.setattr(S, "mingru_scan", lambda z, u: np.concatenate([scan(z[:60], u[:60]), scan(z[60:], u[60:])]))
    elif fault == "no bigram":
        del bad["embedding"]
    elif fault == "first bigram row":
        rows = S.bigram_rows
        monkeypatch.setattr(S, "bigram_rows", lambda t, *a: np.concatenate([[0], rows(t, *a)[1:]]))
    elif fault == "candidate":
        scan = S.mingru_scan
        monkeypatch.setattr(S, "mingru_scan", lambda z, u: scan(z, np.where(u >= 0, u + 0.02, u)))
    elif fault == "depth average":
        wb["l2.dwa"] = w["l2.dwa"][::-1]
    elif fault == "eps":
        bad["norm"]["eps"] = 1e-2
    else:
        monkeypatch.setattr(S, "xielu", lambda z, p, q: np.where(z > 0, S.softplus(p) * z * z, softq(q) * (np.expm1(np.minimum(z, 0)) - np.minimum(z, 0))) + z / 2)
        softq = S.softplus
    err = logit_error(S.forward(ids, bad, wb), want)
    assert err.max() > 2e-3, err.max()                            # the 32-bit tests allow 1e-4
    if fault.startswith("window"):
        assert err[:43].max() < 1e-12                             # nothing has fallen out of the window before
