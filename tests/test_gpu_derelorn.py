"""The Derelorn model through the framework's engine, scheduler and programs, against the plain whole-sequence oracle."""
from __future__ import annotations

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from mini_sgl_integer_b200.engine import Engine, SamplingParams, Scheduler
from mini_sgl_integer_b200.kvcache.manager import OutOfPages
from oracle import derelorn as D
from tests.derelorn_util import CONFIGS, attention_window, float_weights, logit_error, make_weights, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_cache: dict = {}


def weights_of(name):
    if name not in _cache:
        sd = make_weights(CONFIGS[name], 11)
        _cache[name] = (sd, float_weights(sd))
    return _cache[name]


def engine(name, dtype, **kw):
    kw = {"max_tokens": 2048, "max_reqs": 6, **kw}
    return Engine(config=CONFIGS[name], weights=dict(weights_of(name)[0]), dtype=dtype, **kw)


def oracle(name, ids):
    key = (name, tuple(map(int, ids)))
    if key not in _cache:
        _cache[key] = D.forward(ids, CONFIGS[name], weights_of(name)[1])
    return _cache[key]


def limits(name, ids, want, dtype):
    """Allowed error per position: a few times what rounding alone does there in the oracle (positions differ: a read-out
    whose k . q nearly cancels, or attention weights near a tie, pass more of it on), but at least 1e-4 and 0.03.  Rounding is
    noise of an ulp of 32-bit, or half an ulp of bf16, on every weight, and for 32-bit also the oracle in 32-bit."""
    key = (dtype, name, tuple(map(int, ids)))
    if key not in _cache:
        ulp, times, least = (2.0 ** -23, 6, 1e-4) if dtype == "float32" else (2.0 ** -8, 4, 0.03)
        noise = logit_error(D.forward(ids, CONFIGS[name], weights_of(name)[1], np.float32), want)
        for seed in range(2):
            rng = np.random.default_rng(seed)
            w = {k: v * (1 + rng.uniform(-ulp, ulp, v.shape)) for k, v in weights_of(name)[1].items()}
            noise = np.maximum(noise, logit_error(D.forward(ids, CONFIGS[name], w), want))
        _cache[key] = np.maximum(times * noise, least)
    return _cache[key]


def check(got, want, limit):
    got = got.float().cpu().numpy() if isinstance(got, torch.Tensor) else got
    assert got.shape == want.shape and np.isfinite(got).all()
    over = logit_error(got, want) / limit
    assert over.max() <= 1, (int(over.argmax()), over.max())


def feed(e, req, ids, cuts):
    """Logits of every token, the tokens cut at ``cuts``."""
    out = []
    for lo, hi in zip([0] + cuts, cuts + [len(ids)]):
        out.append(e.step([req], [list(map(int, ids[lo:hi]))], [list(range(hi - lo))]))
    return torch.cat(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_portions_and_decoding(name, dtype):
    ids = np.random.default_rng(len(name)).integers(0, CONFIGS[name]["vocab"], 130)
    want = oracle(name, ids)
    limit = limits(name, ids, want, dtype)
    e = engine(name, dtype)
    for cuts in ([], [129], [2, 4, 9, 25, 26, 58, 90, 128], [17, 18, 19, 35, 36, 37, 38, 72, 73, 90, 107, 120], list(range(90, 130)), [1, 2, 3, 100]):
        r = e.open()
        check(feed(e, r, ids, cuts), want, limit)
        e.close(r)
    e.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd sizes", "loop over everything"])
def test_decoding_from_the_first_token(name, dtype):
    ids = np.random.default_rng(5).integers(0, CONFIGS[name]["vocab"], 80)
    e = engine(name, dtype)
    want = oracle(name, ids)
    check(feed(e, e.open(), ids, list(range(1, 80))), want, limits(name, ids, want, dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompt(dtype):
    """Enough tokens per forward for the large linears and for several token blocks of the preparation."""
    name = "mixed"
    ids = np.random.default_rng(13).integers(0, CONFIGS[name]["vocab"], 640)
    want = oracle(name, ids)
    limit = limits(name, ids, want, dtype)
    e = engine(name, dtype)
    for c in ([], [300, 302, 639], [129, 257, 513]):
        r = e.open()
        check(feed(e, r, ids, c), want, limit)
        e.close(r)


@pytest.mark.parametrize("graphs", [True, False])
def test_long_decoding_holds_no_more_pages_than_the_window(graphs):
    name, ids = "mixed", np.random.default_rng(6).integers(0, 123, 400)
    e = engine(name, "float32", cuda_graphs=graphs, max_tokens=432, max_reqs=1)
    r = e.open()
    got = [feed(e, r, ids[:30], [])]
    most = 0
    for k in range(30, 400):
        got.append(e.step([r], [[int(ids[k])]]))
        most = max(most, e.manager.num_pages - e.manager.free_pages)
    want = oracle(name, ids)
    check(torch.cat(got), want, limits(name, ids, want, "float32"))
    assert most <= attention_window(CONFIGS[name]) // 16 + 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "loop over everything", "wide heads"])
def test_batches_of_unequal_requests_and_reused_slots(name, dtype):
    """Requests of different lengths run together in every mixture of prompts, portions and single tokens, come and go,
    and take over pages and slots of others; each must get what it gets alone."""
    rng = np.random.default_rng(7)
    V = CONFIGS[name]["vocab"]
    e = engine(name, dtype, max_reqs=4, max_tokens=1024)
    todo = [rng.integers(0, V, n) for n in (1, 40, 97, 2, 130, 18, 64, 33, 5, 110)]
    want = [oracle(name, ids) for ids in todo]
    live, got, k = {}, [[] for _ in todo], 0
    while k < len(todo) or live:
        while k < len(todo) and len(live) < 4:
            live[k] = [e.open(), 0]
            k += 1
        who = [j for j in live if rng.random() < 0.8] or list(live)
        single = rng.random() < 0.4
        part = {j: 1 if single or rng.random() < 0.2 else int(rng.integers(1, 50)) for j in who}
        toks = [list(map(int, todo[j][live[j][1]:live[j][1] + part[j]])) for j in who]
        logits = e.step([live[j][0] for j in who], toks, [list(range(len(t))) for t in toks])
        at = 0
        for j, t in zip(who, toks):
            got[j].append(logits[at:at + len(t)])
            at += len(t)
            live[j][1] += len(t)
            if live[j][1] == len(todo[j]):
                e.close(live.pop(j)[0])
    for j in range(len(todo)):
        check(torch.cat(got[j]), want[j], limits(name, todo[j], want[j], dtype))
    assert e.manager.free_pages == e.manager.num_pages and e.manager.free_slots == 4


def test_wanted_places_and_long_inputs_in_portions():
    name, ids = "mixed", np.random.default_rng(8).integers(0, 123, 200)
    want = oracle(name, ids)
    limit = limits(name, ids, want, "float32")
    e = engine(name, "float32", max_portion=64)
    a, b = e.open(), e.open()
    places = [0, 1, 63, 64, 65, 128, 199]
    check(e.step([a], [ids.tolist()], [places]), want[places], limit[places])
    got = e.step([b, a], [ids[:90].tolist(), [3]], [[89, 7], []])
    check(got, want[[89, 7]], limit[[89, 7]])
    assert e.step([b], [[int(ids[90])]], [[]]) is None
    check(e.step([b], [[int(ids[91])]]), want[91:92], limit[91:92])
    with pytest.raises(ValueError):
        e.step([b], [[123]])
    check(e.step([b], [[int(ids[92])]]), want[92:93], limit[92:93])   # a refused step left no trace


def test_running_out_of_pages_leaves_the_request_usable():
    name = "loop over everything"                               # its window is one key, so pages come back at once
    e = engine(name, "float32", max_tokens=64, max_reqs=2, max_len=64)
    a, b = e.open(), e.open()
    ids = np.random.default_rng(9).integers(0, 64, 64)
    for k in range(0, 64, 8):
        e.step([a], [ids[k:k + 8].tolist()])
    want = oracle(name, ids)
    check(e.step([b], [ids[:60].tolist()]), want[59:60], 1e-4)
    with pytest.raises(ValueError):
        e.step([b], [ids[:5].tolist()])                         # beyond max_len
    check(e.step([b], [ids[60:62].tolist()]), want[61:62], 1e-4)
    e = engine("wide heads", "float32", max_tokens=64, max_reqs=2, max_len=64)
    a, b = e.open(), e.open()
    ids = ids % 70
    e.step([a], [ids[:48].tolist()])
    with pytest.raises(OutOfPages):
        e.step([b], [ids[:60].tolist()])
    e.close(a)
    check(e.step([b], [ids[:60].tolist()]), oracle("wide heads", ids)[59:60], 1e-4)


def test_stream_after_every_run():
    """The residual stream that leaves every run of a layer, passes of the loop counted each."""
    from mini_sgl_integer_b200.attention.hybrid_backend import HybridMetadata
    name, ids = "mixed", np.random.default_rng(14).integers(0, 123, 45)
    want = []
    D.forward(ids, CONFIGS[name], weights_of(name)[1], trace=want)
    e = engine(name, "float32")
    r, n = e.open(), len(ids)
    e.manager.extend(r.table_idx, 0, n)
    e.manager.sync()
    i32 = lambda a: torch.as_tensor(np.asarray(a, dtype=np.int32)).cuda()
    loc = e.manager.locations(torch.full((n,), r.table_idx), torch.arange(n)).to(torch.int32).cuda()
    md = HybridMetadata(i32(range(n)), loc, e.manager.page_table[r.table_idx:r.table_idx + 1], i32([n]), i32([r.table_idx]), i32([0, n]), i32([0] * n), n, n)
    got = []
    logits = e.model.forward_tokens(i32(ids), md, e.cache, trace=got)
    assert len(got) == len(want) == 8
    for a, b in zip(got, want):
        assert np.abs(a.cpu().numpy() - b).max() < 1e-3 * b.std()
    want = oracle(name, ids)
    check(logits, want, limits(name, ids, want, "float32"))


# ----------------------------------------------------------------------------- generation
def oracle_greedy(name, prompt, n):
    ids = list(map(int, prompt))
    for _ in range(n):
        ids.append(int(np.argmax(D.forward(ids, CONFIGS[name], weights_of(name)[1])[-1])))
    return ids[len(prompt):]


@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation_through_the_scheduler(graphs):
    name, rng = "mixed", np.random.default_rng(10)
    prompts = [rng.integers(0, 123, n).tolist() for n in (3, 50, 1, 21, 80, 7)]
    if "greedy" not in _cache:
        _cache["greedy"] = [oracle_greedy(name, p, 8) for p in prompts]
    want = _cache["greedy"]
    e = engine(name, "float32", max_reqs=3, max_tokens=320, cuda_graphs=graphs)
    assert Scheduler(e, prefill_budget=32).generate(prompts, SamplingParams(8)) == want
    assert e.manager.free_slots == 3 and e.manager.free_pages == e.manager.num_pages
    stop = want[1][4]
    out = Scheduler(e).generate([prompts[1]], SamplingParams(8, stop_ids=(stop,)))[0]
    assert out == want[1][:want[1].index(stop) + 1]


@pytest.fixture(scope="module")
def model_dir(tmp_path_factory):
    d = tmp_path_factory.mktemp("derelorn")
    write_model(str(d), CONFIGS["odd sizes"], weights_of("odd sizes")[0])
    return str(d)


def test_command_line(model_dir):
    prompts = [[5, 17, 3], [9] * 30]
    r = subprocess.run([sys.executable, "-m", "mini_sgl_integer_b200", "--model", model_dir, "--dtype", "float32", "--max-new-tokens", "6",
                        "--max-tokens", "256", "--max-running", "2"], input="\n".join(map(json.dumps, prompts)), text=True, cwd=ROOT, capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(x) for x in r.stdout.splitlines()]
    assert [x["prompt"] for x in lines] == prompts
    assert [x["output"] for x in lines] == [oracle_greedy("odd sizes", p, 6) for p in prompts]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(model_dir, tmp_path, dtype):
    rng = np.random.default_rng(12)
    a, b = rng.integers(0, 57, 60), rng.integers(0, 57, 23)
    wa, wb = oracle("odd sizes", a), oracle("odd sizes", b)
    la, lb = limits("odd sizes", a, wa, dtype), limits("odd sizes", b, wb, dtype)
    limit = {0: la[[0, 32]], 2: la[35:36], 3: lb[[22, 3]], 4: la[59:60], 5: lb[1:2]}
    steps = [([("a", a[:33], [0, 32])], [], wa[[0, 32]]), ([("a", a[33:35], [])], [], None), ([("a", a[35:36], [0])], [], wa[35:36]),
             ([("b", b, [22, 3])], ["b"], wb[[22, 3]]), ([("a", a[36:], [23])], ["a"], wa[59:60]), ([("b", b[:2], [1])], ["b"], wb[1:2])]
    lines = [json.dumps({"step": i, "entries": [{"id": k, "tokens": t.tolist(), "want": w} for k, t, w in s[0]], "end": s[1]}) for i, s in enumerate(steps)]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", model_dir, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "96"],
                       input="\n".join(lines) + "\n", text=True, cwd=str(tmp_path), capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    for i, (_, _, want) in enumerate(steps):
        path = tmp_path / f"{i}.f32"
        assert path.exists() == (want is not None)
        if want is not None:
            check(np.fromfile(path, "<f4").reshape(want.shape), want, limit[i])
