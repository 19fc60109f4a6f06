"""The package's engine serving its integer model: an int8 Qwen3 checkpoint under Hugging Face key names through the model
registry, the weight merge, the page allocator, the scheduler (prompt portions, continuous batching) and CUDA-graph decode;
token ids must be the oracle's, whatever the batching."""
from __future__ import annotations

import numpy as np
import pytest

from mini_sgl_integer_b200.engine import Engine, SamplingParams, Scheduler
from oracle import attention as oattn
from oracle import model as omodel
from tests.test_gpu_engine_reference import HK, HQ, L, VOCAB, _write_model

pytestmark = pytest.mark.gpu
NEW = 5


def _oracle(host, cache, prompt):
    n = len(prompt)
    pages = -(-(n + NEW) // 16)
    table = np.arange(pages, dtype=np.int32)
    pools = [oattn.PagedKV(pages, HK, 128) for _ in range(L)]
    loc = lambda a, b: np.arange(a, b, dtype=np.int32)
    tok, _ = omodel.greedy(np.asarray(prompt, dtype=np.int32), host, cache, pools, loc(0, n), loc(0, n), [table], [n], [n], HQ, HK, np.array([n - 1]))
    out = [int(tok[0])]
    for k in range(NEW - 1):
        tok, _ = omodel.greedy(tok, host, cache, pools, loc(n + k, n + k + 1), loc(n + k, n + k + 1), [table], [n + k + 1], [1], HQ, HK, None)
        out.append(int(tok[0]))
    return out


@pytest.fixture(scope="module")
def case(tmp_path_factory):
    d = tmp_path_factory.mktemp("qwen3")
    rng = np.random.default_rng(23)
    host = _write_model(str(d), rng)
    return str(d), host, [rng.integers(0, VOCAB, n).tolist() for n in (5, 33, 17, 1, 48)]


@pytest.mark.parametrize("graphs", [True, False])
def test_integer_model_through_the_scheduler(case, graphs):
    path, host, prompts = case
    e = Engine(path, max_tokens=192, max_reqs=3, max_len=64, cuda_graphs=graphs)
    cache = e.model.model.layers.op_list[0].self_attn.attn.rotary.cache_q15(e.device).cpu().numpy()
    got = Scheduler(e, prefill_budget=24).generate(prompts, SamplingParams(NEW))
    assert got == [_oracle(host, cache, p) for p in prompts]
    assert e.manager.free_slots == 3 and e.manager.free_pages == e.manager.num_pages


def test_only_the_integer_form_exists(case):
    with pytest.raises(TypeError):
        Engine(case[0], dtype="float32")
