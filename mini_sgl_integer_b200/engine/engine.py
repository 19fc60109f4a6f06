"""The engine: one model on one GPU, its cache, and the step function that runs a batch (engine/engine.py:34-222).

``open`` a request, ``step`` some of its tokens (a whole prompt, a portion of it, one decoded token, several requests
together), ``close`` it.  A step runs the model inside the global context as its layers expect; a step of one token per
request is replayed from a CUDA graph captured per batch size (engine/graph.py:49-158).
"""
from __future__ import annotations

import gc
from typing import Any, Dict, List, Optional, Sequence

import torch

from ..attention import create_attention_backend
from ..core import Batch, Context, Req, set_global_ctx
from ..kvcache.manager import PAGE_SIZE, CacheManager
from ..models.registry import SUPPORTED_MODELS
from ..models.weight import architecture_of, load_checkpoint, load_config_dict

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class Engine:
    def __init__(self, model_dir: Optional[str] = None, *, config: Optional[Dict[str, Any]] = None,
                 weights: Optional[Dict[str, torch.Tensor]] = None, dtype: str | torch.dtype = "bfloat16", max_tokens: int = 65536,
                 max_reqs: int = 64, max_len: Optional[int] = None, max_portion: int = 4096, device: str = "cuda:0",
                 cuda_graphs: bool = True):
        """``model_dir``: a folder with config.json and safetensors; or ``config`` (the dict) and ``weights`` (host or
        device tensors, consumed).  ``max_tokens``: tokens that open requests hold together; ``max_len``: of one request;
        ``max_portion``: most tokens per forward."""
        if model_dir is not None:
            config, weights = load_config_dict(model_dir), load_checkpoint(model_dir)
        if config is None or weights is None:
            raise ValueError("pass model_dir, or config and weights")
        self.entry = SUPPORTED_MODELS[architecture_of(config)]()
        self.config = self.entry.parse_config(config)
        self.dtype = DTYPES[dtype] if isinstance(dtype, str) else dtype
        if self.dtype not in self.entry.dtypes:
            raise TypeError(f"{architecture_of(config)} runs in {[str(d) for d in self.entry.dtypes]}, not {self.dtype}")
        self.device = torch.device(device)
        torch.cuda.set_device(self.device)
        self.max_reqs, self.max_portion = max_reqs, max_portion
        self.max_len = min(max_len or max_tokens, max_tokens)
        self.vocab_size = self.entry.vocab_size(self.config)
        num_pages = -(-max_tokens // PAGE_SIZE) + max_reqs                  # every request may leave its last page partly empty
        self.model = self.entry.create(self.config, weights, self.dtype, self.device, self.max_len)
        self.cache = self.entry.create_cache(self.config, num_pages, max_reqs, self.dtype, self.device)
        self.manager = CacheManager(num_pages, max_reqs, self.max_len, self.entry.window(self.config), self.device,
                                    spare_page=self.cache.spare_page, pages_needed=self.entry.needs_pages(self.config))
        self.backend = create_attention_backend(self.entry.backend, self.config, self.cache)
        self.ctx = Context(page_size=PAGE_SIZE, page_table=self.manager.page_table, attn_backend=self.backend)
        self._graphs: Optional[GraphRunner] = GraphRunner(self) if cuda_graphs else None

    # ------------------------------------------------------------------ requests
    def open(self) -> Req:
        return Req(table_idx=self.manager.allocate(), cached_len=0, device_len=0)

    def close(self, req: Req) -> None:
        self.manager.free(req.table_idx)

    # ------------------------------------------------------------------ steps
    def step(self, reqs: Sequence[Req], tokens: Sequence[Sequence[int]], want: Optional[Sequence[Sequence[int]]] = None) -> Optional[torch.Tensor]:
        """Runs ``tokens[i]`` as the next tokens of ``reqs[i]`` and returns logits [rows, vocab]: of each request's last
        token, or of the places ``want[i]`` among its tokens (None when nothing is wanted).  Longer inputs than
        ``max_portion`` are run in portions."""
        counts = [len(t) for t in tokens]
        if not reqs or len(counts) != len(reqs) or min(counts) < 1:
            raise ValueError("a step needs at least one token for every request")
        for t in tokens:
            if min(t) < 0 or max(t) >= self.vocab_size:
                raise ValueError(f"token ids must lie in [0, {self.vocab_size})")
        if want is None:
            want = [[n - 1] for n in counts]
        for w, n in zip(want, counts):
            if any(not 0 <= k < n for k in w):
                raise ValueError("a wanted place lies outside the request's tokens")
        if sum(counts) <= self.max_portion:
            return self._forward(reqs, tokens, want)
        out = []
        for r, t, w in zip(reqs, tokens, want):
            rows = []
            for lo in range(0, len(t), self.max_portion):
                hi = min(len(t), lo + self.max_portion)
                here = [j for j, k in enumerate(w) if lo <= k < hi]
                logits = self._forward([r], [t[lo:hi]], [[w[j] - lo for j in here]])
                rows.extend(zip(here, logits if logits is not None else []))
            out.extend(v for _, v in sorted(rows, key=lambda jv: jv[0]))
        return torch.stack(out) if out else None

    def _forward(self, reqs, tokens, want) -> Optional[torch.Tensor]:
        done = 0
        try:
            for r, t in zip(reqs, tokens):
                self.manager.extend(r.table_idx, r.cached_len, r.cached_len + len(t))
                r.device_len = r.cached_len + len(t)
                done += 1
        except Exception:
            for r in reqs[:done]:                              # pages already taken stay with their request
                r.device_len = r.cached_len
            raise
        self.manager.sync()
        decode = all(len(t) == 1 for t in tokens)
        batch = Batch(reqs=list(reqs), phase="decode" if decode else "prefill")
        counts = torch.tensor([len(t) for t in tokens])
        first = torch.tensor([r.cached_len for r in reqs]) - counts.cumsum(0) + counts
        pos = torch.arange(int(counts.sum())) + torch.repeat_interleave(first, counts)
        loc = self.manager.locations(torch.repeat_interleave(torch.tensor([r.table_idx for r in reqs]), counts), pos)
        host = torch.stack([torch.tensor([x for t in tokens for x in t], dtype=torch.int64), pos, loc]).to(torch.int32)
        picks, base = [], 0
        for t, w in zip(tokens, want):
            picks.extend(base + k for k in w)
            base += len(t)
        set_global_ctx(self.ctx, replace=True)
        if decode and self._graphs is not None:
            logits = self._graphs.run(batch, host)
            if picks != list(range(base)):
                logits = logits[torch.tensor(picks, device=self.device)] if picks else None
        else:
            dev = host.pin_memory().to(self.device, non_blocking=True)
            batch.input_ids, batch.positions, batch.out_loc = dev[0], dev[1], dev[2]
            batch.logit_rows = torch.tensor(picks, dtype=torch.int64).to(self.device)
            self.backend.prepare_metadata(batch)
            with self.ctx.forward_batch(batch):
                logits = self.model.forward() if picks else self._forward_without_logits()
        for r in reqs:
            r.cached_len = r.device_len
            self.manager.trim(r.table_idx, r.cached_len)
        return logits

    def _forward_without_logits(self) -> None:
        if getattr(self.model, "skips_empty_logits", False):
            self.model.forward()
        else:
            self.ctx.batch.logit_rows = None
            self.model.forward()

    def check_status(self) -> None:
        self.entry.check_status()


class GraphRunner:
    """Decode steps as CUDA graphs, one per padded batch size, captured when first needed."""

    def __init__(self, engine: Engine):
        self.e = engine
        self.sizes: List[int] = [1]
        while self.sizes[-1] < engine.max_reqs:
            self.sizes.append(min(2 * self.sizes[-1], engine.max_reqs))
        n, dev = engine.max_reqs, engine.device
        spare = engine.cache.spare_page * PAGE_SIZE
        self.inputs = torch.tensor([[0], [0], [spare]], dtype=torch.int32).repeat(1, n).to(dev)     # ids | positions | out_loc
        self.graphs: Dict[int, tuple] = {}
        self.pool = None
        self.ready = False

    def _batch(self, reqs, padded) -> Batch:
        batch = Batch(reqs=list(reqs), phase="decode")
        batch.padded_reqs = list(padded)
        n = len(padded)
        batch.input_ids, batch.positions, batch.out_loc = self.inputs[0, :n], self.inputs[1, :n], self.inputs[2, :n]
        return batch

    def _spare(self) -> Req:
        return Req(table_idx=self.e.cache.spare_slot, cached_len=0, device_len=1)

    def _capture(self, n: int) -> None:
        e = self.e
        if not self.ready:
            e.backend.init_capture_graph(e.max_len, self.sizes)
            self.ready = True
        spare = [self._spare() for _ in range(n)]
        self._fill(torch.tensor([[0], [0], [e.cache.spare_page * PAGE_SIZE]], dtype=torch.int32).repeat(1, n))
        batch = self._batch(spare, spare)
        e.backend.prepare_metadata(batch)
        e.backend.prepare_for_replay(batch)                     # padding only, whatever an earlier replay left behind
        e.backend.prepare_for_capture(batch)
        side = torch.cuda.Stream(e.device)
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side), e.ctx.forward_batch(batch):
            e.model.forward()                                   # loads modules and sizes attributes outside the capture
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        collects = gc.isenabled()
        gc.disable()                                            # a graph or tensor freed by a collection would end the capture
        try:
            with torch.cuda.graph(graph, pool=self.pool), e.ctx.forward_batch(batch):
                logits = e.model.forward()
        finally:
            if collects:
                gc.enable()
        self.pool = self.pool or graph.pool()
        self.graphs[n] = (graph, logits)

    def _fill(self, host: torch.Tensor) -> None:
        self.inputs[:, :host.shape[1]].copy_(host.pin_memory(), non_blocking=True)

    def run(self, batch: Batch, host: torch.Tensor) -> torch.Tensor:
        """``host`` int32 [3, bs] ids | positions | cache rows; logits [bs, vocab]."""
        bs = batch.size
        n = next(s for s in self.sizes if s >= bs)
        if n not in self.graphs:
            self._capture(n)
        e = self.e
        pad = n - bs
        if pad:
            host = torch.cat([host, torch.tensor([[0], [0], [e.cache.spare_page * PAGE_SIZE]], dtype=torch.int32).repeat(1, pad)], dim=1)
        self._fill(host)
        padded = self._batch(batch.reqs, batch.reqs + [self._spare() for _ in range(pad)])
        e.backend.prepare_metadata(padded)
        e.backend.prepare_for_replay(padded)
        graph, logits = self.graphs[n]
        graph.replay()
        return logits[:bs].clone()
