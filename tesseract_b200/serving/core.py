"""What every device-resident serving engine shares: the request queue, KV-block and slot bookkeeping, choosing tokens on
the device, instrumentation and metrics. An engine adds the step itself (``step``: admit, run the model, emit)."""
from __future__ import annotations

import time
from collections import deque

import numpy as np
from dataclasses import dataclass, field
from typing import Deque, Dict, List, Optional

import torch

from .. import _native
from .._native import check, lib, stream_ptr
from ..models.llama import GenerateConfig
from ..models.scheduler import EngineConfig
from ..nn.kv_cache import BlockAllocator

P, I, L, F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({
    "tsb_argmax_rows": [P, P, I, I, L, I, P],
    "tsb_argmax_rows_pack": [P, P, I, I, L, I, I, P],
    "tsb_argmax_rows_unpack": [P, P, I, I, I, P],
    "tsb_sample_top_p_rows": [P, P, I, I, L, F, F, _native.ctypes.c_ulonglong, _native.ctypes.c_ulonglong, I, P],
    "tsb_sample_rows": [P, P, I, I, L, F, I, F, _native.ctypes.c_ulonglong, _native.ctypes.c_ulonglong, P, I, P],
    "tsb_repetition_penalty_rows": [P, I, I, L, P, L, P, F, I, P],
})


@dataclass
class _Req:
    id: int
    gen: GenerateConfig
    tokens: List[int]
    prompt_len: int
    generated: int = 0
    finished: bool = False
    blocks: List[int] = field(default_factory=list)
    slot: int = -1                 # row of the engine's host-side state arrays while the request holds KV blocks
    t_submit: float = 0.0
    t_first: float = 0.0
    t_done: float = 0.0
    # engines whose steps cut prompts: the sequence's share of the cache, tokens fed so far, host sampler
    seq: object = None
    fed: int = 0
    sampler: object = None


def argmax_rows(logits: torch.Tensor) -> torch.Tensor:
    out = torch.empty(logits.shape[0], dtype=torch.int32, device=logits.device)
    check(lib().tsb_argmax_rows(logits.data_ptr(), out.data_ptr(), logits.shape[0], logits.shape[1], logits.stride(0),
                                _native.dtype_code(logits.dtype), stream_ptr(logits.device)), "tsb_argmax_rows")
    return out


def sample_rows(logits: torch.Tensor, temperature: float, top_k: int, top_p: float, seed: int, step: int = 0,
                step_counter: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Temperature -> top-k (0 = off) -> top-p -> one draw per row, on the device. With ``step_counter`` (an int64
    device tensor of one element) the step is read from it when the kernel runs, so the launch can be captured in a
    CUDA graph; the caller advances the counter."""
    out = torch.empty(logits.shape[0], dtype=torch.int32, device=logits.device)
    check(lib().tsb_sample_rows(logits.data_ptr(), out.data_ptr(), logits.shape[0], logits.shape[1], logits.stride(0),
                                float(temperature), int(top_k), float(top_p), seed, step,
                                step_counter.data_ptr() if step_counter is not None else None,
                                _native.dtype_code(logits.dtype), stream_ptr(logits.device)), "tsb_sample_rows")
    return out


def repetition_penalty_rows_(logits: torch.Tensor, history: torch.Tensor, hist_len: torch.Tensor, penalty: float) -> None:
    """In place: every occurrence of a token in ``history[row, :hist_len[row]]`` (int32) divides its positive logit
    by ``penalty`` or multiplies its non-positive logit by it (src/models/Sampler.cpp:29-50)."""
    check(lib().tsb_repetition_penalty_rows(logits.data_ptr(), logits.shape[0], logits.shape[1], logits.stride(0),
                                            history.data_ptr(), history.stride(0), hist_len.data_ptr(), float(penalty),
                                            _native.dtype_code(logits.dtype), stream_ptr(logits.device)),
          "tsb_repetition_penalty_rows")


def sample_top_p_rows(logits: torch.Tensor, temperature: float, top_p: float, seed: int, step: int) -> torch.Tensor:
    out = torch.empty(logits.shape[0], dtype=torch.int32, device=logits.device)
    check(lib().tsb_sample_top_p_rows(logits.data_ptr(), out.data_ptr(), logits.shape[0], logits.shape[1],
                                      logits.stride(0), float(temperature), float(top_p), seed, step,
                                      _native.dtype_code(logits.dtype), stream_ptr(logits.device)),
          "tsb_sample_top_p_rows")
    return out


class EngineCore:
    BUCKETS = (1, 2, 4, 8, 16, 32, 64, 128, 256, 512)

    def _init_core(self, cfg: Optional[EngineConfig], vocab_size: int, device, temperature: float, top_p: float, seed: int,
                   top_k: int, repetition_penalty: float) -> None:
        self.cfg = c = cfg or EngineConfig()
        self.vocab_size, self.device = vocab_size, device
        self.temperature, self.top_p, self.seed = temperature, top_p, seed
        self.top_k, self.repetition_penalty = int(top_k), float(repetition_penalty)
        self.greedy = temperature <= 1e-6
        self.allocator = BlockAllocator(c.num_blocks)
        self.max_blocks = (c.max_seq_len + c.block_size - 1) // c.block_size
        self._step_dev = torch.zeros(1, dtype=torch.int64, device=device)   # sampling step counter (graph-safe)
        self.waiting: Deque[_Req] = deque()
        self.running: List[_Req] = []
        self.requests: Dict[int, _Req] = {}
        self._next_id = 0
        self.steps = 0
        # Host-side state of the resident requests as arrays indexed by a stable slot (block table, block count, last
        # token, length): a decode step packs its inputs with a few gathers instead of a Python loop over requests.
        cap = c.max_batch_size
        self._tab = np.zeros((cap, self.max_blocks), dtype=np.int32)
        self._nblk = np.zeros(cap, dtype=np.int32)
        self._last = np.zeros(cap, dtype=np.int32)
        self._len = np.zeros(cap, dtype=np.int32)
        self._free_slots = list(range(cap - 1, -1, -1))
        self.stats = {"prefill_tokens": 0, "decode_tokens": 0, "prefill_s": 0.0, "decode_s": 0.0, "decode_gpu_s": 0.0,
                      "decode_steps": 0}

    # ------------------------------------------------------------------ requests
    def add_request(self, prompt_ids, gen: Optional[GenerateConfig] = None) -> int:
        gen = gen or GenerateConfig()
        prompt = [int(t) for t in prompt_ids]
        if not prompt:
            raise ValueError("add_request: empty prompt")
        V = self.vocab_size
        if any(t < 0 or t >= V for t in prompt):
            raise ValueError("add_request: prompt id outside [0, vocab_size)")
        if gen.max_new_tokens < 0 or len(prompt) + gen.max_new_tokens > self.cfg.max_seq_len:
            raise ValueError("add_request: prompt + max_new_tokens exceeds max_seq_len")
        r = _Req(self._next_id, gen, prompt, len(prompt), t_submit=time.perf_counter())
        self._next_id += 1
        self.waiting.append(r)
        self.requests[r.id] = r
        return r.id

    def has_pending(self) -> bool:
        return bool(self.waiting) or bool(self.running)

    def num_running(self) -> int:
        return len(self.running)

    def num_waiting(self) -> int:
        return len(self.waiting)

    def free_blocks(self) -> int:
        return self.allocator.num_free()

    def allocated_blocks(self) -> int:
        return self.allocator.num_used()

    def is_finished(self, rid: int) -> bool:
        return self.requests[rid].finished

    def result(self, rid: int) -> List[int]:
        r = self.requests[rid]
        if not r.finished:
            raise KeyError(f"request {rid} is not finished")
        return list(r.tokens)

    def _blocks_for(self, n: int) -> int:
        return (n + self.cfg.block_size - 1) // self.cfg.block_size

    def _grow(self, r: _Req, new_len: int) -> None:
        if r.slot < 0:
            r.slot = self._free_slots.pop()
            self._tab[r.slot] = 0
            self._nblk[r.slot] = 0
        while len(r.blocks) < self._blocks_for(new_len):
            b = self.allocator.allocate()
            self._tab[r.slot, len(r.blocks)] = b
            r.blocks.append(b)
        self._nblk[r.slot] = len(r.blocks)

    def _retire(self, r: _Req) -> None:
        for b in r.blocks:
            self.allocator.free(b)
        r.blocks = []
        if r.slot >= 0:
            self._free_slots.append(r.slot)
            r.slot = -1
        r.finished = True
        r.t_done = time.perf_counter()

    # ------------------------------------------------------------------ choosing tokens
    def _pick(self, logits: torch.Tensor, reqs: Optional[List[_Req]] = None) -> torch.Tensor:
        """Next token per row, on the device. Greedy: arg-max. Otherwise the device sampler; its step comes from a
        device counter that is advanced right after, so the pair can sit in a captured graph."""
        if self.repetition_penalty != 1.0 and reqs is not None:
            n = len(reqs)
            width = max(len(r.tokens) for r in reqs)
            hist = torch.zeros((logits.shape[0], width), dtype=torch.int32)
            lens = torch.zeros(logits.shape[0], dtype=torch.int32)
            for i, r in enumerate(reqs):
                hist[i, :len(r.tokens)] = torch.tensor(r.tokens, dtype=torch.int32)
                lens[i] = len(r.tokens)
            repetition_penalty_rows_(logits, hist.to(logits.device), lens.to(logits.device), self.repetition_penalty)
        if self.greedy:
            return argmax_rows(logits)
        out = sample_rows(logits, self.temperature, self.top_k, self.top_p, self.seed, step_counter=self._step_dev)
        self._step_dev.add_(1)
        return out

    def _emit(self, r: _Req, tok: int) -> None:
        if r.gen.max_new_tokens == 0:
            self._retire(r)
            return
        r.tokens.append(tok)
        r.generated += 1
        if r.slot >= 0:
            self._last[r.slot] = tok
            self._len[r.slot] = len(r.tokens)
        if (r.gen.eos_token_id >= 0 and tok == r.gen.eos_token_id) or r.generated >= r.gen.max_new_tokens:
            self._retire(r)

    def _bucket(self, n: int) -> int:
        for b in self.BUCKETS:
            if b >= n:
                return b
        return n

    def instrument(self, metrics=None, watchdog=None, nvtx_ranges: Optional[bool] = None) -> "ServingEngine":
        """Attach a ``utils.metrics.MetricsLogger`` (``run`` writes one summary record; every ``log_every`` steps a
        progress record), a ``utils.watchdog.RankWatchdog`` (tensor-parallel serving: every step beats and checks the
        peers on the host before it launches a collective) and / or NVTX ranges around prefill and decode (default:
        the ``TESSERACT_NVTX`` environment variable)."""
        import os
        if metrics is not None:
            self.metrics_logger = metrics
        if watchdog is not None:
            self.watchdog = watchdog
        self.nvtx = bool(nvtx_ranges) if nvtx_ranges is not None else os.environ.get("TESSERACT_NVTX", "0") == "1"
        return self

    def _range(self, name: str):
        import contextlib
        if not getattr(self, "nvtx", False):
            return contextlib.nullcontext()
        from ..utils import nvtx
        return nvtx.range_(name)

    log_every = 100

    def run(self) -> None:
        try:
            while self.has_pending():
                self.step()
        except Exception as e:
            wd = getattr(self, "watchdog", None)
            if wd is not None:
                wd.report_failure(f"{type(e).__name__}: {e}")
            raise
        ml = getattr(self, "metrics_logger", None)
        if ml is not None:
            ml.log(event="serve_summary", **self.metrics())

    # ------------------------------------------------------------------ metrics
    def metrics(self) -> dict:
        done = [r for r in self.requests.values() if r.finished and r.t_first > 0]
        ttft = sorted((r.t_first - r.t_submit) * 1e3 for r in done)
        s = self.stats
        return {
            "requests": len(done),
            "prefill_tok_s": s["prefill_tokens"] / s["prefill_s"] if s["prefill_s"] > 0 else 0.0,
            "decode_tok_s": s["decode_tokens"] / s["decode_s"] if s["decode_s"] > 0 else 0.0,
            "ttft_p50_ms": ttft[len(ttft) // 2] if ttft else 0.0,
            "steps": self.steps,
            # wall time of a decode step against the device time of its captured graph: the difference is host work
            "decode_ms_per_step": 1e3 * s["decode_s"] / max(1, s["decode_steps"]),
            "decode_gpu_ms_per_step": 1e3 * s["decode_gpu_s"] / max(1, s["decode_steps"]),
        }
