"""Continuous batching for hybrid decoders (``models.hybrid``): every step is ONE ragged batch of portions of prompts beside
single decoded tokens.

* ``execute`` is the step: it runs given tokens of given sequences over the cache and returns the wanted logits. When every
  sequence brings one token it replays a CUDA graph captured for the batch's size bucket (the same launches).
* ``step`` schedules: admission in FIFO order while a slot is free and the request's pages (prompt and everything it may
  generate) fit; every running request decodes one token; the rest of the step's token budget (``max_step_tokens``) goes to
  waiting prompts, which are cut where the budget ends and continue in the next step.

``open`` / ``execute`` / ``close`` also serve callers that bring their own schedule (``serving.trace``).
"""
from __future__ import annotations

import time
from typing import Dict, List, Optional, Sequence

import torch

from ..models.scheduler import EngineConfig
from ..models.sampler import Sampler
from ..models.llama import pick_next_token
from ..nn.ragged import DecodeBatch, HybridSequence
from .core import EngineCore, _Req


class HybridEngine(EngineCore):
    def __init__(self, model, cfg: Optional[EngineConfig] = None, use_cuda_graph: bool = True, temperature: float = 0.0,
                 top_p: float = 1.0, seed: int = 0, top_k: int = 0, repetition_penalty: float = 1.0, max_step_tokens: int = 8192):
        self.model = model
        self._init_core(cfg, model.config.vocab_size, model._device(), temperature, top_p, seed, top_k, repetition_penalty)
        c = self.cfg
        if c.kv_int8:
            raise ValueError("HybridEngine: keys are kept in the model's precision (kv_int8 is not available)")
        if max_step_tokens < 1:
            raise ValueError("HybridEngine: max_step_tokens must be positive")
        self.max_step_tokens = max_step_tokens
        self.cache = model.make_cache(c.num_blocks, c.block_size, c.max_batch_size, self.max_blocks * c.block_size)
        self.allocator = self.cache.allocator
        self.on_gpu = self.device.type == "cuda"
        self.use_cuda_graph = use_cuda_graph and self.on_gpu
        self._graphs: Dict[int, dict] = {}
        self._promised = 0          # pages that admitted requests may still take

    # ------------------------------------------------------------------ the step
    def open(self) -> HybridSequence:
        return HybridSequence(self.cache)

    def close(self, seq: HybridSequence) -> None:
        seq.reset()

    @torch.no_grad()
    def execute(self, entries: Sequence, want: Sequence, keep: bool = True) -> Optional[torch.Tensor]:
        """entries: (sequence, token ids) with each sequence at most once; want[i]: places among entry i's tokens. Returns fp32
        logits [wanted, vocab] on the device in the order of the entries and of their wanted places, or None. ``keep=False``
        may return a buffer that the next step overwrites."""
        V = self.vocab_size
        if any(len(t) and (min(t) < 0 or max(t) >= V) for _, t in entries):
            raise ValueError("execute: token id outside [0, vocab_size)")
        if not entries:
            return None
        # a position's place in a captured launch is bounded by the tables, so every sequence of the engine fits a graph
        if self.use_cuda_graph and len(entries) <= self.BUCKETS[-1] and all(len(t) == 1 for _, t in entries):
            seqs = [s for s, _ in entries]
            if len(set(map(id, seqs))) != len(seqs):
                raise ValueError("execute: a sequence appears twice")
            logits = self._execute_captured(seqs, [t[0] for _, t in entries])
            rows = [i for i, w in enumerate(want) for _ in w]
            if not rows:
                return None
            if rows != list(range(len(entries))):
                return logits[rows]
            return logits[:len(entries)].clone() if keep else logits[:len(entries)]
        batch = self.model.make_batch(self.cache, entries, want)
        logits = self.model.forward_ragged(batch, self.cache)
        batch.commit()
        return logits

    def _execute_captured(self, seqs, tokens) -> torch.Tensor:
        bs, done = self.cfg.block_size, []
        try:
            for s in seqs:
                if s.slot < 0 or s.length >= len(s.blocks) * bs:      # (most tokens land in a page the sequence has)
                    before = (s, len(s.blocks), s.slot)
                    s.reserve(1)
                    done.append(before)
        except Exception:
            for s, nb, slot in done:               # a step that does not fit leaves no trace
                s.release_to(nb, slot)
            raise
        A = self._bucket(len(seqs))
        g = self._graphs.get(A) or self._capture(A)
        if g["copied"] is not None:
            g["copied"].synchronize()            # the host buffer is free again
        DecodeBatch.fill(g["host_np"], self.cache, seqs, tokens)
        g["inp"].copy_(g["host"], non_blocking=True)
        g["copied"] = g["copied"] or torch.cuda.Event()
        g["copied"].record()
        g["graph"].replay()
        for s in seqs:
            s.length += 1
        return g["logits"]

    def _capture(self, A: int) -> dict:
        """Captures the decode step of ``A`` rows, with padding rows only: nothing is appended and no slot is touched."""
        dev = self.device
        host = torch.zeros((A, DecodeBatch.HEAD + self.max_blocks), dtype=torch.int32).pin_memory()
        DecodeBatch.fill(host.numpy(), self.cache, [], [])
        g = {"host": host, "host_np": host.numpy(), "inp": host.to(dev), "copied": None}

        def run():
            return self.model.forward_ragged(DecodeBatch(g["inp"], self.cache.max_len).unpack(), self.cache)
        stream = torch.cuda.Stream(device=dev)
        stream.wait_stream(torch.cuda.current_stream(dev))
        with torch.cuda.stream(stream):
            for _ in range(2):                   # lazy allocations, attribute settings
                run()
        torch.cuda.current_stream(dev).wait_stream(stream)
        torch.cuda.synchronize(dev)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            g["logits"] = run()
        g["graph"] = graph
        self._graphs[A] = g
        return g

    def warm_graphs(self, max_batch: int = 0) -> int:
        """Captures the decode graph of every batch bucket up to ``max_batch`` (default: the configured maximum)."""
        if not self.use_cuda_graph:
            return 0
        top, made = self._bucket(max_batch or self.cfg.max_batch_size), 0
        for A in self.BUCKETS:
            if A <= top and A not in self._graphs:
                self._capture(A)
                made += 1
        return made

    # ------------------------------------------------------------------ requests
    def add_request(self, prompt_ids, gen=None) -> int:
        rid = super().add_request(prompt_ids, gen)
        r = self.requests[rid]
        if self._blocks_for(r.prompt_len + r.gen.max_new_tokens) > self.cfg.num_blocks:
            self.waiting.pop()
            del self.requests[rid]
            raise ValueError("add_request: the request can never fit in the KV pool")
        r.seq, r.fed = self.open(), 0
        r.sampler = Sampler(r.gen.sampling, r.gen.seed) if r.gen.do_sample else None
        return rid

    def _need(self, r: _Req) -> int:
        return self._blocks_for(r.prompt_len + r.gen.max_new_tokens)

    def _retire(self, r: _Req) -> None:
        self._promised -= self._need(r) - len(r.seq.blocks)
        self.close(r.seq)
        r.finished = True
        r.t_done = time.perf_counter()

    def _admit(self) -> List[_Req]:
        admitted = []
        while self.waiting and len(self.running) + len(admitted) < self.cfg.max_batch_size:
            head = self.waiting[0]
            if self.free_blocks() - self._promised < self._need(head):
                break
            self._promised += self._need(head)
            admitted.append(self.waiting.popleft())
        return admitted

    def _schedule(self):
        """[(request, tokens)] of the next step: one token of every request that decodes, then prompts while the budget
        lasts."""
        plan, budget = [], self.max_step_tokens
        for r in self.running:
            if r.fed == len(r.tokens) - 1 and r.fed >= r.prompt_len:
                plan.append((r, r.tokens[-1:]))
                budget -= 1
        for r in self.running:
            left = r.prompt_len - r.fed
            if left > 0 and budget > 0:
                n = min(left, budget)
                plan.append((r, r.tokens[r.fed:r.fed + n]))
                budget -= n
        return plan

    def step(self) -> bool:
        t0 = time.perf_counter()
        wd = getattr(self, "watchdog", None)
        if wd is not None:
            wd.step()
        self.running += self._admit()
        for r in [r for r in self.running if r.gen.max_new_tokens == 0]:
            self._retire(r)
        self.running = [r for r in self.running if not r.finished]
        plan = self._schedule()
        if not plan:
            return self.has_pending()
        new = sum(len(t) for _, t in plan)
        ends = [r.fed + len(t) >= r.prompt_len for r, t in plan]
        with self._range(f"step[{len(plan)} requests, {new} tokens]"):
            before = sum(len(r.seq.blocks) for r, _ in plan)
            logits = self.execute([(r.seq, t) for r, t in plan], [[len(t) - 1] if e else [] for (r, t), e in zip(plan, ends)],
                                  keep=False)
            self._promised -= sum(len(r.seq.blocks) for r, _ in plan) - before
            for r, t in plan:
                r.fed += len(t)
            picking = [r for (r, _), e in zip(plan, ends) if e]
            nxt = self._choose(logits, picking) if picking else []
        now = time.perf_counter()
        for r, t in zip(picking, nxt):
            if r.generated == 0:
                r.t_first = now
            self._emit(r, t)
        self.running = [r for r in self.running if not r.finished]
        self.steps += 1
        decoded = sum(1 for r, t in plan if len(t) == 1 and r.fed > r.prompt_len)
        s, dt = self.stats, now - t0
        s["prefill_tokens"] += new - decoded
        s["decode_tokens"] += decoded
        s["decode_steps"] += 1 if decoded == new else 0
        s["decode_s" if decoded == new else "prefill_s"] += dt      # (a mixed step counts as prompt time)
        ml = getattr(self, "metrics_logger", None)
        if ml is not None and self.steps % self.log_every == 0:
            ml.log(event="serve_progress", step=self.steps, running=len(self.running), waiting=len(self.waiting),
                   decode_tokens=s["decode_tokens"], prefill_tokens=s["prefill_tokens"])
        return self.has_pending()

    def _choose(self, logits: torch.Tensor, reqs: List[_Req]) -> List[int]:
        """Next token per row: the request's own host sampler if it asks for one, else the engine's device sampler."""
        if not self.on_gpu or any(r.sampler is not None for r in reqs):
            if not self.on_gpu and not self.greedy:
                raise ValueError("HybridEngine: on the CPU, sampling is per request (GenerateConfig.do_sample)")
            picked = self._pick(logits.clone(), reqs).cpu().tolist() if self.on_gpu else [None] * len(reqs)
            return [p if r.sampler is None and p is not None else pick_next_token(logits[i], r.sampler, r.tokens)
                    for i, (p, r) in enumerate(zip(picked, reqs))]
        return [int(t) for t in self._pick(logits, reqs).cpu().tolist()]
