"""Decoders that mix recurrent and attention layers, described by a list: every layer has a mixer and, optionally, a
feed-forward, both normed before and after; a range of layers may run several times in a row with the same weights and
separate caches ("loop"). Embedding and output share one table.

``HybridModel`` runs ragged batches (``forward_ragged``: any mix of prompt portions and decoded tokens) over a
``HybridCache``. The serving engine drives that step; ``forward_step`` / ``forward_step_batched`` give it the interface
of ``ContinuousBatchingScheduler`` and of grammar-constrained generation.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional, Union

import torch

from .. import ops
from ..nn.hybrid import ChunkedAttention, ClampedGLU, DynamicTanh, GatedDelta, pad_to
from ..nn.ragged import HybridCache, HybridSequence, RaggedBatch
from .llama import GenerateConfig, pick_next_token


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int = 0


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class GLUSpec:
    ff: int
    limit: float


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, DeltaSpec]
    mlp: Optional[GLUSpec] = None


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int


@dataclass
class HybridConfig:
    vocab_size: int
    width: int
    layers: List[LayerSpec]
    loop: Optional[LoopSpec] = None
    eps: float = 1e-5
    embedding_scale: float = 1.0
    dtype: torch.dtype = torch.bfloat16
    bos_token_id: int = -1
    eos_token_id: int = -1
    max_position_embeddings: int = 1 << 20     # no positions enter the model: a bound for caches only
    architecture: str = ""

    def __post_init__(self):
        if self.vocab_size < 1 or self.width < 1 or not self.layers:
            raise ValueError("HybridConfig: vocabulary, width and layers must not be empty")
        lp = self.loop
        if lp is not None and not (0 <= lp.start < lp.stop <= len(self.layers) and lp.times >= 1):
            raise ValueError("HybridConfig: loop must name a range of layers and run at least once")
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("HybridConfig: dtype is bfloat16 or float32")

    def runs(self):
        """[(layer, pass)] in the order they run; pass is -1 outside the loop."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, -1) for i in range(n)]
        return ([(i, -1) for i in range(lp.start)]
                + [(i, t) for t in range(lp.times) for i in range(lp.start, lp.stop)]
                + [(i, -1) for i in range(lp.stop, n)])


class _Layer:
    def __init__(self, spec: LayerSpec, c: HybridConfig, device):
        m, W, dt = spec.mixer, c.width, c.dtype
        if isinstance(m, AttentionSpec):
            self.mixer = ChunkedAttention(W, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.chunk, dt, device)
        else:
            self.mixer = GatedDelta(W, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, c.eps, dt, device)
        self.norm1, self.norm1b = DynamicTanh(W, dt, device), DynamicTanh(W, dt, device)
        self.mlp = self.norm2 = self.norm2b = None
        if spec.mlp is not None:
            self.mlp = ClampedGLU(W, spec.mlp.ff, spec.mlp.limit, dt, device)
            self.norm2, self.norm2b = DynamicTanh(W, dt, device), DynamicTanh(W, dt, device)

    def parts(self):
        out = [("norm1", self.norm1), ("norm1b", self.norm1b), ("mix.", self.mixer)]
        if self.mlp is not None:
            out += [("norm2", self.norm2), ("norm2b", self.norm2b), ("mlp.", self.mlp)]
        return out


class HybridModel:
    def __init__(self, config: HybridConfig, device=None, init_std: Optional[float] = None, seed: int = 0):
        self.config = c = config
        self.device = torch.device(device) if device is not None else torch.device("cpu")
        # one table for the embedding and the output product; its rows are padded like every matrix the GEMMs read
        self.embed = torch.zeros(c.vocab_size, pad_to(c.width), dtype=c.dtype, device=self.device)
        self.layers = [_Layer(s, c, self.device) for s in c.layers]
        self.final_norm = DynamicTanh(c.width, c.dtype, self.device)
        self.loop_step = (torch.zeros(c.loop.times, c.width, dtype=torch.float32, device=self.device)
                          if c.loop is not None else None)
        self.runs = c.runs()
        self.chunks = sorted({s.mixer.chunk for s in c.layers if isinstance(s.mixer, AttentionSpec)})
        if init_std is not None:
            self.init_weights(init_std, seed)

    # ------------------------------------------------------------------ the parts of a model the framework asks for
    def _device(self):
        return self.device

    def eval(self) -> "HybridModel":
        return self

    def parameters(self):
        yield self.embed
        if self.loop_step is not None:
            yield self.loop_step
        for _, part in self._parts():
            yield from part.tensors()

    def num_layers(self) -> int:
        return len(self.layers)

    def engine_class(self):
        from ..serving.hybrid import HybridEngine
        return HybridEngine

    # ------------------------------------------------------------------ weights
    def _parts(self):
        for i, l in enumerate(self.layers):
            for name, part in l.parts():
                yield f"l{i}.{name}", part
        yield "final.norm", self.final_norm

    def logical_shapes(self) -> Dict[str, tuple]:
        c = self.config
        out = {"embed": (c.vocab_size, c.width)}
        if c.loop is not None:
            out["loop.step"] = (c.loop.times, c.width)
        for name, part in self._parts():
            out.update({name + k: tuple(v) for k, v in part.logical_shapes().items()})
        return out

    @torch.no_grad()
    def load_tensors(self, sd: Dict[str, torch.Tensor]) -> list:
        """Packs a dict of logical tensors; returns the names in it that the model does not have."""
        c = self.config
        known = self.logical_shapes()
        for name in ("embed", "loop.step"):
            if name in known:
                if name not in sd:
                    raise KeyError(f"load: required tensor {name!r} is missing")
                if tuple(sd[name].shape) != known[name]:
                    raise ValueError(f"load: shape of {name!r} is {tuple(sd[name].shape)}, expected {known[name]}")
        self.embed[:, :c.width].copy_(sd["embed"])
        if self.loop_step is not None:
            self.loop_step.copy_(sd["loop.step"])
        for name, part in self._parts():
            try:
                part.load({k: sd[name + k] for k in part.logical_shapes() if name + k in sd})
            except (KeyError, ValueError, TypeError) as e:
                raise type(e)(f"{name}: {e.args[0]}") from None
        return [k for k in sd if k not in known]

    def state_tensors(self) -> Dict[str, torch.Tensor]:
        out = {"embed": self.embed[:, :self.config.width].contiguous()}
        if self.loop_step is not None:
            out["loop.step"] = self.loop_step.to(self.config.dtype)
        for name, part in self._parts():
            out.update({name + k: v for k, v in part.unpack().items()})
        return out

    def load_safetensors(self, path: str) -> list:
        from ..io.safetensors import SafeTensors
        with SafeTensors.open(path) as st:
            return self.load_tensors({k: st.load(k) for k in st.keys()})

    def save_safetensors(self, path: str, metadata: Optional[dict] = None) -> None:
        from ..io.safetensors import save_file
        save_file({k: v.cpu().contiguous() for k, v in self.state_tensors().items()}, path, metadata or {"format": "pt"})

    @torch.no_grad()
    def init_weights(self, std: float = 0.02, seed: int = 0) -> None:
        """N(0, std) matrices from a fixed seed; norms start as tanh(x), decays between slow and fast."""
        gen = torch.Generator(device=self.device)
        gen.manual_seed(seed)

        def draw(name, shape):
            last = name.rsplit(".", 1)[-1]
            if last == "alpha":
                return torch.tensor(1.0)
            if len(shape) == 2:
                s = 0.5 if last == "conv" else std
                return torch.randn(shape, generator=gen, device=self.device) * s
            if last == "A_log":
                return torch.rand(shape, generator=gen, device=self.device) * 2.0 - 2.0
            if last == "dt_bias":
                return torch.rand(shape, generator=gen, device=self.device) - 3.0
            if last == "b":
                return torch.zeros(shape)
            return torch.ones(shape)
        self.load_tensors({n: draw(n, s) for n, s in self.logical_shapes().items()})

    # ------------------------------------------------------------------ the step
    def make_cache(self, num_blocks: int, block_size: int, max_sequences: int, max_len: int) -> HybridCache:
        """K / V pages and recurrent slots of every layer run (a looped layer has one store per pass)."""
        specs = [self.layers[i].mixer.run_spec() for i, _ in self.runs]
        return HybridCache(specs, num_blocks, block_size, max_sequences, max_len, self.config.dtype, self.device)

    def make_batch(self, cache: HybridCache, entries, want=None, max_len: int = 0) -> RaggedBatch:
        return RaggedBatch(cache, entries, want, self.chunks, max_len)

    @torch.no_grad()
    def forward_ragged(self, batch, cache: HybridCache, on_layer: Optional[Callable] = None) -> Optional[torch.Tensor]:
        """Runs one step over the cache; fp32 logits [wanted rows, vocab] (None when nothing is wanted). ``on_layer`` is
        called with (run, residual) after every layer run, before what comes ahead of the next pass."""
        c = self.config
        x = torch.empty((batch.rows, c.width), device=self.device, dtype=torch.float32)
        Kp, emb = pad_to(c.width), dict(tokens=batch.tokens, table=self.embed, scale=c.embedding_scale)

        def ahead(r):
            """What enters the residual right before run ``r``, and the norm that feeds its first product."""
            if r == len(self.runs):
                return {}, self.final_norm
            i, t = self.runs[r]
            add = {}
            if t >= 0 and i == c.loop.start:
                add["step"] = self.loop_step[t]
                if t > 0:
                    add.update(emb, embed="add")
            return add, self.layers[i].norm1

        def step(y=None, bias=None, post=None, add=None, norm=None):
            return ops.dyn_tanh_residual(x, y, bias, post.triple if post is not None else None,
                                         next_norm=norm.triple if norm is not None else None, out_cols=Kp, out_dtype=c.dtype,
                                         **(add or {}))

        add, norm = ahead(0)
        h = step(add={**emb, **add, "embed": "set"}, norm=norm)
        for r, (i, _) in enumerate(self.runs):
            l = self.layers[i]
            y, bias, post = l.mixer.forward(h, cache.runs[r], batch), l.mixer.out_bias, l.norm1b
            if l.mlp is not None:
                h = step(y, bias, post, norm=l.norm2)
                y, bias, post = l.mlp.forward(h), l.mlp.out_bias, l.norm2b
            add, norm = ahead(r + 1)
            if on_layer is not None:
                step(y, bias, post)
                on_layer(r, x)
                y = bias = post = None
            h = step(y, bias, post, add, norm)
        if batch.n_want == 0:
            return None
        if batch.want is not None:
            h = h.index_select(0, batch.want)
        return ops.project(h, self.embed, out_dtype=torch.float32)

    # ------------------------------------------------------------------ interface of the per-request schedulers
    def make_layer_pools(self, num_blocks: int, block_size: int, max_sequences: int = 16, max_len: int = 0) -> list:
        return [self.make_cache(num_blocks, block_size, max_sequences, max_len or num_blocks * block_size)]

    def make_paged_kv_caches(self, pools: list, max_len: int) -> list:
        return [HybridSequence(pools[0])]

    def make_kv_caches(self, batch: int, max_len: int) -> list:
        if batch != 1:
            raise ValueError("HybridModel.make_kv_caches: one sequence per cache (use the serving engine for batches)")
        bs = 16
        blocks = (max_len + bs - 1) // bs
        return [HybridSequence(self.make_cache(blocks, bs, 1, blocks * bs))]

    def _no_int8(self, *a, **k):
        raise ValueError("INT8 caches are not available for this model: keys are kept in the model's precision")

    make_quantized_kv_caches = make_quantized_layer_pools = make_quantized_paged_kv_caches = _no_int8

    def forward_step(self, tokens: torch.Tensor, caches: list) -> torch.Tensor:
        """tokens [1, S_new] through one sequence -> logits [1, S_new, V]."""
        return self.forward_step_batched(tokens, [caches])

    def forward_step_batched(self, tokens: torch.Tensor, caches: list) -> torch.Tensor:
        """tokens [A, S_new], caches[sequence] -> logits [A, S_new, V]."""
        A, S = tokens.shape
        if len(caches) != A or any(len(c) != 1 for c in caches):
            raise ValueError("forward_step_batched: one HybridSequence per row of tokens")
        cache = caches[0][0].cache
        if any(c[0].cache is not cache for c in caches):
            raise ValueError("forward_step_batched: the sequences must share one cache")
        toks = tokens.cpu().numpy()
        batch = self.make_batch(cache, [(c[0], toks[a]) for a, c in enumerate(caches)], [range(S)] * A)
        logits = self.forward_ragged(batch, cache)
        batch.commit()
        return logits.view(A, S, -1)

    def forward(self, tokens: torch.Tensor) -> torch.Tensor:
        """Logits [B, S, V] of B whole sequences, run as one ragged batch."""
        B, S = tokens.shape
        bs = 16
        cache = self.make_cache(B * ((S + bs - 1) // bs), bs, B, S)
        return self.forward_step_batched(tokens, [[HybridSequence(cache)] for _ in range(B)])

    __call__ = forward

    def generate(self, prompt_ids, cfg: Optional[GenerateConfig] = None) -> list:
        """Prompt + generated ids, through the serving engine with one request."""
        from ..models.scheduler import EngineConfig
        cfg = cfg or GenerateConfig()
        if cfg.kv_int8:
            self._no_int8()
        total = len(list(prompt_ids)) + cfg.max_new_tokens
        bs = 16
        eng = self.engine_class()(self, EngineConfig(block_size=bs, num_blocks=(total + bs - 1) // bs + 1, max_seq_len=max(total, 1),
                                                     max_batch_size=1))
        rid = eng.add_request(prompt_ids, cfg)
        eng.run()
        return eng.result(rid)


__all__ = ["AttentionSpec", "DeltaSpec", "GLUSpec", "LayerSpec", "LoopSpec", "HybridConfig", "HybridModel", "pick_next_token"]
