"""Decoders that mix recurrent and attention layers, described by a list: every layer has a mixer and, optionally, a
feed-forward. Four forms of layer:

* ``sandwich``: mixer, then feed-forward, each normed before and after by Dynamic Tanh; a range of layers may run several
  times in a row with the same weights and separate caches ("loop");
* ``parallel``: mixer and feed-forward of the same x side by side, x + m (mixer(norm1 x) + ff(norm2 x)), normed by RMS with one
  gain. The gains ride on the sublayers (``in_scale``), so one normed row feeds one product for both, and one product takes
  both results back. Optionally every layer hands on a weighted sum of the embedding output and all layers' results so far
  ("depth average");
* ``post``: mixer, then feed-forward, which read x itself; their results are normed by RMS (gains stored around zero) and added.
  Optionally every layer then adds a normed side input that depends on the token ("token side");
* ``pre``: mixer, then feed-forward, each of its own norm of x, an RMS norm in equal parts of the row. Optionally a scale per channel on
  what they add ("layer scale"), a mixer input that is mixed with the one of the token before ("token shift"), and a sinusoid of the
  position and a norm at the embedding.

Embedding and output share one table, or the output has its own.

``HybridModel`` runs ragged batches (``forward_ragged``: any mix of prompt portions and decoded tokens) over a
``HybridCache``. The serving engine drives that step; ``forward_step`` / ``forward_step_batched`` give it the interface
of ``ContinuousBatchingScheduler`` and of grammar-constrained generation.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional, Union

import torch

from .. import ops
from ..nn.hybrid import (RGLRU, SSD, ChunkedAttention, ClampedGLU, DynamicTanh, ExpertMLP, GatedDelta, GatedLinear, GeluGLU, LatentAttention,
                         PartRMSNorm, Retention, RMSNorm, ScalarRMSNorm, ShapedAttention, SideBySide, SiluGLU, TimeMix, TokenSide, pad_to)
from ..nn.ragged import HybridCache, HybridSequence, PairRun, RaggedBatch, StateRun
from ..ops.masks import Window
from ..ops.moe import Choice
from ..ops.pre_norm import Shift, sinusoid_frequencies
from ..ops.ragged import ScoreForm
from ..ops.rotary import Rotary, Yarn
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
    """``decay_rank`` and ``gate_rank`` (both or neither): a decay per key channel, which like the gate is a product of that rank."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int = 0
    gate_rank: int = 0


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rotary: Rotary


@dataclass(frozen=True)
class RetentionSpec:
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rotary: Rotary


@dataclass(frozen=True)
class RGLRUSpec:
    width: int
    blocks: int
    conv: int


@dataclass(frozen=True)
class ShapedAttentionSpec:
    """Attention with chosen parts. ``window`` 0: causal; ``norm`` of q and k: "", "unit" (per head), "head" (per head with a
    weight), "whole" (all heads at once with a weight); ``distance_bias``: 2^(-8 (h + 1) / heads) per position; ``sink``: "",
    "learned", "one" (1 more in the denominator); ``gate``: "", "head", "element"; ``v_mix``: values mixed with those of the model's
    first such layer; ``q_temp`` (coef, every): queries times 1 + coef ln(floor((position + 1) / every) + 1); ``out_bias``: a bias on the
    output product."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    bias: bool = False
    keys_as_values: bool = False
    norm: str = ""
    rotary: Optional[Rotary] = None
    softcap: float = 0.0
    distance_bias: bool = False
    sink: str = ""
    gate: str = ""
    v_mix: bool = False
    q_temp: Optional[tuple] = None
    out_bias: bool = False


@dataclass(frozen=True)
class TimeMixSpec:
    heads: int
    dim: int
    rank: int


@dataclass(frozen=True)
class GatedLinearSpec:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int


@dataclass(frozen=True)
class SSDSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_parts: int = 1


@dataclass(frozen=True)
class SideBySideSpec:
    left: object
    right: object
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass(frozen=True)
class GLUSpec:
    ff: int
    limit: float


@dataclass(frozen=True)
class SiluGLUSpec:
    ff: int


@dataclass(frozen=True)
class GeluGLUSpec:
    ff: int


@dataclass(frozen=True)
class ExpertSpec:
    """Squared-ReLU experts of ``ff`` channels."""
    ff: int
    choice: Choice


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, DeltaSpec, LatentSpec, RetentionSpec, RGLRUSpec, ShapedAttentionSpec, TimeMixSpec, GatedLinearSpec, SSDSpec,
                 SideBySideSpec]
    mlp: Union[GLUSpec, SiluGLUSpec, GeluGLUSpec, ExpertSpec, None] = None


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
    max_position_embeddings: int = 1 << 20     # a bound for caches only
    architecture: str = ""
    form: str = "sandwich"                     # or "parallel", "post" or "pre"
    residual_mult: float = 1.0                 # (parallel)
    depth_average: bool = False                # (parallel)
    tied: bool = True                          # the output product uses the embedding table
    token_side: int = 0                        # (post) columns of the side table per layer, 0: no side input
    norm_parts: int = 1                        # (pre)
    layer_scale: bool = False                  # (pre)
    token_shift: bool = False                  # (pre)
    sinusoid: bool = False                     # (pre) positions are added to the embedding
    embed_norm: bool = False                   # (pre)

    def __post_init__(self):
        if self.vocab_size < 1 or self.width < 1 or not self.layers:
            raise ValueError("HybridConfig: vocabulary, width and layers must not be empty")
        lp = self.loop
        if lp is not None and not (0 <= lp.start < lp.stop <= len(self.layers) and lp.times >= 1):
            raise ValueError("HybridConfig: loop must name a range of layers and run at least once")
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("HybridConfig: dtype is bfloat16 or float32")
        if self.form not in ("sandwich", "parallel", "post", "pre"):
            raise ValueError(f"HybridConfig: unknown form {self.form!r}")
        if self.form in ("post", "pre") and lp is not None:
            raise ValueError(f"HybridConfig: {self.form}-normed layers take no loop")
        if self.form == "pre" and self.embedding_scale != 1.0:
            raise ValueError("HybridConfig: pre-normed layers take no embedding scale")
        if self.form != "pre" and (self.norm_parts != 1 or self.layer_scale or self.token_shift or self.sinusoid or self.embed_norm):
            raise ValueError("HybridConfig: norms in parts, layer scales, a token shift, a sinusoid and a norm of the embedding belong to "
                             "pre-normed layers")
        if self.form != "pre" and any(isinstance(l.mlp, ExpertSpec) for l in self.layers):
            raise ValueError("HybridConfig: mixtures of experts run in pre-normed layers")
        if self.form != "post" and self.token_side or self.token_side < 0:
            raise ValueError("HybridConfig: a side input per token belongs to post-normed layers")
        if self.form == "parallel" and (lp is not None or self.embedding_scale != 1.0):
            raise ValueError("HybridConfig: parallel layers take no loop and no embedding scale")
        if self.form != "parallel" and (self.residual_mult != 1.0 or self.depth_average):
            raise ValueError("HybridConfig: a residual multiplier and depth averaging belong to parallel layers")

    def runs(self):
        """[(layer, pass)] in the order they run; pass is -1 outside the loop."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return [(i, -1) for i in range(n)]
        return ([(i, -1) for i in range(lp.start)]
                + [(i, t) for t in range(lp.times) for i in range(lp.start, lp.stop)]
                + [(i, -1) for i in range(lp.stop, n)])


def mixers_of(m) -> list:
    """A mixer's spec, or those of its parts."""
    return mixers_of(m.left) + mixers_of(m.right) if isinstance(m, SideBySideSpec) else [m]


def _make_mixer(m, c: HybridConfig, device):
    W, dt = c.width, c.dtype
    if isinstance(m, SideBySideSpec):
        return SideBySide(_make_mixer(m.left, c, device), _make_mixer(m.right, c, device), m.left_scale, m.right_scale, W, dt, device)
    if isinstance(m, ShapedAttentionSpec):
        if m.sink not in ("", "learned", "one"):
            raise ValueError(f"attention: unknown sink {m.sink!r}")
        slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / m.heads) for h in range(m.heads)]) if m.distance_bias else None
        form = ScoreForm(m.scale, Window(m.window) if m.window else 0, m.softcap, slopes, torch.zeros(m.heads) if m.sink == "one" else None)
        return ShapedAttention(W, m.heads, m.kv_heads, m.dim, m.vdim, form, c.eps, dt, device, m.bias, m.keys_as_values, m.norm, m.rotary,
                               m.sink == "learned", m.v_mix, m.gate, m.q_temp, m.out_bias)
    if isinstance(m, GatedLinearSpec):
        return GatedLinear(W, m.heads, m.dim, m.vdim, m.rank, m.tau, c.eps, dt, device)
    if isinstance(m, TimeMixSpec):
        return TimeMix(W, m.heads, m.dim, m.rank, c.eps, dt, device)
    if isinstance(m, SSDSpec):
        return SSD(W, m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_parts, c.eps, dt, device)
    if isinstance(m, AttentionSpec):
        return ChunkedAttention(W, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.chunk, dt, device)
    if isinstance(m, DeltaSpec):
        return GatedDelta(W, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, c.eps, dt, device, m.decay_rank, m.gate_rank)
    if isinstance(m, LatentSpec):
        return LatentAttention(W, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.rotary, c.eps, dt, device)
    if isinstance(m, RetentionSpec):
        return Retention(W, m.heads, m.dim, m.vdim, m.decay, m.rotary, c.eps, dt, device)
    if isinstance(m, RGLRUSpec):
        return RGLRU(W, m.width, m.blocks, m.conv, dt, device)
    raise ValueError(f"HybridConfig: unknown mixer {m!r}")


def _make_mlp(m, c: HybridConfig, device):
    if m is None:
        return None
    if isinstance(m, SiluGLUSpec):
        return SiluGLU(c.width, m.ff, c.dtype, device)
    if isinstance(m, GeluGLUSpec):
        return GeluGLU(c.width, m.ff, c.dtype, device)
    if isinstance(m, ExpertSpec):
        return ExpertMLP(c.width, m.ff, m.choice, c.dtype, device)
    return ClampedGLU(c.width, m.ff, m.limit, c.dtype, device)


class _Layer:
    extra: dict = {}                  # vectors of the layer itself: name -> tensor

    def run_spec(self):
        return self.mixer.run_spec()


class _SandwichLayer(_Layer):
    def __init__(self, spec: LayerSpec, c: HybridConfig, index: int, device):
        norm = lambda: DynamicTanh(c.width, c.dtype, device)   # noqa: E731
        self.mixer, self.mlp = _make_mixer(spec.mixer, c, device), _make_mlp(spec.mlp, c, device)
        self.norm1, self.norm1b = norm(), norm()
        self.norm2, self.norm2b = (norm(), norm()) if spec.mlp is not None else (None, None)

    def parts(self):
        out = [("norm1", self.norm1), ("norm1b", self.norm1b), ("mix.", self.mixer)]
        if self.mlp is not None:
            out += [("norm2", self.norm2), ("norm2b", self.norm2b), ("mlp.", self.mlp)]
        return out


class _ParallelLayer(_Layer):
    """One input matrix (rows of the mixer, then of the feed-forward) and one output matrix (columns likewise)."""

    def __init__(self, spec: LayerSpec, c: HybridConfig, index: int, device):
        self.mixer, self.mlp = _make_mixer(spec.mixer, c, device), _make_mlp(spec.mlp, c, device)
        self.norm1 = ScalarRMSNorm(c.eps, c.dtype, device)
        self.norm2 = ScalarRMSNorm(c.eps, c.dtype, device) if spec.mlp is not None else None
        subs = [s for s in (self.mixer, self.mlp) if s is not None]
        for s in subs:
            if not s.takes_in_scale or s.out_bias is not None:
                raise ValueError(f"HybridConfig: {type(s).__name__} does not run in parallel layers")
        self.in_cut, self.out_cut = self.mixer.cols, self.mixer.out_cols
        if self.mlp is None:
            self.w_in, self.w_out = self.mixer.w_in, self.mixer.w_out
        else:
            new = lambda *shape: torch.zeros(shape, dtype=c.dtype, device=device)   # noqa: E731
            self.w_in = new(sum(s.cols for s in subs), self.mixer.w_in.shape[1])
            self.w_out = new(c.width, sum(s.out_cols for s in subs))
            self.mixer.place(self.w_in[:self.in_cut], self.w_out[:, :self.out_cut])
            self.mlp.place(self.w_in[self.in_cut:], self.w_out[:, self.out_cut:])
        self.average = torch.zeros(index + 2, dtype=torch.float32, device=device) if c.depth_average else None
        self.extra = {"dwa": self.average} if c.depth_average else {}

    def parts(self):
        out = [("norm1", self.norm1), ("mix.", self.mixer)]
        if self.mlp is not None:
            out += [("norm2", self.norm2), ("mlp.", self.mlp)]
        return out

    def set_gains(self) -> None:
        self.mixer.in_scale = self.norm1.gain
        if self.mlp is not None:
            self.mlp.in_scale = self.norm2.gain

    def forward(self, h, storage, batch):
        """h: the normed row without a gain."""
        p = ops.project(h, self.w_in)
        if self.mlp is None:
            return ops.project(self.mixer.core(p, storage, batch), self.w_out)
        z = torch.empty((h.shape[0], self.w_out.shape[1]), device=h.device, dtype=h.dtype)
        self.mixer.core(p[:, :self.in_cut], storage, batch, out=z[:, :self.out_cut])
        self.mlp.core(p[:, self.in_cut:], out=z[:, self.out_cut:])
        return ops.project(z, self.w_out)


class _PostLayer(_Layer):
    def __init__(self, spec: LayerSpec, c: HybridConfig, index: int, device):
        norm = lambda: RMSNorm(c.width, c.eps, 1.0, c.dtype, device)   # noqa: E731
        self.mixer, self.mlp = _make_mixer(spec.mixer, c, device), _make_mlp(spec.mlp, c, device)
        self.norm1, self.norm2 = norm(), norm() if spec.mlp is not None else None
        self.side = TokenSide(c.width, c.token_side, c.eps, c.dtype, device) if c.token_side else None
        for s in (self.mixer, self.mlp):
            if s is not None and s.out_bias is not None:
                raise ValueError(f"HybridConfig: {type(s).__name__} does not run in post-normed layers")

    def parts(self):
        out = [("norm1", self.norm1), ("mix.", self.mixer)]
        if self.mlp is not None:
            out += [("norm2", self.norm2), ("mlp.", self.mlp)]
        if self.side is not None:
            out.append(("side.", self.side))
        return out


class _PreLayer(_Layer):
    def __init__(self, spec: LayerSpec, c: HybridConfig, index: int, device):
        norm = lambda: PartRMSNorm(c.width, c.norm_parts, c.eps, c.dtype, device)   # noqa: E731
        vec = lambda on: torch.zeros(c.width, dtype=torch.float32, device=device) if on else None   # noqa: E731
        self.mixer, self.mlp = _make_mixer(spec.mixer, c, device), _make_mlp(spec.mlp, c, device)
        self.norm1, self.norm2 = norm(), norm() if spec.mlp is not None else None
        self.ls1, self.ls2, self.shift = vec(c.layer_scale), vec(c.layer_scale and spec.mlp is not None), None
        self.extra = {n: t for n, t in (("ls1", self.ls1), ("ls2", self.ls2)) if t is not None}
        if c.token_shift:
            self.shift = torch.zeros(pad_to(c.width), dtype=torch.float32, device=device)
            self.extra["shift"] = self.shift[:c.width]

    def parts(self):
        out = [("norm1", self.norm1), ("mix.", self.mixer)]
        if self.mlp is not None:
            out += [("norm2", self.norm2), ("mlp.", self.mlp)]
        return out

    def run_spec(self):
        """With a token shift: the mixer's storage, and the last input of every sequence."""
        spec = self.mixer.run_spec()
        return PairRun(spec, StateRun((0,), (1, self.shift.shape[0]))) if self.shift is not None else spec

    def storage(self, run):
        """(the mixer's storage, what the norm takes for the shift)"""
        return (run[0], Shift(self.shift, run[1][0])) if self.shift is not None else (run, None)


_LAYERS = {"sandwich": _SandwichLayer, "parallel": _ParallelLayer, "post": _PostLayer, "pre": _PreLayer}


class HybridModel:
    def __init__(self, config: HybridConfig, device=None, init_std: Optional[float] = None, seed: int = 0):
        self.config = c = config
        self.device = torch.device(device) if device is not None else torch.device("cpu")
        # one table for the embedding and, unless it has its own, the output product; rows are padded like every matrix the
        # GEMMs read
        self.embed = torch.zeros(c.vocab_size, pad_to(c.width), dtype=c.dtype, device=self.device)
        self.head = self.embed if c.tied else torch.zeros_like(self.embed)
        values = {(m.kv_heads, m.vdim) for l in c.layers for m in mixers_of(l.mixer) if getattr(m, "v_mix", False)}
        if len(values) > 1:
            raise ValueError("HybridConfig: layers that mix values have the same value heads")
        self.layers = [_LAYERS[c.form](s, c, i, self.device) for i, s in enumerate(c.layers)]
        final = {"sandwich": lambda: DynamicTanh(c.width, c.dtype, self.device), "parallel": lambda: ScalarRMSNorm(c.eps, c.dtype, self.device),
                 "post": lambda: RMSNorm(c.width, c.eps, 1.0, c.dtype, self.device),
                 "pre": lambda: PartRMSNorm(c.width, c.norm_parts, c.eps, c.dtype, self.device)}
        self.final_norm = final[c.form]()
        self.embed_norm = final["pre"]() if c.embed_norm else None
        self.frequencies = sinusoid_frequencies(c.width).to(self.device) if c.sinusoid else None
        self.side_table = (torch.zeros(c.vocab_size, c.token_side * len(c.layers), dtype=c.dtype, device=self.device)
                           if c.token_side else None)
        self.loop_step = (torch.zeros(c.loop.times, c.width, dtype=torch.float32, device=self.device)
                          if c.loop is not None else None)
        self.runs = c.runs()
        # what the mixers ask a batch for: masks of prompt attention, sizes of prompt tiles
        self.masks = list(dict.fromkeys(m for l in self.layers for m in l.mixer.masks))
        self.tiles = sorted({t for l in self.layers for t in l.mixer.tiles})
        if init_std is not None:
            self.init_weights(init_std, seed)

    # ------------------------------------------------------------------ the parts of a model the framework asks for
    def _device(self):
        return self.device

    def eval(self) -> "HybridModel":
        return self

    def parameters(self):
        for _, t in self._tables():
            yield t
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
        if self.embed_norm is not None:
            yield "embed.norm", self.embed_norm
        yield "final.norm", self.final_norm

    def _tables(self):
        """Tensors of the model itself: (name, packed tensor; its first columns are the logical ones)."""
        yield "embed", self.embed
        if not self.config.tied:
            yield "head", self.head
        if self.side_table is not None:
            yield "side.embed", self.side_table
        if self.loop_step is not None:
            yield "loop.step", self.loop_step
        for i, l in enumerate(self.layers):
            for name, t in l.extra.items():
                yield f"l{i}.{name}", t

    def _logical(self, t: torch.Tensor) -> torch.Tensor:
        return t[:, :self.config.width] if t.dim() == 2 and t is not self.side_table else t

    def logical_shapes(self) -> Dict[str, tuple]:
        out = {name: tuple(self._logical(t).shape) for name, t in self._tables()}
        for name, part in self._parts():
            out.update({name + k: tuple(v) for k, v in part.logical_shapes().items()})
        return out

    @torch.no_grad()
    def load_tensors(self, sd: Dict[str, torch.Tensor]) -> list:
        """Packs a dict of logical tensors; returns the names in it that the model does not have."""
        known = self.logical_shapes()
        for name, t in self._tables():
            if name not in sd:
                raise KeyError(f"load: required tensor {name!r} is missing")
            if tuple(sd[name].shape) != known[name]:
                raise ValueError(f"load: shape of {name!r} is {tuple(sd[name].shape)}, expected {known[name]}")
            self._logical(t).copy_(sd[name])
        for name, part in self._parts():
            try:
                part.load({k: sd[name + k] for k in part.logical_shapes() if name + k in sd})
            except (KeyError, ValueError, TypeError) as e:
                raise type(e)(f"{name}: {e.args[0]}") from None
        if self.config.form == "parallel":
            for l in self.layers:
                l.set_gains()
        return [k for k in sd if k not in known]

    def state_tensors(self) -> Dict[str, torch.Tensor]:
        out = {name: self._logical(t).to(self.config.dtype).contiguous() for name, t in self._tables()}
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
        """N(0, std) matrices from a fixed seed; norms start with unit gains, decays between slow and fast, and a depth average
        passes the newest result on."""
        gen = torch.Generator(device=self.device)
        gen.manual_seed(seed)
        around_zero = {f"l{i}.{n}" for i in range(len(self.layers)) for n in ("norm1", "norm2")} | {"final.norm"}

        def draw(name, shape):
            last = name.rsplit(".", 1)[-1]
            if self.config.form == "post" and name in around_zero or last == "sink":
                return torch.zeros(shape)
            if last == "vmix":
                return torch.tensor(0.5)
            if last == "alpha" or shape == ():
                return torch.tensor(1.0)
            if ".mu." in name or last == "shift":
                return torch.rand(shape, generator=gen, device=self.device)
            if last == "correction":
                return 0.05 * torch.randn(shape, generator=gen, device=self.device)
            if last == "w0":
                return torch.rand(shape, generator=gen, device=self.device) * 5.0 - 6.0
            if last == "u":
                return torch.rand(shape, generator=gen, device=self.device)
            if last == "dwa":
                return torch.eye(shape[0])[-1]
            if len(shape) == 3:
                return torch.randn(shape, generator=gen, device=self.device) * shape[-1] ** -0.5
            if last == "lam":
                return torch.rand(shape, generator=gen, device=self.device) * 3.0 - 4.0
            if last == "b":
                return torch.zeros(shape)
            if len(shape) == 2:
                s = 0.5 if last == "conv" else std
                return torch.randn(shape, generator=gen, device=self.device) * s
            if last == "A_log":
                return torch.rand(shape, generator=gen, device=self.device) * 2.0 - 2.0
            if last == "dt_bias":
                return torch.rand(shape, generator=gen, device=self.device) - 3.0
            return torch.ones(shape)
        self.load_tensors({n: draw(n, s) for n, s in self.logical_shapes().items()})

    # ------------------------------------------------------------------ the step
    def make_cache(self, num_blocks: int, block_size: int, max_sequences: int, max_len: int) -> HybridCache:
        """K / V pages and recurrent slots of every layer run (a looped layer has one store per pass)."""
        specs = [self.layers[i].run_spec() for i, _ in self.runs]
        return HybridCache(specs, num_blocks, block_size, max_sequences, max_len, self.config.dtype, self.device)

    def make_batch(self, cache: HybridCache, entries, want=None, max_len: int = 0) -> RaggedBatch:
        return RaggedBatch(cache, entries, want, self.masks, max_len, self.tiles)

    @torch.no_grad()
    def forward_ragged(self, batch, cache: HybridCache, on_layer: Optional[Callable] = None) -> Optional[torch.Tensor]:
        """Runs one step over the cache; fp32 logits [wanted rows, vocab] (None when nothing is wanted). ``on_layer`` is
        called with (run, residual) after every layer run, before what comes ahead of the next pass."""
        run = {"sandwich": self._run_sandwich, "parallel": self._run_parallel, "post": self._run_post, "pre": self._run_pre}[self.config.form]
        h = run(batch, cache, on_layer)
        if batch.n_want == 0:
            return None
        if batch.want is not None:
            h = h.index_select(0, batch.want)
        return ops.project(h, self.head, out_dtype=torch.float32)

    def _run_sandwich(self, batch, cache: HybridCache, on_layer) -> torch.Tensor:
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
        return h

    def _run_parallel(self, batch, cache: HybridCache, on_layer) -> torch.Tensor:
        c = self.config
        n = len(self.layers)
        form = dict(out_cols=pad_to(c.width), out_dtype=c.dtype, eps=c.eps)
        # what the depth average looks back on: the embedding output and every layer's result
        history = (torch.empty((n, batch.rows, c.width), device=self.device, dtype=torch.float32) if c.depth_average else None)
        x, h = ops.depth_residual(tokens=batch.tokens, table=self.embed, width=c.width, history=history, **form)
        for r, l in enumerate(self.layers):
            y = l.forward(h, cache.runs[r], batch)
            last = r == n - 1
            x, h = ops.depth_residual(x, y, c.residual_mult, history=history, depth=r + 1, average=l.average, store=not last,
                                      gain=self.final_norm.gain if last else 1.0, **form)
            if on_layer is not None:
                on_layer(r, x)
        return h

    def _run_post(self, batch, cache: HybridCache, on_layer) -> torch.Tensor:
        c = self.config
        x = torch.empty((batch.rows, c.width), device=self.device, dtype=torch.float32)
        form = dict(out_cols=pad_to(c.width), out_dtype=c.dtype)

        def add(y, norm, last):
            return ops.post_norm_step(x, y, norm.gain, c.eps, final=self.final_norm.gain if last else None, **form)

        h = ops.post_norm_step(x, tokens=batch.tokens, table=self.embed, scale=c.embedding_scale, eps=c.eps, **form)
        for r, l in enumerate(self.layers):
            last = r == len(self.layers) - 1
            h = add(l.mixer.forward(h, cache.runs[r], batch), l.norm1, last and l.mlp is None and l.side is None)
            if l.mlp is not None:
                h = add(l.mlp.forward(h), l.norm2, last and l.side is None)
            if l.side is not None:
                h = add(l.side.forward(h, batch.tokens, self.side_table, r * c.token_side), l.side.norm, last)
            if on_layer is not None:
                on_layer(r, x)
        return h

    def _run_pre(self, batch, cache: HybridCache, on_layer) -> torch.Tensor:
        c = self.config
        x = moved = None

        def step(norm, shift=None, **kw):
            nonlocal x, moved
            x, h, moved = ops.pre_norm_step(batch, c.width, norm.gain, c.norm_parts, c.eps, x, shift=shift, moved=moved, out_cols=pad_to(c.width),
                                            out_dtype=c.dtype, **kw)
            return h

        kept = [l.storage(run) for l, run in zip(self.layers, cache.runs)]
        h = step(self.layers[0].norm1, kept[0][1], table=self.embed, freq=self.frequencies,
                 embed_gain=self.embed_norm.gain if self.embed_norm is not None else None)
        for r, l in enumerate(self.layers):
            add = dict(y=l.mixer.forward(h, kept[r][0], batch), bias=l.mixer.out_bias, scale=l.ls1)
            if l.mlp is not None:
                h = step(l.norm2, **add)
                add = dict(y=l.mlp.forward(h), bias=l.mlp.out_bias, scale=l.ls2)
            last = r == len(self.layers) - 1
            h = step(self.final_norm if last else self.layers[r + 1].norm1, None if last else kept[r + 1][1], **add)
            if on_layer is not None:
                on_layer(r, x)
        return h

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


__all__ = ["AttentionSpec", "Choice", "DeltaSpec", "ExpertSpec", "GLUSpec", "GatedLinearSpec", "GeluGLUSpec", "HybridConfig", "HybridModel", "LatentSpec", "LayerSpec", "LoopSpec", "RGLRUSpec",
           "RetentionSpec", "Rotary", "SSDSpec", "ShapedAttentionSpec", "SideBySideSpec", "SiluGLUSpec", "TimeMixSpec", "Yarn",
           "pick_next_token"]
