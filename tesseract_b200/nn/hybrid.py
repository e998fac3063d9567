"""Building blocks of hybrid decoders for inference over ragged batches: norms (Dynamic Tanh, RMS with one gain or one per
channel, over the row or equal parts of it), mixers (chunked attention, attention with norms, rotations, windows, sinks and gates, latent
attention, the gated delta rule with decays per head or per channel, retention, the real-gated linear recurrence, time mixing, gated linear
attention, state-space duality, two of them side by side), feed-forwards (gated: clamped, SiLU, GELU; a mixture of squared-ReLU experts)
and a side input per token.

A mixer or feed-forward is two matrix products around a ``core``: rows of ``w_in`` make its packed input, ``w_out`` takes what
the core leaves. Layers whose sublayers run side by side lay several of them into one matrix (``place``) and call the cores on
columns of the shared product.

A block holds its parameters packed for the kernels (adjacent projections in one matrix, sections and heads padded with
zeros, everything that the kernels use in fp32 already widened) and translates to and from its logical tensors:
``logical_shapes`` names them, ``load`` packs a dict of them, ``unpack`` gives them back.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import ops
from ..ops.delta import DeltaGeometry, DeltaWeights, gated_delta
from ..ops.pre_norm import NORM_UNIT, NORM_UNITS
from ..ops.latent import LatentGeometry, LatentWeights, latent_attention
from ..ops.gemm import input_columns
from ..ops.masks import Window
from ..ops.ragged import AttentionGeometry, AttentionWeights, ScoreForm, padded_head_dim, ragged_attention, shaped_attention
from ..ops.retention import SPAN, RetentionGeometry, log2_decays, retention
from ..ops.rglru import CHUNK, RGLRUGeometry, RGLRUWeights, rglru
from ..ops.rotary import Rotary
from ..ops.ssd import CONV_TILE, SSDGeometry, SSDWeights, ssd
from ..ops.moe import Choice, relu2_experts, router_logits
from ..ops.timemix import (SPAN as STATE_SPAN, STREAMS, GatedLinearGeometry, GatedLinearWeights, TimeMixGeometry, TimeMixWeights, gated_linear,
                           time_mix, token_shift)
from .ragged import LatentRun, PagedRun, PairRun, StateRun


def pad_to(n: int, m: int = 16) -> int:
    return (n + m - 1) // m * m


class _Packed:
    def __init__(self, dtype, device):
        self.dtype, self.device = dtype, torch.device(device) if device is not None else torch.device("cpu")

    def _zeros(self, *shape, dtype=None):
        return torch.zeros(shape, dtype=dtype or self.dtype, device=self.device)

    def tensors(self):
        return [t for t in vars(self).values() if isinstance(t, torch.Tensor)]

    def load(self, t: Dict[str, torch.Tensor]) -> None:
        for name, shape in self.logical_shapes().items():
            if name not in t:
                raise KeyError(f"load: required tensor {name!r} is missing")
            if tuple(t[name].shape) != tuple(shape):
                raise ValueError(f"load: shape of {name!r} is {tuple(t[name].shape)}, expected {tuple(shape)}")
            if not t[name].is_floating_point():
                raise TypeError(f"load: {name!r} is not a floating-point tensor")
        self._pack(t)


class _Sublayer(_Packed):
    """Two products around a core. ``in_scale`` multiplies the packed input inside the core: the gain of a norm that has only
    one, where the layer leaves it to the sublayers. ``tile``: size of the prompt tiles that the core asks the batch for, ``masks``:
    the attention masks."""
    out_bias = None
    in_scale = 1.0
    takes_in_scale = False
    tile = 0
    masks = ()

    @property
    def cols(self) -> int:
        return self.w_in.shape[0]

    @property
    def out_cols(self) -> int:
        return self.w_out.shape[1]

    def place(self, w_in: torch.Tensor, w_out: torch.Tensor) -> None:
        """Moves the two matrices into rows and columns of larger ones."""
        w_in.copy_(self.w_in)
        w_out.copy_(self.w_out)
        self.w_in, self.w_out = w_in, w_out


class _Mixer(_Sublayer):
    """``streams``: first packed column of every input that the first product reads (a mixer that makes its own inputs from h has
    ``mix_inputs``). ``out_scale`` multiplies what the core leaves."""
    streams = (0,)
    out_scale = 1.0

    @property
    def tiles(self) -> tuple:
        return (self.tile,) if self.tile else ()

    def forward(self, h, storage, batch):
        p = ops.project(h, self.w_in) if len(self.streams) == 1 else ops.project_inputs(self.mix_inputs(h, storage, batch), self.w_in,
                                                                                         self.streams)
        return ops.project(self.core(p, storage, batch), self.w_out)


class _FeedForward(_Sublayer):
    def forward(self, h):
        return ops.project(self.core(ops.project(h, self.w_in)), self.w_out)


class ScalarRMSNorm(_Packed):
    """x / sqrt(mean(x^2) + eps) * gain with one gain for all channels."""

    def __init__(self, eps: float, dtype, device):
        super().__init__(dtype, device)
        self.eps, self.gain = float(eps), 1.0

    def logical_shapes(self):
        return {"": ()}

    def _pack(self, t):
        self.gain = float(t[""])

    def unpack(self):
        return {"": torch.tensor(self.gain, dtype=self.dtype, device=self.device)}


class RMSNorm(_Packed):
    """x / sqrt(mean(x^2) + eps) times a gain per channel, stored as it is or, with ``offset`` 1, around zero."""

    def __init__(self, width: int, eps: float, offset: float, dtype, device):
        super().__init__(dtype, device)
        self.width, self.eps, self.offset = width, float(eps), float(offset)
        self.gain = self._zeros(width, dtype=torch.float32) + 1.0

    def logical_shapes(self):
        return {"": (self.width,)}

    def _pack(self, t):
        self.gain.copy_(t[""].float() + self.offset)

    def unpack(self):
        return {"": (self.gain - self.offset).to(self.dtype)}


class PartRMSNorm(RMSNorm):
    """The row in ``parts`` equal runs of channels, every one over its own root mean square, times a gain per channel."""

    def __init__(self, width: int, parts: int, eps: float, dtype, device):
        if parts < 1 or width % parts:
            raise ValueError("norm: the width is a multiple of its parts")
        if parts * -(-(width // parts) // NORM_UNIT[width // parts % 4 == 0]) > NORM_UNITS:
            raise ValueError("norm: the row has too many parts or columns")
        super().__init__(width, eps, 0.0, dtype, device)
        self.parts = parts


class DynamicTanh(_Packed):
    """tanh(alpha x) * weight + bias per channel; computes no statistics."""

    def __init__(self, width: int, dtype, device):
        super().__init__(dtype, device)
        self.width = width
        self.alpha = 1.0
        self.weight, self.bias = self._zeros(width, dtype=torch.float32) + 1.0, self._zeros(width, dtype=torch.float32)

    def logical_shapes(self):
        return {"": (self.width,), ".b": (self.width,), ".alpha": ()}

    def _pack(self, t):
        self.alpha = float(t[".alpha"])
        self.weight.copy_(t[""])
        self.bias.copy_(t[".b"])

    def unpack(self):
        return {"": self.weight.to(self.dtype), ".b": self.bias.to(self.dtype),
                ".alpha": torch.tensor(self.alpha, dtype=self.dtype, device=self.device)}

    @property
    def triple(self):
        return self.alpha, self.weight, self.bias


class ChunkedAttention(_Mixer):
    """Grouped-query attention without positions whose mask is causal inside runs of ``chunk`` positions (0: causal over
    everything); biases on q, k and v. Query / key heads are ``dim`` wide, value heads ``vdim``."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, chunk: int, dtype, device):
        super().__init__(dtype, device)
        if heads % kv_heads or min(heads, kv_heads, dim, vdim) < 1 or chunk < 0:
            raise ValueError("attention: positive sizes, and heads a multiple of kv_heads")
        self.width, self.heads, self.kv_heads, self.dim, self.vdim = width, heads, kv_heads, dim, vdim
        self.scale, self.chunk = float(scale), int(chunk)
        self.masks = (self.chunk,)
        self.D = padded_head_dim(dim, vdim, dtype)
        self.w_in = self._zeros((heads + 2 * kv_heads) * self.D, pad_to(width))
        self.b_in = self._zeros((heads + 2 * kv_heads) * self.D, dtype=torch.float32)
        self.w_out = self._zeros(width, heads * self.D)

    def run_spec(self) -> PagedRun:
        return PagedRun(self.kv_heads, self.D)

    def _sections(self):
        at = 0
        for name, n, d in (("q", self.heads, self.dim), ("k", self.kv_heads, self.dim), ("v", self.kv_heads, self.vdim)):
            yield name, at, n, d
            at += n * self.D

    def logical_shapes(self):
        out = {}
        for name, _, n, d in self._sections():
            out[name], out[name + ".b"] = (n * d, self.width), (n * d,)
        out["o"] = (self.width, self.heads * self.vdim)
        return out

    def _views(self, name, at, n, d):
        w = self.w_in[at:at + n * self.D].view(n, self.D, -1)[:, :d, :self.width]
        b = self.b_in[at:at + n * self.D].view(n, self.D)[:, :d]
        return w, b

    def _pack(self, t):
        for name, at, n, d in self._sections():
            w, b = self._views(name, at, n, d)
            w.copy_(t[name].view(n, d, self.width))
            b.copy_(t[name + ".b"].view(n, d))
        self.w_out.view(self.width, self.heads, self.D)[:, :, :self.vdim].copy_(t["o"].view(self.width, self.heads, self.vdim))

    def unpack(self):
        out = {}
        for name, at, n, d in self._sections():
            w, b = self._views(name, at, n, d)
            out[name], out[name + ".b"] = w.reshape(n * d, self.width), b.reshape(n * d).to(self.dtype)
        out["o"] = self.w_out.view(self.width, self.heads, self.D)[:, :, :self.vdim].reshape(self.width, -1)
        return out

    def core(self, qkv, storage, batch):
        return ragged_attention(qkv, self.b_in, storage[0], storage[1], batch, self.heads, self.kv_heads, self.scale, self.chunk)


class GatedDelta(_Mixer):
    """The gated delta rule with short convolutions (see ``ops.delta``). With ``decay_rank`` and ``gate_rank``: decays per key channel, and
    these and a sigmoid gate from products of that rank."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, conv: int, eps: float, dtype, device,
                 decay_rank: int = 0, gate_rank: int = 0):
        super().__init__(dtype, device)
        self.width = width
        self.geo = g = DeltaGeometry(kv_heads, heads, dim, vdim, conv, decay_rank, gate_rank)
        self.w_in = self._zeros(g.cols, pad_to(width))
        self.w_out = self._zeros(width, g.out_cols)
        f32 = torch.float32
        self.w = DeltaWeights(self._zeros(conv, g.conv_cols, dtype=f32), self._zeros(heads, dtype=f32),
                              self._zeros(heads * dim if g.channels else heads, dtype=f32), self._zeros(vdim, dtype=f32), float(eps))
        if g.channels:
            self.w.w_decay = self._zeros(pad_to(heads * dim, 8), pad_to(decay_rank))
            self.w.w_gate = self._zeros(pad_to(heads * vdim, 8), pad_to(gate_rank))

    def tensors(self):
        return super().tensors() + [t for t in vars(self.w).values() if isinstance(t, torch.Tensor)]

    def run_spec(self) -> StateRun:
        g = self.geo
        return StateRun((g.heads, g.dim, g.vdim_pad), (g.taps - 1, g.conv_cols))

    def _sections(self):
        g = self.geo
        qk, hv = g.kv_heads * g.dim, g.heads * g.vdim
        own = (("q", 0, qk), ("k", g.off_k, qk), ("v", g.off_v, hv))
        if g.channels:
            return own + (("b", g.off_b, g.heads), ("a1", g.off_a, g.decay_rank), ("g1", g.off_low_gate, g.gate_rank))
        return own + (("g", g.off_gate, hv), ("b", g.off_b, g.heads), ("a", g.off_a, g.heads))

    def _second(self):
        """name -> (matrix, rows, columns) of the products that follow the first."""
        g = self.geo
        return {"a2": (self.w.w_decay, g.heads * g.dim, g.decay_rank),
                "g2": (self.w.w_gate, g.heads * g.vdim, g.gate_rank)} if g.channels else {}

    def logical_shapes(self):
        g = self.geo
        out = {}
        for name, _, n in self._sections():
            out[name] = (n, self.width)
            if name in "qkv":
                out[name + ".conv"] = (n, g.taps)
        out.update({"A_log": (g.heads,), "dt_bias": tuple(self.w.dt_bias.shape), "norm": (g.vdim,), "o": (self.width, g.heads * g.vdim)})
        out.update({name: (n, k) for name, (_, n, k) in self._second().items()})
        return out

    def _pack(self, t):
        for name, at, n in self._sections():
            self.w_in[at:at + n, :self.width].copy_(t[name])
            if name in "qkv":
                self.w.conv[:, at:at + n].copy_(t[name + ".conv"].t())
        self.w.a_log.copy_(t["A_log"])
        self.w.dt_bias.copy_(t["dt_bias"])
        self.w.norm.copy_(t["norm"])
        self.w_out[:, :t["o"].shape[1]].copy_(t["o"])
        for name, (w, n, k) in self._second().items():
            w[:n, :k].copy_(t[name])

    def unpack(self):
        out = {}
        for name, at, n in self._sections():
            out[name] = self.w_in[at:at + n, :self.width].contiguous()
            if name in "qkv":
                out[name + ".conv"] = self.w.conv[:, at:at + n].t().contiguous().to(self.dtype)
        out.update({"A_log": self.w.a_log.to(self.dtype), "dt_bias": self.w.dt_bias.to(self.dtype),
                    "norm": self.w.norm.to(self.dtype), "o": self.w_out[:, :self.geo.heads * self.geo.vdim].contiguous()})
        out.update({name: w[:n, :k].contiguous() for name, (w, n, k) in self._second().items()})
        return out

    def core(self, proj, storage, batch, out=None):
        return gated_delta(proj, self.geo, self.w, storage[0], storage[1], batch, out)


class ClampedGLU(_FeedForward):
    """g = min(W_gate h, limit), u = clamp(W_up h, -limit, limit); W_down (g sigmoid(slope g) (u + 1)), biases on all three.
    The bias of the last product is left to the residual step (``out_bias``)."""

    def __init__(self, width: int, ff: int, limit: float, dtype, device, slope: float = 1.702):
        super().__init__(dtype, device)
        if ff < 1:
            raise ValueError("feed-forward: ff must be positive")
        self.width, self.ff, self.limit, self.slope = width, ff, float(limit), float(slope)
        self.F = F = pad_to(ff)
        self.w_in, self.b_in = self._zeros(2 * F, pad_to(width)), self._zeros(2 * F, dtype=torch.float32)
        self.w_out, self.out_bias = self._zeros(width, F), self._zeros(width, dtype=torch.float32)

    def logical_shapes(self):
        return {"gate": (self.ff, self.width), "gate.b": (self.ff,), "up": (self.ff, self.width), "up.b": (self.ff,),
                "down": (self.width, self.ff), "down.b": (self.width,)}

    def _pack(self, t):
        for name, at in (("gate", 0), ("up", self.F)):
            self.w_in[at:at + self.ff, :self.width].copy_(t[name])
            self.b_in[at:at + self.ff].copy_(t[name + ".b"])
        self.w_out[:, :self.ff].copy_(t["down"])
        self.out_bias.copy_(t["down.b"])

    def unpack(self):
        out = {}
        for name, at in (("gate", 0), ("up", self.F)):
            out[name] = self.w_in[at:at + self.ff, :self.width].contiguous()
            out[name + ".b"] = self.b_in[at:at + self.ff].to(self.dtype)
        out["down"], out["down.b"] = self.w_out[:, :self.ff].contiguous(), self.out_bias.to(self.dtype)
        return out

    def core(self, gate_up, out=None):
        return ops.clamped_glu(gate_up, self.b_in, self.limit, self.slope, out=out)


class SiluGLU(_FeedForward):
    """W_down (silu(W_gate h) * (W_up h)) without biases."""
    takes_in_scale = True

    def __init__(self, width: int, ff: int, dtype, device):
        super().__init__(dtype, device)
        if ff < 1:
            raise ValueError("feed-forward: ff must be positive")
        self.width, self.ff = width, ff
        self.F = F = pad_to(ff)
        self.w_in, self.w_out = self._zeros(2 * F, pad_to(width)), self._zeros(width, F)

    def logical_shapes(self):
        return {"gate": (self.ff, self.width), "up": (self.ff, self.width), "down": (self.width, self.ff)}

    def _pack(self, t):
        for name, at in (("gate", 0), ("up", self.F)):
            self.w_in[at:at + self.ff, :self.width].copy_(t[name])
        self.w_out[:, :self.ff].copy_(t["down"])

    def unpack(self):
        out = {name: self.w_in[at:at + self.ff, :self.width].contiguous() for name, at in (("gate", 0), ("up", self.F))}
        out["down"] = self.w_out[:, :self.ff].contiguous()
        return out

    def core(self, gate_up, out=None):
        return ops.silu_glu(gate_up, self.in_scale, out)


class GeluGLU(SiluGLU):
    """W_down (gelu(W_gate h) * (W_up h)), the tanh form of GELU, without biases."""

    def core(self, gate_up, out=None):
        return ops.gelu_glu(gate_up, self.in_scale, out)


class ExpertMLP(_Packed):
    """A mixture of experts W_down relu(W_up h)^2 (see ``ops.moe.relu2_experts``); their weighted sum is left to the residual step."""
    out_bias = None

    def __init__(self, width: int, ff: int, choice: Choice, dtype, device):
        super().__init__(dtype, device)
        if ff < 1:
            raise ValueError("feed-forward: ff must be positive")
        self.width, self.ff, self.choice = width, ff, choice
        E, F, K = choice.experts, pad_to(ff), pad_to(width)
        self.w_router, self.correction = self._zeros(pad_to(E, 8), K), self._zeros(E, dtype=torch.float32)
        self.w_up, self.w_down = self._zeros(E, F, K), self._zeros(E, width, F)

    def logical_shapes(self):
        E = self.choice.experts
        out = {"router": (E, self.width), "correction": (E,)}
        for e in range(E):
            out[f"e{e}.up"], out[f"e{e}.down"] = (self.ff, self.width), (self.width, self.ff)
        return out

    def _pack(self, t):
        self.w_router[:self.choice.experts, :self.width].copy_(t["router"])
        self.correction.copy_(t["correction"])
        for e in range(self.choice.experts):
            self.w_up[e, :self.ff, :self.width].copy_(t[f"e{e}.up"])
            self.w_down[e, :, :self.ff].copy_(t[f"e{e}.down"])

    def unpack(self):
        out = {"router": self.w_router[:self.choice.experts, :self.width].contiguous(), "correction": self.correction.to(self.dtype)}
        for e in range(self.choice.experts):
            out[f"e{e}.up"] = self.w_up[e, :self.ff, :self.width].contiguous()
            out[f"e{e}.down"] = self.w_down[e, :, :self.ff].contiguous()
        return out

    def forward(self, h):
        return relu2_experts(h, router_logits(h, self.w_router), self.correction, self.choice, self.w_up, self.w_down)


def _head_rows(at: int, heads: int, stride: int, columns: torch.Tensor) -> torch.Tensor:
    """Packed row of every coordinate of a section of heads: ``columns`` places a head's coordinates inside its ``stride``."""
    return (at + torch.arange(heads)[:, None] * stride + columns[None, :]).reshape(-1)


class _RowPacked(_Mixer):
    """A mixer whose projections are rows of ``w_in`` at places given by index (``_rows``: name -> packed row of every logical
    row), and whose output product reads columns ``_out_columns()``."""

    def _pack_rows(self, t):
        for name, rows in self._rows().items():
            self.w_in[rows.to(self.device), :self.width] = t[name].to(self.device, self.dtype)
        self.w_out[:, self._out_columns().to(self.device)] = t["o"].to(self.device, self.dtype)

    def _unpack_rows(self):
        out = {name: self.w_in[rows.to(self.device), :self.width] for name, rows in self._rows().items()}
        out["o"] = self.w_out[:, self._out_columns().to(self.device)]
        return out

    def _row_shapes(self):
        out = {name: (len(rows), self.width) for name, rows in self._rows().items()}
        out["o"] = (self.width, len(self._out_columns()))
        return out


class LatentAttention(_RowPacked):
    """Attention whose keys and values are products of a cached latent, with a rotated key part shared by all heads and a
    sigmoid gate on the heads (see ``ops.latent``)."""
    takes_in_scale = True
    masks = (0,)

    def __init__(self, width: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, scale: float, rotary: Rotary, eps: float,
                 dtype, device):
        super().__init__(dtype, device)
        self.width = width
        self.geo = g = LatentGeometry(heads, dim, rot_dim, vdim, kv_rank, rotary)
        self.w_in, self.w_out = self._zeros(g.cols, pad_to(width)), self._zeros(width, g.out_cols)
        self.w = LatentWeights(self._zeros(g.cp, dtype=torch.float32), self._zeros(2 * heads * g.D, g.row),
                               self._zeros(heads, g.cp, pad_to(dim)), float(eps), float(scale))
        # the rows that copy the rotated part of a cached row into every head's key
        up = self.w.w_up[:heads * g.D].view(heads, g.D, g.row)
        for j in range(2 * rotary.hp):
            up[:, g.np + j, g.cp + j] = 1.0

    def tensors(self):
        return super().tensors() + [self.w.norm, self.w.w_up, self.w.w_absorb]

    def run_spec(self) -> LatentRun:
        return LatentRun(self.geo.row, self.geo.rotary)

    def _rows(self):
        g = self.geo
        rot = g.rotary.columns(g.rot_dim)
        head = torch.cat([torch.arange(g.dim), g.np + rot])
        down = torch.cat([torch.arange(g.kv_rank), pad_to(g.kv_rank, 8) + rot])
        return {"q": _head_rows(0, g.heads, g.q_cols, head), "dkv": g.off_c + down,
                "g": _head_rows(g.off_gate, g.heads, g.vp, torch.arange(g.vdim))}

    def _out_columns(self):
        return _head_rows(0, self.geo.heads, self.geo.vp, torch.arange(self.geo.vdim))

    def logical_shapes(self):
        g = self.geo
        return {**self._row_shapes(), "dkv.norm": (g.kv_rank,), "uk": (g.heads * g.dim, g.kv_rank), "uv": (g.heads * g.vdim, g.kv_rank)}

    def _up_views(self):
        g = self.geo
        up = self.w.w_up.view(2, g.heads, g.D, g.row)
        return up[0, :, :g.dim, :g.kv_rank], up[1, :, :g.vdim, :g.kv_rank]

    def _pack(self, t):
        g = self.geo
        self._pack_rows(t)
        self.w.norm[:g.kv_rank].copy_(t["dkv.norm"])
        k, v = self._up_views()
        k.copy_(t["uk"].view(g.heads, g.dim, g.kv_rank))
        v.copy_(t["uv"].view(g.heads, g.vdim, g.kv_rank))
        self.w.w_absorb[:, :g.kv_rank, :g.dim].copy_(t["uk"].view(g.heads, g.dim, g.kv_rank).transpose(1, 2))

    def unpack(self):
        g = self.geo
        k, v = self._up_views()
        return {**self._unpack_rows(), "dkv.norm": self.w.norm[:g.kv_rank].to(self.dtype), "uk": k.reshape(-1, g.kv_rank),
                "uv": v.reshape(-1, g.kv_rank)}

    def core(self, proj, storage, batch, out=None):
        return latent_attention(proj, self.geo, self.w, storage[0], storage[1], batch, self.in_scale, out)


class Retention(_RowPacked):
    """Linear attention with a fixed decay per head (see ``ops.retention``)."""
    takes_in_scale = True
    tile = SPAN

    def __init__(self, width: int, heads: int, dim: int, vdim: int, decay, rotary: Rotary, eps: float, dtype, device):
        super().__init__(dtype, device)
        if len(decay) != heads:
            raise ValueError("retention: one decay per head")
        self.width, self.eps = width, float(eps)
        self.geo = g = RetentionGeometry(heads, dim, vdim, rotary)
        self.w_in, self.w_out = self._zeros(g.cols, pad_to(width)), self._zeros(width, g.out_cols)
        self.log2_decay = log2_decays(decay).to(self.device)

    def run_spec(self) -> StateRun:
        g = self.geo
        return StateRun((g.heads, g.dp, g.vp), rotary=g.rotary)

    def _rows(self):
        g = self.geo
        qk, v = g.rotary.columns(g.dim), torch.arange(g.vdim)
        return {"q": _head_rows(0, g.heads, g.dp, qk), "k": _head_rows(g.off_k, g.heads, g.dp, qk),
                "v": _head_rows(g.off_v, g.heads, g.vp, v), "g": _head_rows(g.off_gate, g.heads, g.vp, v)}

    def _out_columns(self):
        return _head_rows(0, self.geo.heads, self.geo.vp, torch.arange(self.geo.vdim))

    def logical_shapes(self):
        return self._row_shapes()

    def _pack(self, t):
        self._pack_rows(t)

    def unpack(self):
        return self._unpack_rows()

    def core(self, proj, storage, batch, out=None):
        return retention(proj, self.geo, self.log2_decay, self.eps, storage[0], storage[1], batch, self.in_scale, out)


class RGLRU(_RowPacked):
    """A short convolution and a real-gated linear recurrence, times a GELU branch (see ``ops.rglru``)."""
    takes_in_scale = True
    tile = CHUNK
    _vectors = ("x_bias", "y_bias", "conv_b", "ra_b", "ri_b", "decay")

    def __init__(self, width: int, channels: int, blocks: int, conv: int, dtype, device):
        super().__init__(dtype, device)
        self.width = width
        self.geo = g = RGLRUGeometry(channels, blocks, conv)
        self.w_in, self.w_out = self._zeros(g.cols, pad_to(width)), self._zeros(width, g.out_cols)
        vec = {n: self._zeros(g.channels, dtype=torch.float32) for n in self._vectors}
        self.w = RGLRUWeights(conv=self._zeros(conv, g.channels, dtype=torch.float32), ra=self._zeros(blocks, g.kp, g.kp),
                              ri=self._zeros(blocks, g.kp, g.kp), **vec)
        self.lam = self._zeros(channels, dtype=torch.float32)

    def tensors(self):
        return super().tensors() + [t for t in vars(self.w).values()]

    def run_spec(self) -> StateRun:
        g = self.geo
        return StateRun((g.channels,), (g.taps - 1, g.channels))

    def _rows(self):
        c = self.geo.columns()
        return {"x": c, "y": self.geo.channels + c}

    def _out_columns(self):
        return self.geo.columns()

    def logical_shapes(self):
        g = self.geo
        return {**self._row_shapes(), "x.b": (g.width,), "y.b": (g.width,), "conv": (g.width, g.taps), "conv.b": (g.width,),
                "ra": (g.blocks, g.k, g.k), "ra.b": (g.blocks, g.k), "ri": (g.blocks, g.k, g.k), "ri.b": (g.blocks, g.k),
                "lam": (g.width,)}

    def _pack(self, t):
        g, w = self.geo, self.w
        self._pack_rows(t)
        c = g.columns().to(self.device)
        put = lambda dst, src: dst.__setitem__(c, src.to(self.device).float().reshape(-1))   # noqa: E731
        put(w.x_bias, t["x.b"])
        put(w.y_bias, t["y.b"])
        put(w.conv_b, t["conv.b"])
        put(w.ra_b, t["ra.b"])
        put(w.ri_b, t["ri.b"])
        put(w.decay, 8.0 * torch.nn.functional.softplus(t["lam"].double(), threshold=700.0))
        w.conv[:, c] = t["conv"].to(self.device).float().t()
        w.ra[:, :g.k, :g.k].copy_(t["ra"])
        w.ri[:, :g.k, :g.k].copy_(t["ri"])
        self.lam.copy_(t["lam"])

    def unpack(self):
        g, w, c = self.geo, self.w, self.geo.columns().to(self.device)
        get = lambda v: v[c].to(self.dtype)   # noqa: E731
        return {**self._unpack_rows(), "x.b": get(w.x_bias), "y.b": get(w.y_bias), "conv": w.conv[:, c].t().contiguous().to(self.dtype),
                "conv.b": get(w.conv_b), "ra": w.ra[:, :g.k, :g.k].contiguous(), "ra.b": get(w.ra_b).view(g.blocks, g.k),
                "ri": w.ri[:, :g.k, :g.k].contiguous(), "ri.b": get(w.ri_b).view(g.blocks, g.k), "lam": self.lam.to(self.dtype)}

    def core(self, proj, storage, batch, out=None):
        return rglru(proj, self.geo, self.w, storage[0], storage[1], batch, self.in_scale, out)


class ShapedAttention(_RowPacked):
    """Grouped-query attention whose parts can be chosen (see ``ops.ragged``): biases on the projections, values of their own or the
    keys as projected, a norm of q and k, rotation, queries that grow with the position, a mask, what becomes of the scores, values mixed
    with those of the model's first such layer, a gate per head or per element, a bias on the result."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, form: ScoreForm, eps: float, dtype, device, bias: bool = False,
                 keys_as_values: bool = False, norm: str = "", rotary: Optional[Rotary] = None, learned_sink: bool = False, v_mix: bool = False,
                 gate: str = "", q_temp: Optional[tuple] = None, out_bias: bool = False):
        super().__init__(dtype, device)
        self.width, self.v_mix, self.learned_sink = width, bool(v_mix), bool(learned_sink)
        self.geo = g = AttentionGeometry(heads, kv_heads, dim, vdim, dtype, rotary, keys_as_values, gate)
        self.w_in, self.w_out = self._zeros(g.cols, pad_to(width)), self._zeros(width, g.out_cols)
        vec = lambda n: self._zeros(n, dtype=torch.float32)   # noqa: E731
        form.slopes, form.sink = (t.to(self.device) if t is not None else None for t in (form.slopes, form.sink))
        if learned_sink:
            form.sink = vec(heads)
        sizes = {"head": (g.D, g.D), "whole": (heads * g.D, kv_heads * g.D)}.get(norm)
        if norm not in ("", "unit", "head", "whole"):
            raise ValueError(f"attention: unknown norm {norm!r}")
        self.w = AttentionWeights(form, vec(g.off_gate) if bias else None, norm, vec(sizes[0]) if sizes else None,
                                  vec(sizes[1]) if sizes else None, float(eps), q_temp=q_temp)
        if out_bias:
            self.out_bias = vec(width)
        self.masks = (form.mask,)
        if norm == "unit":
            form.product_bound = 1.02 * dim               # (two unit vectors times sqrt(dim), rounded)

    def tensors(self):
        w = self.w
        return super().tensors() + [t for t in (w.bias, w.q_norm, w.k_norm, w.form.slopes, w.form.sink) if t is not None]

    def run_spec(self) -> PagedRun:
        return PagedRun(self.geo.kv_heads, self.geo.D, self.geo.rotary, self.v_mix)

    def _rows(self):
        g = self.geo
        qk, v = g.columns(), torch.arange(g.vdim)
        out = {"q": _head_rows(0, g.heads, g.D, qk), "k": _head_rows(g.off_k, g.kv_heads, g.D, qk)}
        if not g.keys_as_values:
            out["v"] = _head_rows(g.off_v, g.kv_heads, g.D, v)
        if g.gate:
            out["g"] = g.off_gate + torch.arange(g.heads) if g.gate == "head" else _head_rows(g.off_gate, g.heads, g.D, v)
        return out

    def _out_columns(self):
        return _head_rows(0, self.geo.heads, self.geo.D, torch.arange(self.geo.vdim))

    def _vectors(self):
        """name -> (fp32 vector, its places)"""
        g, w, rows, out = self.geo, self.w, self._rows(), {}
        if w.bias is not None:
            out.update({n + ".b": (w.bias, rows[n]) for n in "qkv" if n in rows})
        if w.norm == "head":
            out.update({"q.norm": (w.q_norm, g.columns()), "k.norm": (w.k_norm, g.columns())})
        elif w.norm == "whole":
            out.update({"q.norm": (w.q_norm, rows["q"]), "k.norm": (w.k_norm, rows["k"] - g.off_k)})
        if self.learned_sink:
            out["sink"] = (w.form.sink, torch.arange(g.heads))
        if self.out_bias is not None:
            out["o.b"] = (self.out_bias, torch.arange(self.width))
        return out

    def logical_shapes(self):
        out = {**self._row_shapes(), **{n: (len(at),) for n, (_, at) in self._vectors().items()}}
        if self.v_mix:
            out["vmix"] = ()
        return out

    def _pack(self, t):
        self._pack_rows(t)
        for n, (vec, at) in self._vectors().items():
            vec[at.to(self.device)] = t[n].to(self.device).float()
        if self.v_mix:
            self.w.vmix = float(t["vmix"])

    def unpack(self):
        out = {**self._unpack_rows(), **{n: vec[at.to(self.device)].to(self.dtype) for n, (vec, at) in self._vectors().items()}}
        if self.v_mix:
            out["vmix"] = torch.tensor(self.w.vmix, dtype=self.dtype, device=self.device)
        return out

    def core(self, proj, storage, batch, out=None):
        k, v, angles, first = storage if len(storage) == 4 else (*storage, None, None)
        return shaped_attention(proj, self.geo, self.w, k, v, angles, first, batch, self.out_scale, out)


class TimeMix(_RowPacked):
    """Linear attention with a decay per channel and token, fed by mixes of a token's input and the one before (see
    ``ops.timemix``)."""
    tile = STATE_SPAN

    def __init__(self, width: int, heads: int, dim: int, rank: int, eps: float, dtype, device):
        super().__init__(dtype, device)
        self.width = width
        self.geo = g = TimeMixGeometry(heads, dim, rank)
        self.streams = g.starts
        self.w_in, self.w_out = self._zeros(g.cols, pad_to(width)), self._zeros(width, g.out_cols)
        f32, n = torch.float32, heads * g.dp
        self.mu = self._zeros(len(STREAMS), pad_to(width), dtype=f32)
        self.w = TimeMixWeights(self._zeros(n, g.rp), self._zeros(n, dtype=f32), self._zeros(n, dtype=f32), self._zeros(n, dtype=f32), float(eps))

    def tensors(self):
        return super().tensors() + [self.w.w2, self.w.w0, self.w.u, self.w.norm]

    def run_spec(self) -> StateRun:
        g = self.geo
        return StateRun((g.heads, g.dp, g.dp), (1, pad_to(self.width)))

    def _rows(self):
        g = self.geo
        head = lambda i: _head_rows(i * g.section, g.heads, g.dp, torch.arange(g.dim))   # noqa: E731
        return {"r": head(0), "k": head(1), "v": head(2), "g": head(3), "w1": 4 * g.section + torch.arange(g.rank)}

    def _out_columns(self):
        return _head_rows(0, self.geo.heads, self.geo.dp, torch.arange(self.geo.dim))

    def logical_shapes(self):
        g, n = self.geo, self.geo.heads * self.geo.dim
        return {**{"mu." + s: (self.width,) for s in STREAMS}, **self._row_shapes(), "w2": (n, g.rank), "w0": (n,), "u": (g.heads, g.dim),
                "norm": (n,)}

    def _pack(self, t):
        self._pack_rows(t)
        for i, s in enumerate(STREAMS):
            self.mu[i, :self.width].copy_(t["mu." + s])
        at = self._out_columns().to(self.device)
        self.w.w2[at, :self.geo.rank] = t["w2"].to(self.device, self.dtype)
        for n in ("w0", "u", "norm"):
            getattr(self.w, n)[at] = t[n].to(self.device).float().reshape(-1)

    def unpack(self):
        g, at = self.geo, self._out_columns().to(self.device)
        out = {**self._unpack_rows(), **{"mu." + s: self.mu[i, :self.width].to(self.dtype) for i, s in enumerate(STREAMS)},
               "w2": self.w.w2[at, :g.rank]}
        out.update({n: getattr(self.w, n)[at].to(self.dtype) for n in ("w0", "u", "norm")})
        out["u"] = out["u"].view(g.heads, g.dim)
        return out

    def mix_inputs(self, h, storage, batch, keep=False):
        return token_shift(h, self.mu, storage[0], batch, keep)

    def core(self, proj, storage, batch, out=None):
        return time_mix(proj, self.geo, self.w, storage[1], batch, self.out_scale, out)


class GatedLinear(_RowPacked):
    """Gated linear attention: a decay per key channel from a product of low rank (see ``ops.timemix.gated_linear``)."""
    tile = STATE_SPAN

    def __init__(self, width: int, heads: int, dim: int, vdim: int, rank: int, tau: float, eps: float, dtype, device):
        super().__init__(dtype, device)
        if tau <= 0:
            raise ValueError("gated linear attention: tau must be positive")
        self.width = width
        self.geo = g = GatedLinearGeometry(heads, dim, vdim, rank)
        self.w_in, self.w_out = self._zeros(g.cols, pad_to(width)), self._zeros(width, g.out_cols)
        f32 = torch.float32
        self.w = GatedLinearWeights(self._zeros(heads * g.dp, g.rp), self._zeros(heads * g.dp, dtype=f32), self._zeros(heads * g.ep, dtype=f32),
                                    float(tau), float(eps))

    def tensors(self):
        return super().tensors() + [self.w.w2, self.w.w0, self.w.norm]

    def run_spec(self) -> StateRun:
        g = self.geo
        return StateRun((g.heads, g.ep, g.dp))

    def _keys(self, at=0):
        return _head_rows(at, self.geo.heads, self.geo.dp, torch.arange(self.geo.dim))

    def _values(self, at=0):
        return _head_rows(at, self.geo.heads, self.geo.ep, torch.arange(self.geo.vdim))

    def _rows(self):
        g = self.geo
        return {"q": self._keys(), "k": self._keys(g.off_k), "v": self._values(g.off_v), "g": self._values(g.off_gate),
                "a1": g.off_low + torch.arange(g.rank)}

    def _out_columns(self):
        return self._values()

    def logical_shapes(self):
        g = self.geo
        return {**self._row_shapes(), "norm": (g.vdim,), "a2": (g.heads * g.dim, g.rank), "a2.b": (g.heads * g.dim,)}

    def _pack(self, t):
        g, at = self.geo, self._keys().to(self.device)
        self._pack_rows(t)
        self.w.w2[at, :g.rank] = t["a2"].to(self.device, self.dtype)
        self.w.w0[at] = t["a2.b"].to(self.device).float()
        self.w.norm.view(g.heads, g.ep)[:, :g.vdim] = t["norm"].to(self.device).float()

    def unpack(self):
        g, at = self.geo, self._keys().to(self.device)
        return {**self._unpack_rows(), "norm": self.w.norm[:g.vdim].to(self.dtype), "a2": self.w.w2[at, :g.rank], "a2.b": self.w.w0[at].to(self.dtype)}

    def core(self, proj, storage, batch, out=None):
        return gated_linear(proj, self.geo, self.w, storage[0], batch, self.out_scale, out)


class SSD(_RowPacked):
    """State-space duality with a short convolution, normed in parts after its gate (see ``ops.ssd``)."""
    tiles = (CONV_TILE, STATE_SPAN)

    def __init__(self, width: int, heads: int, vdim: int, state: int, groups: int, conv: int, norm_parts: int, eps: float, dtype, device):
        super().__init__(dtype, device)
        self.width = width
        self.geo = g = SSDGeometry(heads, vdim, state, groups, conv, norm_parts)
        self.w_in, self.w_out = self._zeros(g.cols, pad_to(width)), self._zeros(width, g.out_cols)
        vec = lambda *n: self._zeros(*n, dtype=torch.float32)   # noqa: E731
        self.w = SSDWeights(vec(conv, g.conv_cols), vec(g.conv_cols), vec(heads), vec(heads), vec(heads), vec(heads * g.vp), float(eps))

    def tensors(self):
        return super().tensors() + [t for t in vars(self.w).values() if isinstance(t, torch.Tensor)]

    def run_spec(self) -> StateRun:
        g = self.geo
        return StateRun((g.heads, g.vp, g.np), (g.taps - 1, g.conv_cols))

    def _inner(self, at):
        return _head_rows(at, self.geo.heads, self.geo.vp, torch.arange(self.geo.vdim))

    def _rows(self):
        g = self.geo
        group = lambda at: _head_rows(at, g.groups, g.np, torch.arange(g.state))   # noqa: E731
        return {"in": torch.cat([self._inner(0), self._inner(g.off_x), group(g.off_b), group(g.off_c), g.off_dt + torch.arange(g.heads)])}

    def _conv_columns(self):
        g, rows = self.geo, self._rows()["in"]
        return rows[g.heads * g.vdim:len(rows) - g.heads] - g.off_x

    def _out_columns(self):
        return self._inner(0)

    def logical_shapes(self):
        g = self.geo
        n = len(self._conv_columns())
        return {**self._row_shapes(), "conv": (n, g.taps), "conv.b": (n,), "dt_bias": (g.heads,), "A_log": (g.heads,), "D": (g.heads,),
                "norm": (g.heads * g.vdim,)}

    def _pack(self, t):
        w, c, at = self.w, self._conv_columns().to(self.device), self._out_columns().to(self.device)
        self._pack_rows(t)
        w.conv[:, c] = t["conv"].to(self.device).float().t()
        w.conv_b[c] = t["conv.b"].to(self.device).float()
        w.norm[at] = t["norm"].to(self.device).float()
        for vec, n in ((w.dt_bias, "dt_bias"), (w.a_log, "A_log"), (w.d, "D")):
            vec.copy_(t[n])

    def unpack(self):
        w, c, at = self.w, self._conv_columns().to(self.device), self._out_columns().to(self.device)
        return {**self._unpack_rows(), "conv": w.conv[:, c].t().contiguous().to(self.dtype), "conv.b": w.conv_b[c].to(self.dtype),
                "norm": w.norm[at].to(self.dtype), "dt_bias": w.dt_bias.to(self.dtype), "A_log": w.a_log.to(self.dtype), "D": w.d.to(self.dtype)}

    def core(self, proj, storage, batch, out=None):
        return ssd(proj, self.geo, self.w, storage[0], storage[1], batch, self.out_scale, out)


class SideBySide(_Mixer):
    """left_scale left(h) + right_scale right(h): one product feeds both cores, one takes both results back and sums them. Tensors
    are the parts' own, under "left." and "right."."""

    def __init__(self, left: _Mixer, right: _Mixer, left_scale: float, right_scale: float, width: int, dtype, device):
        super().__init__(dtype, device)
        if len(left.streams) > 1:
            raise ValueError("side by side: the mixer that makes its own inputs is the right one")
        self.left, self.right = left, right
        left.out_scale, right.out_scale = float(left_scale), float(right_scale)
        own = len(right.streams) > 1
        self.cut = input_columns(left.cols) if own else pad_to(left.cols, 8)
        self.streams = (0,) + tuple(self.cut + s for s in right.streams) if own else (0,)
        self.w_in, self.w_out = self._zeros(self.cut + right.cols, pad_to(width)), self._zeros(width, left.out_cols + right.out_cols)
        left.place(self.w_in[:left.cols], self.w_out[:, :left.out_cols])
        right.place(self.w_in[self.cut:], self.w_out[:, left.out_cols:])
        self.masks = left.masks + right.masks
        if any(p.out_bias is not None for p in (left, right)):
            self.out_bias = self._zeros(width, dtype=torch.float32)

    @property
    def tiles(self) -> tuple:
        return self.left.tiles + self.right.tiles

    def tensors(self):
        parts = [t for p in (self.left, self.right) for t in p.tensors() if t is not p.w_in and t is not p.w_out]
        return super().tensors() + parts

    def run_spec(self) -> PairRun:
        return PairRun(self.left.run_spec(), self.right.run_spec())

    def _both(self):
        return (("left.", self.left), ("right.", self.right))

    def logical_shapes(self):
        return {pre + n: s for pre, p in self._both() for n, s in p.logical_shapes().items()}

    def _pack(self, t):
        for pre, p in self._both():
            p._pack({n: t[pre + n] for n in p.logical_shapes()})
        if self.out_bias is not None:
            self.out_bias.zero_()
            for _, p in self._both():
                if p.out_bias is not None:
                    self.out_bias += p.out_scale * p.out_bias

    def unpack(self):
        return {pre + n: v for pre, p in self._both() for n, v in p.unpack().items()}

    def mix_inputs(self, h, storage, batch):
        return self.right.mix_inputs(h, storage[1], batch, keep=True)

    def core(self, proj, storage, batch, out=None):
        z = out if out is not None else torch.empty((proj.shape[0], self.out_cols), device=proj.device, dtype=proj.dtype)
        k = self.left.out_cols
        self.left.core(proj[:, :self.left.cols], storage[0], batch, out=z[:, :k])
        self.right.core(proj[:, self.cut:], storage[1], batch, out=z[:, k:])
        return z


class TokenSide(_Packed):
    """A side input per token and layer: y = W_proj (gelu_tanh(W_gate x) * e), e the token's row of a table; x + y / rms(y) *
    norm."""

    def __init__(self, width: int, dim: int, eps: float, dtype, device):
        super().__init__(dtype, device)
        self.width, self.dim = width, dim
        self.w_gate, self.w_proj = self._zeros(pad_to(dim), pad_to(width)), self._zeros(width, pad_to(dim))
        self.norm = RMSNorm(width, eps, 0.0, dtype, device)

    def tensors(self):
        return super().tensors() + self.norm.tensors()

    def logical_shapes(self):
        return {"gate": (self.dim, self.width), "proj": (self.width, self.dim), "norm": (self.width,)}

    def _pack(self, t):
        self.w_gate[:self.dim, :self.width].copy_(t["gate"])
        self.w_proj[:, :self.dim].copy_(t["proj"])
        self.norm._pack({"": t["norm"]})

    def unpack(self):
        return {"gate": self.w_gate[:self.dim, :self.width].contiguous(), "proj": self.w_proj[:, :self.dim].contiguous(),
                "norm": self.norm.unpack()[""]}

    def forward(self, h, tokens, table, first: int):
        """What is normed and added; ``table`` [vocab, ..], this layer's part from column ``first`` on."""
        return ops.project(ops.gelu_lookup(ops.project(h, self.w_gate), tokens, table, first, self.dim), self.w_proj)
