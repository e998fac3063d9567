"""Building blocks of hybrid decoders for inference over ragged batches: Dynamic Tanh norms, chunked attention, the gated
delta rule and the clamped GLU feed-forward.

A block holds its parameters packed for the kernels (adjacent projections in one matrix, sections and heads padded with
zeros, everything that the kernels use in fp32 already widened) and translates to and from its logical tensors:
``logical_shapes`` names them, ``load`` packs a dict of them, ``unpack`` gives them back.
"""
from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..ops.delta import DeltaGeometry, DeltaWeights, gated_delta
from ..ops.ragged import padded_head_dim, ragged_attention
from .ragged import PagedRun, StateRun


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


class ChunkedAttention(_Packed):
    """Grouped-query attention without positions whose mask is causal inside runs of ``chunk`` positions (0: causal over
    everything); biases on q, k and v. Query / key heads are ``dim`` wide, value heads ``vdim``."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, chunk: int, dtype, device):
        super().__init__(dtype, device)
        if heads % kv_heads or min(heads, kv_heads, dim, vdim) < 1 or chunk < 0:
            raise ValueError("attention: positive sizes, and heads a multiple of kv_heads")
        self.width, self.heads, self.kv_heads, self.dim, self.vdim = width, heads, kv_heads, dim, vdim
        self.scale, self.chunk = float(scale), int(chunk)
        self.D = padded_head_dim(dim, vdim, dtype)
        self.w_in = self._zeros((heads + 2 * kv_heads) * self.D, pad_to(width))
        self.b_in = self._zeros((heads + 2 * kv_heads) * self.D, dtype=torch.float32)
        self.w_out = self._zeros(width, heads * self.D)

    out_bias = None

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

    def forward(self, h, storage, batch):
        qkv = ops.project(h, self.w_in)
        o = ragged_attention(qkv, self.b_in, storage[0], storage[1], batch, self.heads, self.kv_heads, self.scale, self.chunk)
        return ops.project(o, self.w_out)


class GatedDelta(_Packed):
    """The gated delta rule with short convolutions (see ``ops.delta``)."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, conv: int, eps: float, dtype, device):
        super().__init__(dtype, device)
        self.width = width
        self.geo = g = DeltaGeometry(kv_heads, heads, dim, vdim, conv)
        self.w_in = self._zeros(g.cols, pad_to(width))
        self.w_out = self._zeros(width, g.out_cols)
        f32 = torch.float32
        self.w = DeltaWeights(self._zeros(conv, g.conv_cols, dtype=f32), self._zeros(heads, dtype=f32),
                              self._zeros(heads, dtype=f32), self._zeros(vdim, dtype=f32), float(eps))

    out_bias = None

    def tensors(self):
        return super().tensors() + [self.w.conv, self.w.a_log, self.w.dt_bias, self.w.norm]

    def run_spec(self) -> StateRun:
        g = self.geo
        return StateRun((g.heads, g.dim, g.vdim_pad), (g.taps - 1, g.conv_cols))

    def _sections(self):
        g = self.geo
        qk, hv = g.kv_heads * g.dim, g.heads * g.vdim
        return (("q", 0, qk), ("k", g.off_k, qk), ("v", g.off_v, hv), ("g", g.off_gate, hv), ("b", g.off_b, g.heads),
                ("a", g.off_a, g.heads))

    def logical_shapes(self):
        g = self.geo
        out = {}
        for name, _, n in self._sections():
            out[name] = (n, self.width)
            if name in "qkv":
                out[name + ".conv"] = (n, g.taps)
        out.update({"A_log": (g.heads,), "dt_bias": (g.heads,), "norm": (g.vdim,), "o": (self.width, g.heads * g.vdim)})
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

    def unpack(self):
        out = {}
        for name, at, n in self._sections():
            out[name] = self.w_in[at:at + n, :self.width].contiguous()
            if name in "qkv":
                out[name + ".conv"] = self.w.conv[:, at:at + n].t().contiguous().to(self.dtype)
        out.update({"A_log": self.w.a_log.to(self.dtype), "dt_bias": self.w.dt_bias.to(self.dtype),
                    "norm": self.w.norm.to(self.dtype), "o": self.w_out[:, :self.geo.heads * self.geo.vdim].contiguous()})
        return out

    def forward(self, h, storage, batch):
        y = gated_delta(ops.project(h, self.w_in), self.geo, self.w, storage[0], storage[1], batch)
        return ops.project(y, self.w_out)


class ClampedGLU(_Packed):
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

    def forward(self, h):
        return ops.project(ops.clamped_glu(ops.project(h, self.w_in), self.b_in, self.limit, self.slope), self.w_out)
