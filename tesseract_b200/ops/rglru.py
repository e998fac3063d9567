"""Real-gated linear recurrent unit over ragged batches (``csrc/rglru.cu``). Per channel, after a short causal convolution
u of the x projection:

    r = sigmoid(ra u + ra_b), i = sigmoid(ri u + ri_b)        (ra, ri block-diagonal)
    a = exp(-8 softplus(lam) r);  S <- a S + sqrt(1 - a^2) i u;  out = S gelu(y)

``rglru`` takes the packed projection [x | y] (decoded rows first, then portions of prompts), advances the slots of a state
pool and returns the gated states. CPU tensors run the torch restatement below.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr

P, I, L, F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({"tsb_rglru": [P, F, P, L] + [P] * 23 + [L, I, P]})

CHUNK = 64          # tokens of a portion that the gates are computed for at once


@dataclass(frozen=True)
class RGLRUGeometry:
    """``width`` channels in ``blocks`` parts, each padded to ``kp`` columns; a channel has the same column in x, y, the
    convolution, the state and the result."""
    width: int
    blocks: int
    taps: int

    def __post_init__(self):
        if min(self.width, self.blocks, self.taps) < 1 or self.width % self.blocks:
            raise ValueError("rglru: positive sizes, and width a multiple of blocks")

    @property
    def k(self) -> int:
        return self.width // self.blocks

    @property
    def kp(self) -> int:
        return (self.k + 15) // 16 * 16

    @property
    def channels(self) -> int:
        return self.blocks * self.kp

    @property
    def cols(self) -> int:
        return 2 * self.channels

    out_cols = channels

    def columns(self) -> torch.Tensor:
        """Column of every logical channel."""
        c = torch.arange(self.width)
        return c // self.k * self.kp + c % self.k


@dataclass
class RGLRUWeights:
    """fp32 except the gate matrices ra, ri [blocks, kp, kp] (out, in; the projection's dtype): biases [channels], convolution
    [taps, channels] and its bias, ``decay`` = 8 softplus(lam) [channels]."""
    x_bias: torch.Tensor
    y_bias: torch.Tensor
    conv: torch.Tensor
    conv_b: torch.Tensor
    ra: torch.Tensor
    ri: torch.Tensor
    ra_b: torch.Tensor
    ri_b: torch.Tensor
    decay: torch.Tensor


def rglru(proj: torch.Tensor, geo: RGLRUGeometry, w: RGLRUWeights, conv_state: torch.Tensor, state: torch.Tensor, batch,
          in_scale: float = 1.0, out: torch.Tensor | None = None) -> torch.Tensor:
    """proj [T, geo.cols] of a ragged batch -> [T, channels] (``out`` may be columns of a wider matrix). ``conv_state`` [slots,
    taps - 1, channels] (projection dtype) and ``state`` [slots, channels] (fp32) are advanced in place; a sequence whose
    first row is at position 0 starts from zeros whatever its slot holds. ``in_scale`` multiplies the projection before its
    biases."""
    T, C, dev = proj.shape[0], geo.channels, proj.device
    if out is None:
        out = torch.empty((T, C), device=dev, dtype=proj.dtype)
    if T == 0:
        return out
    if not proj.is_cuda:
        return _rglru_torch(proj, geo, w, conv_state, state, batch, in_scale, out)
    nd, n = batch.n_decode, T - batch.n_decode
    tiles = batch.tiles(CHUNK) if n else None
    chunks = tiles.n if n else 0
    f32 = dict(device=dev, dtype=torch.float32)
    u = torch.empty((T, C), device=dev, dtype=proj.dtype)
    s_local, a_prod, carry = (torch.empty((r, C), **f32) for r in (n, n, chunks)) if n else (None, None, None)
    ptr = lambda t: t.data_ptr() if t is not None else None   # noqa: E731
    v = (geo.blocks, geo.kp, C, geo.taps, T, nd, batch.n_prompts if n else 0, chunks)
    check(lib().tsb_rglru((ctypes.c_int * len(v))(*v), float(in_scale), proj.data_ptr(), proj.stride(0), w.x_bias.data_ptr(),
                          w.y_bias.data_ptr(), w.conv.data_ptr(), w.conv_b.data_ptr(), w.ra.data_ptr(), w.ri.data_ptr(),
                          w.ra_b.data_ptr(), w.ri_b.data_ptr(), w.decay.data_ptr(), conv_state.data_ptr(), state.data_ptr(),
                          batch.state_slots.data_ptr(), batch.positions.data_ptr(), ptr(batch.seq_of) if n else None,
                          ptr(batch.cu) if n else None, ptr(batch.pos0) if n else None, ptr(tiles.seq) if n else None,
                          ptr(tiles.first) if n else None, u.data_ptr(), ptr(s_local), ptr(a_prod), ptr(carry), out.data_ptr(),
                          out.stride(0), dtype_code(proj.dtype), stream_ptr(dev)), "tsb_rglru")
    _native.add_launches((1 if nd else 0) + ((4 if geo.taps > 1 else 3) if n else 0))
    return out


def _rglru_torch(proj, geo, w, conv_state, state, batch, in_scale, out):
    C, K, N = geo.channels, geo.taps, geo.blocks
    for row0, n, slot, pos0 in batch.spans():
        if slot < 0:
            out[row0:row0 + n] = 0
            continue
        p = proj[row0:row0 + n]
        raw = torch.cat([conv_state[slot], p[:, :C]], dim=0)
        x = raw.float() * in_scale + w.x_bias
        x[:max(K - 1 - pos0, 0)] = 0                           # before the start of the sequence
        conv_state[slot] = raw[n:]
        u = (sum(w.conv[j] * x[j:j + n] for j in range(K)) + w.conv_b).to(proj.dtype)
        ub = u.view(n, N, geo.kp).transpose(0, 1).float()

        def gate(m, b):
            return torch.sigmoid((ub @ m.float().transpose(1, 2)).transpose(0, 1).reshape(n, C) + b)
        log_a = -gate(w.ra, w.ra_b) * w.decay
        a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * gate(w.ri, w.ri_b) * u.float()
        S = state[slot].clone() if pos0 > 0 else torch.zeros(C)
        s = torch.empty(n, C)
        for t in range(n):
            S = a[t] * S + b[t]
            s[t] = S
        state[slot] = S
        y = torch.nn.functional.gelu(p[:, C:2 * C].float() * in_scale + w.y_bias, approximate="tanh")
        out[row0:row0 + n] = (s * y).to(out.dtype)
    return out
