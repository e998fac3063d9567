"""Gated delta rule over ragged batches (``csrc/delta_rule.cu``): per value head a state S [dim, vdim] with

    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q

fed by short causal convolutions of a packed projection and read out through a per-head RMS norm and a gate (SiLU or sigmoid).
The decay g is a number per head, from the projection, or a vector over the head's key channels, from a product of low rank, as the
gate then is. ``gated_delta`` takes the projection of a ragged batch (decoded rows first, then portions of prompts), advances the
slots of a state pool and returns the gated read-outs. CPU tensors run the torch restatement below.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr
from .gemm import project

P, I, L, F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({
    "tsb_delta_prefill": [P, L, P, P, L, P, L] + [P] * 17 + [L, I, I, I, I, I, F, I, P],
    "tsb_delta_step": [P, L, P, P, L, P, L] + [P] * 9 + [L, I, I, I, F, I, P],
})

MAX_TAPS = 8
MAX_DIM = 256


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class DeltaGeometry:
    """Sizes of one mixer and the layout of its packed projection row: [q | k | v | gate | b | a], every section padded to
    a multiple of 8 columns. With ``decay_rank`` and ``gate_rank`` the decays are per key channel, and both they and the gate are
    products of that many inputs: [q | k | v | b | decay inputs | gate inputs]."""
    kv_heads: int
    heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int = 0
    gate_rank: int = 0

    def __post_init__(self):
        if min(self.decay_rank, self.gate_rank) < 0 or (self.decay_rank > 0) != (self.gate_rank > 0):
            raise ValueError("delta rule: decays per channel and their gate come together")
        if min(self.kv_heads, self.heads, self.dim, self.vdim, self.taps) < 1 or self.heads % self.kv_heads:
            raise ValueError("delta rule: positive sizes, and heads a multiple of kv_heads")
        if self.dim > MAX_DIM or self.taps > MAX_TAPS:
            raise ValueError(f"delta rule: dim <= {MAX_DIM} and at most {MAX_TAPS} convolution taps")

    @property
    def dim_pad(self) -> int:
        return next(d for d in (32, 64, 128, 256) if d >= self.dim)

    @property
    def vdim_pad(self) -> int:
        return _up(self.vdim, 4)

    @property
    def off_k(self) -> int:
        return _up(self.kv_heads * self.dim, 8)

    @property
    def off_v(self) -> int:
        return 2 * self.off_k

    @property
    def channels(self) -> bool:
        return self.decay_rank > 0

    @property
    def conv_cols(self) -> int:
        return self.off_v + _up(self.heads * self.vdim, 8)

    @property
    def off_gate(self) -> int:
        return self.conv_cols

    @property
    def off_b(self) -> int:
        return self.conv_cols + (0 if self.channels else _up(self.heads * self.vdim, 8))

    @property
    def off_a(self) -> int:
        """Decays, or their inputs."""
        return self.off_b + _up(self.heads, 8)

    @property
    def decay_inputs(self) -> int:
        return _up(self.decay_rank, 16)

    @property
    def off_low_gate(self) -> int:
        return self.off_a + self.decay_inputs

    @property
    def cols(self) -> int:
        return self.off_low_gate + _up(self.gate_rank, 16) if self.channels else self.off_a + _up(self.heads, 8)

    @property
    def out_cols(self) -> int:
        return _up(self.heads * self.vdim, 16)

    def as_ints(self):
        v = (self.kv_heads, self.heads, self.dim, self.vdim, self.dim_pad, self.vdim_pad, self.off_k, self.off_v, self.off_b, self.off_a,
             self.conv_cols, int(self.channels))
        return (ctypes.c_int * len(v))(*v)


@dataclass
class DeltaWeights:
    """fp32 parameters of the mixer besides its projections: convolution taps [taps, conv_cols], A_log [heads], dt_bias [heads] or,
    with decays per channel, [heads * dim], norm [vdim]. In the model's type, with decays per channel: ``w_decay`` [heads * dim, decay
    inputs] and ``w_gate`` [heads * vdim, gate inputs], rows padded to multiples of 8."""
    conv: torch.Tensor
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    norm: torch.Tensor
    eps: float
    w_decay: torch.Tensor | None = None
    w_gate: torch.Tensor | None = None


def _side(proj, geo: DeltaGeometry, w: DeltaWeights):
    """(gate [T, >= heads * vdim], inputs of the decays [T, >= heads * dim] in fp32 or None)."""
    if not geo.channels:
        return proj[:, geo.off_gate:], None
    return (project(proj[:, geo.off_low_gate:geo.cols], w.w_gate),
            project(proj[:, geo.off_a:geo.off_low_gate], w.w_decay, out_dtype=torch.float32))


def gated_delta(proj: torch.Tensor, geo: DeltaGeometry, w: DeltaWeights, conv_state: torch.Tensor, state: torch.Tensor,
                batch, out: torch.Tensor | None = None) -> torch.Tensor:
    """proj [T, geo.cols] of a ragged batch -> [T, geo.out_cols]. ``conv_state`` [slots, taps - 1, conv_cols] (projection
    dtype) and ``state`` [slots, heads, dim, vdim_pad] (fp32) are advanced in place for the batch's sequences; a sequence
    whose first row is at position 0 starts from zeros whatever its slot holds."""
    T = proj.shape[0]
    y = out if out is not None else torch.empty((T, geo.out_cols), device=proj.device, dtype=proj.dtype)
    if T == 0:
        return y
    gate, dec = _side(proj, geo, w)
    if not proj.is_cuda:
        return _gated_delta_torch(proj, gate, dec, geo, w, conv_state, state, batch, y)
    nd = batch.n_decode
    g = geo.as_ints()
    dt, st = dtype_code(proj.dtype), stream_ptr(proj.device)

    def rows(first):
        """Pointers and strides of the projection, the geometry, the gate and the decays from this row on."""
        return (proj[first:].data_ptr(), proj.stride(0), g, gate[first:].data_ptr(), gate.stride(0),
                dec[first:].data_ptr() if dec is not None else None, dec.stride(0) if dec is not None else 0)
    if nd:
        check(lib().tsb_delta_step(*rows(0), w.conv.data_ptr(), w.a_log.data_ptr(), w.dt_bias.data_ptr(),
                                   w.norm.data_ptr(), conv_state.data_ptr(), state.data_ptr(), batch.state_slots.data_ptr(),
                                   batch.positions.data_ptr(), y.data_ptr(), y.stride(0), geo.out_cols, nd, geo.taps,
                                   float(w.eps), dt, st), "tsb_delta_step")
    n = T - nd
    if n:
        H, dev = geo.heads, proj.device
        blocks = batch.blk_seq.shape[0]
        f32 = lambda *s: torch.empty(s, device=dev, dtype=torch.float32)   # noqa: E731
        kq = f32(n, H, 3, geo.dim_pad) if geo.channels else f32(n, geo.kv_heads, 2, geo.dim_pad)
        g4 = f32(blocks, H, geo.dim_pad) if geo.channels else None
        v, coef, o = f32(n, H, geo.vdim_pad), f32(blocks, H, 36), f32(n, H, geo.vdim_pad)
        check(lib().tsb_delta_prefill(*rows(nd), w.conv.data_ptr(), w.a_log.data_ptr(), w.dt_bias.data_ptr(),
                                      w.norm.data_ptr(), conv_state.data_ptr(), state.data_ptr(), batch.cu.data_ptr(),
                                      batch.state_slots[nd:].data_ptr(), batch.pos0.data_ptr(), batch.blk_seq.data_ptr(),
                                      batch.blk0.data_ptr(), kq.data_ptr(), g4.data_ptr() if g4 is not None else None, v.data_ptr(),
                                      coef.data_ptr(), o.data_ptr(), y[nd:].data_ptr(), y.stride(0), geo.out_cols, n, blocks, batch.n_prompts,
                                      geo.taps, float(w.eps), dt, st), "tsb_delta_prefill")
        _native.add_launches(3 if geo.taps > 1 else 2)
    return y


def _gated_delta_torch(proj, gates, dec, geo, w, conv_state, state, batch, y):
    H, G, D, E, K = geo.heads, geo.kv_heads, geo.dim, geo.vdim, geo.taps
    y.zero_()
    for row0, n, slot, pos0 in batch.spans():
        if slot < 0:
            continue
        p = proj[row0:row0 + n].float()
        past = conv_state[slot].float() if pos0 > 0 else torch.zeros(K - 1, geo.conv_cols)
        x = torch.cat([past, p[:, :geo.conv_cols]], dim=0)
        c = torch.nn.functional.silu(sum(w.conv[j] * x[j:j + n] for j in range(K)))
        conv_state[slot] = x[n:].to(conv_state.dtype)
        q, k = (c[:, o:o + G * D].view(n, G, D) for o in (0, geo.off_k))
        q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
        k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        q, k = (t.repeat_interleave(H // G, dim=1) for t in (q, k))
        v = c[:, geo.off_v:geo.off_v + H * E].view(n, H, E)
        beta = torch.sigmoid(p[:, geo.off_b:geo.off_b + H])
        a = dec[row0:row0 + n, :H * D] if geo.channels else p[:, geo.off_a:geo.off_a + H]
        a = torch.nn.functional.softplus(a + w.dt_bias, threshold=1e9).view(n, H, -1)
        decay = torch.exp(-torch.exp(w.a_log)[:, None] * a)                       # [n, H, 1 or D]
        S = state[slot, :, :, :E].clone() if pos0 > 0 else torch.zeros(H, D, E)
        o = torch.empty(n, H, E)
        for t in range(n):
            S = S * decay[t, :, :, None]
            u = beta[t, :, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
            S = S + k[t, :, :, None] * u[:, None, :]
            o[t] = torch.einsum("hde,hd->he", S, q[t])
        state[slot, :, :, :E] = S
        gate = gates[row0:row0 + n, :H * E].float().view(n, H, E)
        gate = torch.sigmoid(gate) if geo.channels else torch.nn.functional.silu(gate)
        o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + w.eps) * w.norm * gate
        y[row0:row0 + n, :H * E] = o.reshape(n, H * E).to(y.dtype)
    return y
