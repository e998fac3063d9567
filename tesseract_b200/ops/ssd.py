"""State-space duality mixer over ragged batches (``csrc/ssd.cu``). Per head a state S [state, vdim] with a scalar decay per token:

    dt = softplus(dt + dt_bias);  S <- exp(-exp(A_log) dt) S + dt B x^T;  y = S^T C + D x

x, B and C come through one short causal convolution (with bias and SiLU) of a packed projection; heads share the B and C of their
group. y * silu(z) is normed in equal parts and scaled. ``ssd`` takes the projection of a ragged batch (decoded rows first, then
portions of prompts) and advances the slots of a state pool. CPU tensors run the torch restatement below.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr
from .timemix import spans_for

P, I, L, F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({
    "tsb_ssd_conv": [P, P, I, P],
    "tsb_ssd_step": [P, P, I, P],
    "tsb_ssd_prefill": [P, P, I, I, P],
    "tsb_part_norm": [P, L, P, L, P, I, I, I, I, I, F, F, I, P],
})
MAX_STATE = 256
MAX_TAPS = 8
CONV_TILE = 16          # tokens of a portion that a thread of the convolution walks


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class SSDGeometry:
    """Sizes of one mixer and the layout of its packed projection row [z | x | B | C | dt]: z and x in heads of ``vp`` columns, B
    and C in groups of ``np`` columns. A slot's convolution state holds the last taps - 1 rows of x, B and C."""
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_parts: int

    def __post_init__(self):
        if min(self.heads, self.vdim, self.state, self.groups, self.taps, self.norm_parts) < 1 or self.heads % self.groups:
            raise ValueError("ssd: positive sizes, and heads a multiple of groups")
        if (self.heads * self.vdim) % self.norm_parts:
            raise ValueError("ssd: the norm's parts are equal")
        if self.np > MAX_STATE or self.taps > MAX_TAPS:
            raise ValueError(f"ssd: states of at most {MAX_STATE} rows and at most {MAX_TAPS} convolution taps")

    @property
    def vp(self) -> int:
        return _up(self.vdim, 8)

    @property
    def np(self) -> int:
        return _up(self.state, 16)

    @property
    def off_x(self) -> int:
        return self.heads * self.vp

    @property
    def off_b(self) -> int:
        return 2 * self.off_x

    @property
    def off_c(self) -> int:
        return self.off_b + self.groups * self.np

    @property
    def off_dt(self) -> int:
        return self.off_c + self.groups * self.np

    @property
    def conv_cols(self) -> int:
        return self.off_dt - self.off_x

    @property
    def cols(self) -> int:
        return self.off_dt + _up(self.heads, 8)

    @property
    def out_cols(self) -> int:
        return _up(self.heads * self.vp, 16)

    def ints(self, rows: int, n_decode: int, n_seq: int, blocks: int, ld: int, ldo: int):
        v = (self.heads, self.vdim, self.vp, self.state, self.np, self.groups, self.taps, rows, n_decode, n_seq, blocks, ld, ldo)
        return (ctypes.c_int * len(v))(*v)


@dataclass
class SSDWeights:
    """fp32 parameters besides the projections: convolution [taps, conv_cols] and its bias, a_log, dt_bias, d [heads], norm
    [heads * vp]."""
    conv: torch.Tensor
    conv_b: torch.Tensor
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    d: torch.Tensor
    norm: torch.Tensor
    eps: float


def part_norm_(t: torch.Tensor, z, weight: torch.Tensor, heads: int, vdim: int, vp: int, parts: int, eps: float, scale: float) -> torch.Tensor:
    """In place on t [T, >= heads * vp], heads of ``vdim`` columns stored ``vp`` apart: t * silu(z) (z laid out like t, or None), then
    each of ``parts`` equal runs of the logical columns over its root mean square, times weight [heads * vp] and ``scale``."""
    T = t.shape[0]
    if T == 0:
        return t
    if t.is_cuda:
        check(lib().tsb_part_norm(t.data_ptr(), t.stride(0), z.data_ptr() if z is not None else None,
                                  z.stride(0) if z is not None else 0, weight.data_ptr(), T, heads, vdim, vp, parts, float(eps), float(scale),
                                  dtype_code(t.dtype), stream_ptr(t.device)), "tsb_part_norm")
        return t
    x = t[:, :heads * vp].float().clone()
    if z is not None:
        x *= torch.nn.functional.silu(z[:, :heads * vp].float())
    x = x.view(T, heads, vp)
    flat = x[:, :, :vdim].reshape(T, parts, -1)
    flat = (flat / torch.sqrt((flat * flat).mean(-1, keepdim=True) + eps)).view(T, heads, vdim) * scale
    x[:, :, :vdim] = flat * weight.view(heads, vp)[:, :vdim]
    t[:, :heads * vp] = x.reshape(T, -1).to(t.dtype)
    return t


def ssd(proj: torch.Tensor, geo: SSDGeometry, w: SSDWeights, conv_state: torch.Tensor, state: torch.Tensor, batch,
        out_scale: float = 1.0, out: torch.Tensor | None = None) -> torch.Tensor:
    """proj [T, geo.cols] of a ragged batch -> [T, geo.out_cols] (``out`` may be columns of a wider matrix). ``conv_state`` [slots,
    taps - 1, conv_cols] (projection dtype) and ``state`` [slots, heads, vp, np] (fp32, values x state) are advanced in place; a
    sequence whose first row is at position 0 starts from zeros whatever its slot holds."""
    T, H = proj.shape[0], geo.heads
    if out is None:
        out = torch.empty((T, geo.out_cols), device=proj.device, dtype=proj.dtype)
    if T == 0:
        return out
    if geo.out_cols > H * geo.vp:
        out[:, H * geo.vp:geo.out_cols] = 0
    if not proj.is_cuda:
        _ssd_torch(proj, geo, w, conv_state, state, batch, out)
    else:
        nd, dt, st = batch.n_decode, dtype_code(proj.dtype), stream_ptr(proj.device)
        n = T - nd
        xbc = torch.empty((T, geo.conv_cols), device=proj.device, dtype=proj.dtype)
        gates = torch.empty((T, H, 2), device=proj.device, dtype=torch.float32)       # dt, log2 of the decay
        tiles = batch.tiles(CONV_TILE) if n else None
        ints = geo.ints(T, nd, batch.n_prompts, tiles.n if n else 0, proj.stride(0), out.stride(0))
        some = lambda name: getattr(batch, name).data_ptr() if n else None   # noqa: E731
        ptrs = (ctypes.c_void_p * 14)(proj.data_ptr(), w.conv.data_ptr(), w.conv_b.data_ptr(), w.a_log.data_ptr(), w.dt_bias.data_ptr(),
                                      conv_state.data_ptr(), xbc.data_ptr(), gates.data_ptr(), batch.state_slots.data_ptr(),
                                      batch.positions.data_ptr(), some("cu"), some("pos0"), tiles.seq.data_ptr() if n else None,
                                      tiles.first.data_ptr() if n else None)
        check(lib().tsb_ssd_conv(ints, ptrs, dt, st), "tsb_ssd_conv")
        if nd:
            ptrs = (ctypes.c_void_p * 8)(proj.data_ptr(), xbc.data_ptr(), gates.data_ptr(), w.d.data_ptr(), state.data_ptr(),
                                         batch.state_slots.data_ptr(), batch.positions.data_ptr(), out.data_ptr())
            check(lib().tsb_ssd_step(ints, ptrs, dt, st), "tsb_ssd_step")
        if n:
            spans = spans_for(batch, H * batch.n_prompts * ((geo.vp + 63) // 64)) if proj.dtype == torch.bfloat16 else None
            extra = (None,) * 4
            if spans is not None:
                carry = torch.empty((spans.n, H, geo.vp, geo.np), device=proj.device, dtype=torch.float32)
                left = torch.empty((spans.n, H), device=proj.device, dtype=torch.float32)
                extra = tuple(t.data_ptr() for t in (spans.seq, spans.first, carry, left))
            ptrs = (ctypes.c_void_p * 13)(proj[nd:].data_ptr(), xbc[nd:].data_ptr(), gates[nd:].data_ptr(), w.d.data_ptr(), state.data_ptr(),
                                         batch.state_slots[nd:].data_ptr(), batch.cu.data_ptr(), batch.pos0.data_ptr(),
                                          out[nd:].data_ptr(), *extra)
            check(lib().tsb_ssd_prefill(ints, ptrs, spans.n if spans is not None else 0, dt, st), "tsb_ssd_prefill")
            _native.add_launches(2 if spans is not None else 0)
            _native.add_launches(2 if nd and geo.taps > 1 else 1 if nd or geo.taps > 1 else 0)
    return part_norm_(out, proj, w.norm, H, geo.vdim, geo.vp, geo.norm_parts, w.eps, out_scale)


def _ssd_torch(proj, geo, w, conv_state, state, batch, out):
    H, E, N, G, K = geo.heads, geo.vp, geo.np, geo.groups, geo.taps
    X = H * E
    for row0, n, slot, pos0 in batch.spans():
        if slot < 0:
            out[row0:row0 + n, :X] = 0
            continue
        p = proj[row0:row0 + n].float()
        past = conv_state[slot].float() if pos0 > 0 else torch.zeros(K - 1, geo.conv_cols)
        x = torch.cat([past, p[:, geo.off_x:geo.off_dt]], dim=0)
        c = torch.nn.functional.silu(sum(w.conv[j] * x[j:j + n] for j in range(K)) + w.conv_b)
        conv_state[slot] = x[n:].to(conv_state.dtype)
        c = c.to(proj.dtype).float()
        xv = c[:, :X].view(n, H, E)
        B, C = (c[:, X + s * G * N:X + (s + 1) * G * N].view(n, G, N).repeat_interleave(H // G, dim=1) for s in (0, 1))
        dt = torch.nn.functional.softplus(p[:, geo.off_dt:geo.off_dt + H] + w.dt_bias, threshold=1e9)
        decay = torch.exp(-torch.exp(w.a_log) * dt)
        S = state[slot].clone() if pos0 > 0 else torch.zeros(H, E, N)
        y = torch.empty(n, H, E)
        for t in range(n):
            S = decay[t][:, None, None] * S + (dt[t][:, None] * xv[t])[:, :, None] * B[t][:, None, :]
            y[t] = (S * C[t][:, None, :]).sum(-1) + w.d[:, None] * xv[t]
        state[slot] = S
        out[row0:row0 + n, :X] = y.reshape(n, X).to(out.dtype)
