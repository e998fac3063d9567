"""Retention over ragged batches (``csrc/retention.cu``): linear attention with one fixed decay per head,

    S <- decay S + k v^T;  o = S^T q;  out = o / rms(o) * silu(gate)

with rotary positions on q and k and dim^-1/2 on k. ``retention`` takes a packed projection [q | k | v | gate] (decoded rows
first, then portions of prompts), advances the slots of a state pool and returns the gated read-outs. CPU tensors run the
torch restatement below.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr
from .rotary import Rotary, rotate_stored

P, I, L, F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({
    "tsb_retention_prefill": [P, P, L, F, F] + [P] * 11 + [L, F, I, I, P],
    "tsb_retention_step": [P, P, L, F, F] + [P] * 6 + [L, F, I, P],
})

MAX_DIM = 256
SPAN = 256          # tokens of a portion that one CTA walks


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class RetentionGeometry:
    """Sizes of one mixer and the layout of its packed projection row [q | k | v | gate]: query and key heads in the stored
    rotary layout, value heads padded to a multiple of 8 columns."""
    heads: int
    dim: int
    vdim: int
    rotary: Rotary

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim) < 1 or self.rotary.dims > self.dim:
            raise ValueError("retention: positive sizes, and at most dim rotated dims")
        if self.dp > MAX_DIM:
            raise ValueError(f"retention: query and key heads take at most {MAX_DIM} columns")

    @property
    def dp(self) -> int:
        return self.rotary.stored(self.dim, 16)

    @property
    def vp(self) -> int:
        return _up(self.vdim, 8)

    @property
    def off_k(self) -> int:
        return self.heads * self.dp

    @property
    def off_v(self) -> int:
        return 2 * self.heads * self.dp

    @property
    def off_gate(self) -> int:
        return self.off_v + self.heads * self.vp

    @property
    def cols(self) -> int:
        return self.off_gate + self.heads * self.vp

    @property
    def out_cols(self) -> int:
        return _up(self.heads * self.vp, 16)

    def ints(self, rows: int, n_seq: int, spans: int):
        v = (self.heads, self.dp, self.rotary.hp, self.vp, self.vdim, self.off_k, self.off_v, self.off_gate, rows, n_seq, spans)
        return (ctypes.c_int * len(v))(*v)


def log2_decays(decay) -> torch.Tensor:
    """fp32 logarithms of the decays; a decay of 0 becomes a number whose every multiple underflows to 0."""
    for d in decay:
        if not 0.0 <= d <= 1.0:
            raise ValueError("retention: decays lie between 0 and 1")
    return torch.tensor([math.log2(d) if d > 0 else -1e30 for d in decay], dtype=torch.float64).float()


def retention(proj: torch.Tensor, geo: RetentionGeometry, log2_decay: torch.Tensor, eps: float, state: torch.Tensor, table: torch.Tensor,
              batch, in_scale: float = 1.0, out: torch.Tensor | None = None) -> torch.Tensor:
    """proj [T, geo.cols] of a ragged batch -> [T, geo.out_cols] (``out`` may be columns of a wider matrix). ``state`` [slots,
    heads, dp, vp] (fp32) is advanced in place; a sequence whose first row is at position 0 starts from zeros whatever its
    slot holds. ``in_scale`` multiplies the projection."""
    T = proj.shape[0]
    if out is None:
        out = torch.empty((T, geo.out_cols), device=proj.device, dtype=proj.dtype)
    if T == 0:
        return out
    if geo.out_cols > geo.heads * geo.vp:
        out[:, geo.heads * geo.vp:] = 0
    k_scale = geo.dim ** -0.5 * in_scale * in_scale        # (the values' factor rides on the keys)
    if not proj.is_cuda:
        return _retention_torch(proj, geo, log2_decay, eps, state, table, batch, in_scale, k_scale, out)
    nd, dt, st = batch.n_decode, dtype_code(proj.dtype), stream_ptr(proj.device)
    if nd:
        check(lib().tsb_retention_step(geo.ints(nd, nd, 0), proj.data_ptr(), proj.stride(0), float(in_scale), float(k_scale),
                                       log2_decay.data_ptr(), table.data_ptr(), state.data_ptr(), batch.state_slots.data_ptr(),
                                       batch.positions.data_ptr(), out.data_ptr(), out.stride(0), float(eps), dt, st),
              "tsb_retention_step")
    n = T - nd
    if n:
        f32 = dict(device=proj.device, dtype=torch.float32)
        chunked = proj.dtype == torch.bfloat16
        tiles = batch.tiles(SPAN) if chunked else None
        spans = tiles.n if chunked else 0
        cols = 128 if geo.dp <= 128 and geo.vp > 64 else 64
        carry = torch.empty((spans, geo.heads, geo.dp, geo.vp), **f32) if spans > batch.n_prompts else None
        o = torch.empty((n, geo.heads, geo.vp), **f32) if not chunked or geo.vp > cols else None
        ptr = lambda t: t.data_ptr() if t is not None else None   # noqa: E731
        pr, res = proj[nd:], out[nd:]
        check(lib().tsb_retention_prefill(geo.ints(n, batch.n_prompts, spans), pr.data_ptr(), pr.stride(0), float(in_scale),
                                          float(k_scale), log2_decay.data_ptr(), table.data_ptr(), state.data_ptr(),
                                          batch.state_slots[nd:].data_ptr(), batch.cu.data_ptr(), batch.pos0.data_ptr(),
                                          tiles.seq.data_ptr() if chunked else None, tiles.first.data_ptr() if chunked else None,
                                          ptr(carry), ptr(o), res.data_ptr(), res.stride(0), float(eps), int(chunked), dt, st),
              "tsb_retention_prefill")
        _native.add_launches((2 if carry is not None else 0) + (1 if o is not None else 0))
    return out


def _retention_torch(proj, geo, log2_decay, eps, state, table, batch, in_scale, k_scale, out):
    H, D, E = geo.heads, geo.dp, geo.vp
    decay = torch.exp2(log2_decay)[:, None, None]
    for row0, n, slot, pos0 in batch.spans():
        if slot < 0:
            continue
        p = proj[row0:row0 + n].float()
        pos = torch.arange(pos0, pos0 + n)
        q = rotate_stored(p[:, :geo.off_k].view(n, H, D), table, pos) * in_scale
        k = rotate_stored(p[:, geo.off_k:geo.off_v].view(n, H, D), table, pos) * k_scale
        v = p[:, geo.off_v:geo.off_gate].view(n, H, E)
        gate = p[:, geo.off_gate:geo.cols].view(n, H, E) * in_scale
        S = state[slot].clone() if pos0 > 0 else torch.zeros(H, D, E)
        o = torch.empty(n, H, E)
        for t in range(n):
            S = decay * S + k[t, :, :, None] * v[t, :, None, :]
            o[t] = torch.einsum("hde,hd->he", S, q[t])
        state[slot] = S
        o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / geo.vdim + eps) * torch.nn.functional.silu(gate)
        out[row0:row0 + n, :H * E] = o.reshape(n, H * E).to(out.dtype)
    return out
