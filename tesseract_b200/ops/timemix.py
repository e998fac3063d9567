"""Time mixing with a decay per channel over ragged batches (``csrc/time_mix.cu``). Per head a state S [dim, dim] with

    o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T;  w = exp(-exp(W2 tanh(d) + w0))

where r, k, v, a gate and d are projections of five different mixes of a token's input and the one before it (``token_shift``).
``time_mix`` takes the packed projection [r | k | v | gate | d] (decoded rows first, then portions of prompts), advances the slots
of a state pool and returns o / rms(o) * norm * silu(gate). CPU tensors run the torch restatement below.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr
from .gemm import input_columns, project

P, I, L, F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({
    "tsb_token_shift": [P, L, P, P, P, L, L, P, P, P, P, P, I, I, I, I, I, I, I, P],
    "tsb_tanh_rows": [P, L, P, I, I, I, P],
    "tsb_time_mix_step": [P, P, F, F, I, P],
    "tsb_time_mix_prefill": [P, P, I, F, F, I, P],
})
MAX_DIM = 256
CHUNK_DIM = 128          # widest heads of the tensor-core kernel
STREAMS = "rkvgw"
SPAN = 512               # tokens of a portion that one CTA walks where there are few portions


def spans_for(batch, ctas: int):
    """The batch's portions cut into spans, where whole portions would keep at most ``ctas`` CTAs, less than one per SM, busy; else
    None."""
    tiles = batch.tiles(SPAN)
    return tiles if ctas <= 148 and tiles.n > batch.n_prompts else None


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def _ptr(t):
    return t.data_ptr() if t is not None else None


@dataclass(frozen=True)
class TimeMixGeometry:
    """Sizes of one mixer and the layout of its packed projection row: r, k, v and the gate (heads of ``dp`` columns), then the
    ``rank`` inputs of the decay; every section starts where ``project_inputs`` wants an input to start."""
    heads: int
    dim: int
    rank: int

    def __post_init__(self):
        if min(self.heads, self.dim, self.rank) < 1:
            raise ValueError("time mix: positive sizes")
        if self.dp > MAX_DIM:
            raise ValueError(f"time mix: heads are at most {MAX_DIM} wide")

    @property
    def dp(self) -> int:
        return _up(self.dim, 16)

    @property
    def rp(self) -> int:
        return _up(self.rank, 16)

    @property
    def section(self) -> int:
        return input_columns(self.heads * self.dp)

    @property
    def starts(self) -> tuple:
        return tuple(i * self.section for i in range(5))

    @property
    def cols(self) -> int:
        return 4 * self.section + self.rp

    @property
    def out_cols(self) -> int:
        return self.heads * self.dp

    def ints(self, rows: int, n_seq: int, ld: int, ldo: int):
        v = (self.heads, self.dim, self.dp, self.rp, self.section, rows, n_seq, ld, ldo)
        return (ctypes.c_int * len(v))(*v)


@dataclass
class TimeMixWeights:
    """``w2`` [heads * dp, rp] in the model's type; fp32: ``w0`` and ``norm`` [heads * dp], ``u`` [heads * dp]."""
    w2: torch.Tensor
    w0: torch.Tensor
    u: torch.Tensor
    norm: torch.Tensor
    eps: float


def token_shift(h: torch.Tensor, mu: torch.Tensor, last: torch.Tensor, batch, keep: bool = False) -> torch.Tensor:
    """h [T, cols] (zero past the width) -> [n, T, cols]: h + (h' - h) mu[s] for every row s of ``mu`` [n, cols] (fp32), h' the row
    of the token before (zeros at position 0). ``last`` [slots, 1, cols] carries the last row of every sequence. ``keep``: h
    itself comes first."""
    T, C = h.shape
    n = mu.shape[0]
    xs = torch.empty((n + int(keep), T, C), device=h.device, dtype=h.dtype)
    if T == 0:
        return xs
    if h.is_cuda:
        nd = batch.n_decode
        check(lib().tsb_token_shift(h.data_ptr(), h.stride(0), mu.data_ptr(), last.data_ptr(), xs.data_ptr(), xs.stride(0), xs.stride(1),
                                    batch.positions.data_ptr(), batch.seq_of.data_ptr(), batch.state_slots.data_ptr(),
                                    batch.cu.data_ptr() if T > nd else None, batch.pos0.data_ptr() if T > nd else None, nd, T, C, n,
                                    int(keep), batch.n_prompts, dtype_code(h.dtype), stream_ptr(h.device)), "tsb_token_shift")
        if T > nd:
            _native.add_launches(1)
        return xs
    for row0, rows, slot, pos0 in batch.spans():
        x = h[row0:row0 + rows].float()
        first = last[slot].float() if pos0 > 0 and slot >= 0 else torch.zeros(1, C)
        before = torch.cat([first, x[:-1]])
        for s in range(n):
            xs[s + int(keep), row0:row0 + rows] = (x + (before - x) * mu[s]).to(h.dtype)
        if slot >= 0:
            last[slot] = h[row0 + rows - 1]
    if keep:
        xs[0] = h
    return xs


def time_mix(proj: torch.Tensor, geo: TimeMixGeometry, w: TimeMixWeights, state: torch.Tensor, batch, out_scale: float = 1.0,
             out: torch.Tensor | None = None) -> torch.Tensor:
    """proj [T, geo.cols] of a ragged batch -> [T, geo.out_cols] (``out`` may be columns of a wider matrix). ``state`` [slots,
    heads, dp, dp] (fp32, values x keys) is advanced in place; a sequence whose first row is at position 0 starts from zeros
    whatever its slot holds."""
    T = proj.shape[0]
    if out is None:
        out = torch.empty((T, geo.out_cols), device=proj.device, dtype=proj.dtype)
    if T == 0:
        return out
    if not proj.is_cuda:
        return _time_mix_torch(proj, geo, w, state, batch, out_scale, out)
    nd, dt, st = batch.n_decode, dtype_code(proj.dtype), stream_ptr(proj.device)
    if nd:
        ptrs = (ctypes.c_void_p * 9)(proj.data_ptr(), w.w2.data_ptr(), w.w0.data_ptr(), w.u.data_ptr(), w.norm.data_ptr(), state.data_ptr(),
                                     batch.state_slots.data_ptr(), batch.positions.data_ptr(), out.data_ptr())
        check(lib().tsb_time_mix_step(geo.ints(nd, nd, proj.stride(0), out.stride(0)), ptrs, float(w.eps), float(out_scale), dt, st),
              "tsb_time_mix_step")
    n = T - nd
    if n:
        pr = proj[nd:]
        low = torch.empty((n, geo.rp), device=proj.device, dtype=proj.dtype)
        check(lib().tsb_tanh_rows(pr[:, 4 * geo.section:].data_ptr(), pr.stride(0), low.data_ptr(), n, geo.rp, dt, st), "tsb_tanh_rows")
        dec = project(low, w.w2, out_dtype=torch.float32)
        chunked = proj.dtype == torch.bfloat16 and geo.dp <= CHUNK_DIM
        o = None if chunked else torch.empty((n, geo.heads, geo.dp), device=proj.device, dtype=torch.float32)
        spans = spans_for(batch, geo.heads * batch.n_prompts) if chunked else None
        carry = left = None
        if spans is not None:
            carry = torch.empty((spans.n, geo.heads, geo.dp, geo.dp), device=proj.device, dtype=torch.float32)
            left = torch.empty((spans.n, geo.heads, geo.dp), device=proj.device, dtype=torch.float32)
        ptrs = (ctypes.c_void_p * 15)(pr.data_ptr(), dec.data_ptr(), w.w0.data_ptr(), w.u.data_ptr(), w.norm.data_ptr(), state.data_ptr(),
                                      batch.state_slots[nd:].data_ptr(), batch.cu.data_ptr(), batch.pos0.data_ptr(), out[nd:].data_ptr(), _ptr(o),
                                      *((_ptr(spans.seq), _ptr(spans.first)) if spans is not None else (None, None)), _ptr(carry), _ptr(left))
        check(lib().tsb_time_mix_prefill(geo.ints(n, batch.n_prompts, proj.stride(0), out.stride(0)), ptrs,
                                         spans.n if spans is not None else 0, float(w.eps), float(out_scale), dt, st),
              "tsb_time_mix_prefill")
        _native.add_launches(2 if spans is not None else 0 if chunked else 1)
    return out


def _time_mix_torch(proj, geo, w, state, batch, out_scale, out):
    H, D, S0 = geo.heads, geo.dp, geo.section
    u = w.u.view(H, D)
    for row0, n, slot, pos0 in batch.spans():
        if slot < 0:
            continue
        p = proj[row0:row0 + n].float()
        r, k, v, g = (p[:, i * S0:i * S0 + H * D].view(n, H, D) for i in range(4))
        d = torch.tanh(p[:, 4 * S0:geo.cols]).to(proj.dtype).float() @ w.w2.float().t()
        decay = torch.exp(-torch.exp(d + w.w0)).view(n, H, D)
        S = state[slot].clone() if pos0 > 0 else torch.zeros(H, D, D)
        o = torch.empty(n, H, D)
        for t in range(n):
            kv = v[t][:, :, None] * k[t][:, None, :]
            o[t] = ((S + u[:, None, :] * kv) * r[t][:, None, :]).sum(-1)
            S = S * decay[t][:, None, :] + kv
        state[slot] = S
        o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / geo.dim + w.eps) * w.norm.view(H, D) * out_scale
        out[row0:row0 + n, :H * D] = (o * torch.nn.functional.silu(g)).reshape(n, H * D).to(out.dtype)
    return out
