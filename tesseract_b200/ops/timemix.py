"""Linear attention with a decay per key channel and token over ragged batches (``csrc/time_mix.cu``).

``time_mix``: per head a state S [dim, dim] with

    o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T;  w = exp(-exp(W2 tanh(d) + w0))

where r, k, v, a gate and d are projections of five different mixes of a token's input and the one before it (``token_shift``).
``time_mix`` takes the packed projection [r | k | v | gate | d] (decoded rows first, then portions of prompts), advances the slots
of a state pool and returns o / rms(o) * norm * silu(gate).

``gated_linear``: per head a state S [dim, vdim] with

    S <- diag(w) S + k v^T;  o = S^T q dim^-1/2;  w = sigmoid(W2 d + w0)^(1 / tau)

from the packed projection [q | k | v | gate | d] of one input, and out as above. CPU tensors run the torch restatements below.
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
    "tsb_time_mix_step": [P, P, P, I, P],
    "tsb_time_mix_prefill": [P, P, P, I, I, P],
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

    def ints(self, rows: int, n_seq: int, ld: int, ldo: int, ld_dec: int):
        S = self.section
        v = (self.heads, self.dim, self.dp, self.dp, self.rp, S, 2 * S, 3 * S, 4 * S, rows, n_seq, ld, ldo, ld_dec, 0)
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
    floats = _floats(w.eps, out_scale)
    if nd:
        ptrs = (ctypes.c_void_p * 10)(proj.data_ptr(), w.w2.data_ptr(), w.w0.data_ptr(), w.u.data_ptr(), w.norm.data_ptr(), state.data_ptr(),
                                      batch.state_slots.data_ptr(), batch.positions.data_ptr(), out.data_ptr(), None)
        check(lib().tsb_time_mix_step(geo.ints(nd, nd, proj.stride(0), out.stride(0), 0), floats, ptrs, dt, st), "tsb_time_mix_step")
    n = T - nd
    if n:
        pr = proj[nd:]
        low = torch.empty((n, geo.rp), device=proj.device, dtype=proj.dtype)
        check(lib().tsb_tanh_rows(pr[:, 4 * geo.section:].data_ptr(), pr.stride(0), low.data_ptr(), n, geo.rp, dt, st), "tsb_tanh_rows")
        dec = project(low, w.w2, out_dtype=torch.float32)
        _prompts(pr, dec, geo, geo.dp, geo.dp, w.w0, w.u, w.norm, state, batch, out[nd:], floats)
    return out


def _floats(eps, out_scale, r_scale=1.0, tau=1.0):
    return (ctypes.c_float * 4)(eps, out_scale, r_scale, 1.0 / tau)


def _prompts(pr, dec, geo, dp, ep, w0, u, norm, state, batch, out, floats):
    """The prompt rows of either form: pr [n, geo.cols], dec [n, heads * dp] (fp32)."""
    nd, n, dev, H = batch.n_decode, pr.shape[0], pr.device, geo.heads
    chunked = pr.dtype == torch.bfloat16 and max(dp, ep) <= CHUNK_DIM
    f32 = lambda *s: torch.empty(s, device=dev, dtype=torch.float32)   # noqa: E731
    o = None if chunked else f32(n, H, ep)
    spans = spans_for(batch, H * batch.n_prompts) if chunked else None
    carry, left = (f32(spans.n, H, ep, dp), f32(spans.n, H, dp)) if spans is not None else (None, None)
    ptrs = (ctypes.c_void_p * 15)(pr.data_ptr(), dec.data_ptr(), w0.data_ptr(), _ptr(u), norm.data_ptr(), state.data_ptr(),
                                  batch.state_slots[nd:].data_ptr(), batch.cu.data_ptr(), batch.pos0.data_ptr(), out.data_ptr(), _ptr(o),
                                  *((_ptr(spans.seq), _ptr(spans.first)) if spans is not None else (None, None)), _ptr(carry), _ptr(left))
    check(lib().tsb_time_mix_prefill(geo.ints(n, batch.n_prompts, pr.stride(0), out.stride(0), dec.stride(0)), floats, ptrs,
                                     spans.n if spans is not None else 0, dtype_code(pr.dtype), stream_ptr(dev)), "tsb_time_mix_prefill")
    _native.add_launches(2 if spans is not None else 0 if chunked else 1)


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


# ------------------------------------------------------------------------------ gated linear attention
@dataclass(frozen=True)
class GatedLinearGeometry:
    """Sizes of one mixer and the layout of its packed projection row: q, k (heads of ``dp`` columns), v and the gate (of ``ep``), then
    the ``rank`` inputs of the decay."""
    heads: int
    dim: int
    vdim: int
    rank: int

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim, self.rank) < 1:
            raise ValueError("gated linear attention: positive sizes")
        if self.dp > MAX_DIM:
            raise ValueError(f"gated linear attention: query and key heads are at most {MAX_DIM} wide")

    @property
    def dp(self) -> int:
        return _up(self.dim, 16)

    @property
    def ep(self) -> int:
        return _up(self.vdim, 16)

    @property
    def rp(self) -> int:
        return _up(self.rank, 16)

    @property
    def off_k(self) -> int:
        return self.heads * self.dp

    @property
    def off_v(self) -> int:
        return 2 * self.off_k

    @property
    def off_gate(self) -> int:
        return self.off_v + self.heads * self.ep

    @property
    def off_low(self) -> int:
        return self.off_gate + self.heads * self.ep

    @property
    def cols(self) -> int:
        return self.off_low + self.rp

    @property
    def out_cols(self) -> int:
        return self.heads * self.ep

    def ints(self, rows: int, n_seq: int, ld: int, ldo: int, ld_dec: int):
        v = (self.heads, self.vdim, self.dp, self.ep, self.rp, self.off_k, self.off_v, self.off_gate, self.off_low, rows, n_seq, ld, ldo,
             ld_dec, 1)
        return (ctypes.c_int * len(v))(*v)


@dataclass
class GatedLinearWeights:
    """``w2`` [heads * dp, rp] in the model's type; fp32: ``w0`` [heads * dp], ``norm`` [heads * ep]."""
    w2: torch.Tensor
    w0: torch.Tensor
    norm: torch.Tensor
    tau: float
    eps: float


def gated_linear(proj: torch.Tensor, geo: GatedLinearGeometry, w: GatedLinearWeights, state: torch.Tensor, batch, out_scale: float = 1.0,
                 out: torch.Tensor | None = None) -> torch.Tensor:
    """proj [T, geo.cols] of a ragged batch -> [T, geo.out_cols] (``out`` may be columns of a wider matrix). ``state`` [slots,
    heads, ep, dp] (fp32, values x keys) is advanced in place; a sequence whose first row is at position 0 starts from zeros
    whatever its slot holds."""
    T = proj.shape[0]
    if out is None:
        out = torch.empty((T, geo.out_cols), device=proj.device, dtype=proj.dtype)
    if T == 0:
        return out
    dec = project(proj[:, geo.off_low:geo.cols], w.w2, out_dtype=torch.float32)
    if not proj.is_cuda:
        return _gated_linear_torch(proj, dec, geo, w, state, batch, out_scale, out)
    nd = batch.n_decode
    floats = _floats(w.eps, out_scale, geo.dim ** -0.5, w.tau)
    if nd:
        ptrs = (ctypes.c_void_p * 10)(proj.data_ptr(), None, w.w0.data_ptr(), None, w.norm.data_ptr(), state.data_ptr(),
                                      batch.state_slots.data_ptr(), batch.positions.data_ptr(), out.data_ptr(), dec.data_ptr())
        check(lib().tsb_time_mix_step(geo.ints(nd, nd, proj.stride(0), out.stride(0), dec.stride(0)), floats, ptrs, dtype_code(proj.dtype),
                                      stream_ptr(proj.device)), "tsb_time_mix_step")
    if T > nd:
        _prompts(proj[nd:], dec[nd:], geo, geo.dp, geo.ep, w.w0, None, w.norm, state, batch, out[nd:], floats)
    return out


def _gated_linear_torch(proj, dec, geo, w, state, batch, out_scale, out):
    H, D, E = geo.heads, geo.dp, geo.ep
    for row0, n, slot, pos0 in batch.spans():
        if slot < 0:
            continue
        p = proj[row0:row0 + n].float()
        q, k = (p[:, o:o + H * D].view(n, H, D) for o in (0, geo.off_k))
        v, g = (p[:, o:o + H * E].view(n, H, E) for o in (geo.off_v, geo.off_gate))
        decay = torch.exp(torch.nn.functional.logsigmoid(dec[row0:row0 + n] + w.w0) / w.tau).view(n, H, D)
        S = state[slot].clone() if pos0 > 0 else torch.zeros(H, E, D)
        o = torch.empty(n, H, E)
        for t in range(n):
            S = S * decay[t][:, None, :] + v[t][:, :, None] * k[t][:, None, :]
            o[t] = (S * (q[t] * geo.dim ** -0.5)[:, None, :]).sum(-1)
        state[slot] = S
        o = o / torch.sqrt((o * o).sum(-1, keepdim=True) / geo.vdim + w.eps) * w.norm.view(H, E) * out_scale
        out[row0:row0 + n, :H * E] = (o * torch.nn.functional.silu(g)).reshape(n, H * E).to(out.dtype)
    return out
