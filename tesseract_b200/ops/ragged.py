"""Attention over paged pools for ragged batches: decoded rows (one token per sequence) first, then portions of prompts.

``ragged_attention`` takes a packed [q | k | v] projection, adds its biases and appends keys and values to the pool;
``shaped_attention`` takes [q | k | v | gate], and on the way norms and rotates q and k, mixes values and gates the result.
Both attend under a mask (chunks: token i sees the tokens j <= i of its own run of positions; a window: the last tokens):

* decoded rows: the split-K paged kernel (``csrc/decode_attn_mma.cu``), which starts at the first key of the chunk or window;
* prompt rows: the tcgen05 kernel (``csrc/flash_attn_fwd.cu``) with every chunk of a portion as a sequence of its own; the
  keys that a portion needs from earlier ones are copied from the pool in front of its own;
* fp32 models and head sizes other than 64 / 128: one warp per (row, head) over the pool (``csrc/ragged_attn.cu``).

Query, key and value heads share one padded size ``D`` (zero columns change no score and no result).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr
from .masks import Mask, Window
from .paged import _decode_scratch, _gather_request, _scratch_floats
from .rotary import Rotary, rotate_stored

P, I, L, F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({
    "tsb_ragged_append": [P, L, P, P, P, P, P, P, P, I, I, I, I, I, I, I, P],
    "tsb_stage_gather": [P, P, P, P, P, I, I, I, I, P],
    "tsb_ragged_attn": [P, L, P, P, P, I, P, P, P, I, I, I, I, I, I, P, P, P, I, P],
    "tsb_paged_decode_shaped": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, P, P, P, I, P],
    "tsb_flash_fwd_shaped": [P, P, P, P, P, P, I, I, I, I, I, I, I, P, P, P, F, P],
    "tsb_attn_prepare": [P, P, P, I, P],
    "tsb_flash_fwd_varlen_keys": [P, P, P, P, P, P, I, I, I, I, I, I, I, L, L, L, L, L, L, L, L, F, P],
})
MAX_HEAD = 256


def padded_head_dim(dim: int, vdim: int, dtype: torch.dtype) -> int:
    """Common head size of the pools: 64 or 128 where the tensor-core kernels serve it, else a multiple of 32."""
    d = max(dim, vdim)
    if d > MAX_HEAD:
        raise ValueError(f"attention heads are at most {MAX_HEAD} wide")
    if dtype == torch.bfloat16 and d <= 128:
        return 64 if d <= 64 else 128
    return (d + 31) // 32 * 32


def tensor_core_heads(D: int, dtype: torch.dtype) -> bool:
    return dtype == torch.bfloat16 and D in (64, 128)


@dataclass
class ScoreForm:
    """What becomes of the products q . k before and in the softmax: s = scale (q . k); s = softcap tanh(s / softcap) where a
    softcap is given; s -= slopes[h] (i - j) (``slopes`` fp32 [heads]); exp(sink[h]) joins the denominator (``sink`` fp32
    [heads]). ``product_bound``: no |q . k| is larger (0: not known)."""
    scale: float
    mask: Mask = 0
    softcap: float = 0.0
    slopes: Optional[torch.Tensor] = None
    sink: Optional[torch.Tensor] = None
    product_bound: float = 0.0

    @property
    def bound(self) -> float:
        """No |score| is larger before distances are taken off (0: not known)."""
        known = [b for b in (self.softcap, self.product_bound * abs(self.scale)) if b > 0.0]
        return min(known) * 1.001 if known else 0.0      # (products of rounded vectors may end slightly above)


@dataclass
class OutputGate:
    """The result times ``scale``, and times sigmoid(gate): ``gate`` [T, heads] or, element by element, [T, heads * D]."""
    gate: Optional[torch.Tensor] = None
    per_element: bool = False
    scale: float = 1.0


_PLAIN_GATE = OutputGate()


def _ptr(t):
    return t.data_ptr() if t is not None else None


def _attention_args(form: ScoreForm, gate: OutputGate, ldo: int):
    """(ints, floats, pointers) of ``csrc/attn_form.cuh``."""
    window = form.mask.size if isinstance(form.mask, Window) else 0
    chunk = 0 if window else form.mask
    kind = 0 if gate.gate is None else 2 if gate.per_element else 1
    ints = (ctypes.c_longlong * 5)(chunk, window, kind, gate.gate.stride(0) if kind else 0, ldo)
    floats = (ctypes.c_float * 3)(form.scale, form.softcap, gate.scale)
    ptrs = (ctypes.c_void_p * 3)(_ptr(form.slopes), _ptr(form.sink), _ptr(gate.gate))
    return ints, floats, ptrs


def _attend(q, stage, k_pool, v_pool, batch, form: ScoreForm, gate: OutputGate, out):
    """q [T, H, D]; stage: the key axis [keys, 2 G, D] of the prompt rows with this step's own keys in place (None where the
    tensor-core kernels do not serve). ``out`` [T, >= H * D]."""
    T, H, D = q.shape
    nb, G, bs, _ = k_pool.shape
    st, dt, nd = stream_ptr(q.device), dtype_code(q.dtype), batch.n_decode
    n, tables, ldo = T - nd, batch.tables, out.stride(0)
    if not (tensor_core_heads(D, q.dtype) and bs % 8 == 0):
        check(lib().tsb_ragged_attn(q.data_ptr(), H * D, k_pool.data_ptr(), v_pool.data_ptr(), tables.data_ptr(), tables.stride(0),
                                    batch.seq_of.data_ptr(), batch.positions.data_ptr(), out.data_ptr(), T, H, G, D, bs, nb,
                                    *_attention_args(form, gate, ldo), dt, st), "tsb_ragged_attn")
        return
    if nd:
        # planned for the longest sequence the tables can hold, so that a captured launch serves every later step
        longest = batch.max_len
        reach = form.mask.size if isinstance(form.mask, Window) else form.mask
        scratch = _decode_scratch(q.device, _scratch_floats(nd, H, G, D, min(longest, reach) if reach else longest, False))
        check(lib().tsb_paged_decode_shaped(q.data_ptr(), k_pool.data_ptr(), v_pool.data_ptr(), tables.data_ptr(), batch.lens.data_ptr(),
                                            out.data_ptr(), scratch.data_ptr(), nd, H, G, D, bs, nb, tables.stride(0), longest,
                                            *_attention_args(form, gate, ldo), dt, st), "tsb_paged_decode_shaped")
    if n:
        seg = batch.segments(form.mask)
        if seg.n_gather:
            check(lib().tsb_stage_gather(k_pool.data_ptr(), v_pool.data_ptr(), stage.data_ptr(), seg.gather_dst.data_ptr(),
                                         seg.gather_src.data_ptr(), seg.n_gather, G, D, bs, st), "tsb_stage_gather")
        later = OutputGate(gate.gate[nd:] if gate.gate is not None else None, gate.per_element, gate.scale)
        check(lib().tsb_flash_fwd_shaped(q[nd:].data_ptr(), stage.data_ptr(), stage[:, G:].data_ptr(), out[nd:].data_ptr(), seg.cu_q.data_ptr(),
                                         seg.cu_k.data_ptr(), seg.n, seg.max_q, n, seg.keys, H, G, D, *_attention_args(form, later, ldo),
                                         float(form.bound), st), "tsb_flash_fwd_shaped")


def ragged_attention(qkv: torch.Tensor, bias, k_pool: torch.Tensor, v_pool: torch.Tensor, batch, heads: int, kv_heads: int,
                     scale: float, chunk: int = 0) -> torch.Tensor:
    """qkv [T, (heads + 2 kv_heads) D] -> [T, heads * D]; pools [blocks, kv_heads, block, D]."""
    T, H, G, D = qkv.shape[0], heads, kv_heads, k_pool.shape[3]
    bs = k_pool.shape[2]
    if T == 0:
        return qkv.new_empty((0, H * D))
    form = ScoreForm(scale, chunk)
    if not qkv.is_cuda:
        z = (qkv.float() + bias if bias is not None else qkv.float()).to(qkv.dtype).view(T, H + 2 * G, D)
        out = torch.zeros(T, H * D, dtype=qkv.dtype)
        return _attend_torch(z[:, :H], z[:, H:H + G], z[:, H + G:], k_pool, v_pool, batch, form, _PLAIN_GATE, out)
    st, dt = stream_ptr(qkv.device), dtype_code(qkv.dtype)
    nd, n = batch.n_decode, T - batch.n_decode
    q = torch.empty((T, H, D), device=qkv.device, dtype=qkv.dtype)
    seg = batch.segments(chunk) if n and tensor_core_heads(D, qkv.dtype) and bs % 8 == 0 else None
    stage = torch.empty((seg.keys, 2 * G, D), device=qkv.device, dtype=qkv.dtype) if seg is not None else None
    check(lib().tsb_ragged_append(qkv.data_ptr(), qkv.stride(0), _ptr(bias), batch.slots.data_ptr(), q.data_ptr(), k_pool.data_ptr(),
                                  v_pool.data_ptr(), _ptr(stage), _ptr(seg.stage_rows) if seg is not None else None, nd, T, H, G, D,
                                  bs, dt, st), "tsb_ragged_append")
    out = torch.empty((T, H * D), device=qkv.device, dtype=qkv.dtype)
    _attend(q, stage, k_pool, v_pool, batch, form, _PLAIN_GATE, out)
    return out


# ------------------------------------------------------------------------------ with norms, rotation, values of other layers, gates
@dataclass(frozen=True)
class AttentionGeometry:
    """Sizes of one mixer and the layout of its packed projection row [q | k | v | gate], every head D columns wide, query and key
    heads in the stored rotary layout. With ``keys_as_values`` there is no v section. ``gate``: "" (none), "head" or "element"."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    dtype: torch.dtype
    rotary: Optional[Rotary] = None
    keys_as_values: bool = False
    gate: str = ""

    def __post_init__(self):
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads:
            raise ValueError("attention: positive sizes, and heads a multiple of kv_heads")
        if self.keys_as_values and (self.vdim != self.dim or self.rotary is not None):
            raise ValueError("attention: values that are the keys have their size, and the keys are not rotated")
        if self.gate not in ("", "head", "element"):
            raise ValueError(f"attention: unknown gate {self.gate!r}")
        self.D                               # (checks the size)

    @property
    def hp(self) -> int:
        return self.rotary.hp if self.rotary is not None else 0

    def columns(self) -> torch.Tensor:
        """Column of each coordinate of a query or key head."""
        return self.rotary.columns(self.dim) if self.rotary is not None else torch.arange(self.dim)

    @property
    def D(self) -> int:
        stored = self.rotary.stored(self.dim) if self.rotary is not None else self.dim
        return padded_head_dim(stored, self.vdim, self.dtype)

    @property
    def off_k(self) -> int:
        return self.heads * self.D

    @property
    def off_v(self) -> int:
        return self.off_k if self.keys_as_values else self.off_k + self.kv_heads * self.D

    @property
    def off_gate(self) -> int:
        return self.off_v + self.kv_heads * self.D

    @property
    def gate_cols(self) -> int:
        return {"": 0, "head": (self.heads + 7) // 8 * 8, "element": self.heads * self.D}[self.gate]

    @property
    def cols(self) -> int:
        return self.off_gate + self.gate_cols

    @property
    def out_cols(self) -> int:
        return self.heads * self.D


@dataclass
class AttentionWeights:
    """fp32 parameters besides the projections. ``bias`` [off_gate] or None. ``norm``: "" (none), "unit" (every q and k head over its
    root mean square), "head" (times q_norm, k_norm [D]), "whole" (all heads together, times q_norm [heads * D], k_norm). Values:
    (1 - vmix) v + vmix v_first where a first layer's values are given. Queries at position p times 1 + coef ln(floor((p + 1) / every) + 1)
    for ``q_temp`` = (coef, every)."""
    form: ScoreForm
    bias: Optional[torch.Tensor] = None
    norm: str = ""
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    eps: float = 0.0
    vmix: float = 0.0
    q_temp: Optional[tuple] = None


_NORMS = {"": 0, "unit": 1, "head": 2, "whole": 3}


def shaped_attention(proj: torch.Tensor, geo: AttentionGeometry, w: AttentionWeights, k_pool: torch.Tensor, v_pool: torch.Tensor,
                     angles, first_values, batch, out_scale: float = 1.0, out: torch.Tensor | None = None) -> torch.Tensor:
    """proj [T, geo.cols] -> [T, geo.out_cols] (``out`` may be columns of a wider matrix). ``angles``: the cache's table for
    ``geo.rotary``; ``first_values``: V pages (of any padded head size) whose values are mixed in, or None."""
    T, H, G, D = proj.shape[0], geo.heads, geo.kv_heads, geo.D
    bs = k_pool.shape[2]
    if out is None:
        out = torch.empty((T, geo.out_cols), device=proj.device, dtype=proj.dtype)
    if T == 0:
        return out
    gate = OutputGate(proj[:, geo.off_gate:geo.cols] if geo.gate else None, geo.gate == "element", out_scale)
    if not proj.is_cuda:
        return _shaped_torch(proj, geo, w, k_pool, v_pool, angles, first_values, batch, gate, out)
    st, dt = stream_ptr(proj.device), dtype_code(proj.dtype)
    nd, n = batch.n_decode, T - batch.n_decode
    q = torch.empty((T, H, D), device=proj.device, dtype=proj.dtype)
    seg = batch.segments(w.form.mask) if n and tensor_core_heads(D, proj.dtype) and bs % 8 == 0 else None
    stage = torch.empty((seg.keys, 2 * G, D), device=proj.device, dtype=proj.dtype) if seg is not None else None
    ints = (ctypes.c_int * 13)(T, H, G, D, geo.dim, geo.hp, geo.off_k, geo.off_v, _NORMS[w.norm], bs, nd, proj.stride(0),
                               first_values.shape[3] if first_values is not None else 0)
    floats = (ctypes.c_float * 4)(w.eps, w.vmix, *(w.q_temp or (0.0, 1.0)))
    ptrs = (ctypes.c_void_p * 13)(proj.data_ptr(), _ptr(w.bias), _ptr(w.q_norm), _ptr(w.k_norm), _ptr(angles), batch.positions.data_ptr(),
                                  batch.slots.data_ptr(), q.data_ptr(), k_pool.data_ptr(), v_pool.data_ptr(), _ptr(first_values), _ptr(stage),
                                  _ptr(seg.stage_rows) if seg is not None else None)
    check(lib().tsb_attn_prepare(ints, floats, ptrs, dt, st), "tsb_attn_prepare")
    _attend(q, stage, k_pool, v_pool, batch, w.form, gate, out)
    return out


def _shaped_torch(proj, geo, w, k_pool, v_pool, angles, first_values, batch, gate, out):
    T, H, G, D, bs = proj.shape[0], geo.heads, geo.kv_heads, geo.D, k_pool.shape[2]
    z = proj[:, :geo.off_gate].float()
    if w.bias is not None:
        z = z + w.bias
    q, k = z[:, :geo.off_k].view(T, H, D), z[:, geo.off_k:geo.off_k + G * D].view(T, G, D)
    v = z[:, geo.off_v:geo.off_gate].view(T, G, D)

    def norm(x, weight):
        if w.norm == "whole":
            s = (x * x).sum((1, 2), keepdim=True) / (x.shape[1] * geo.dim)
            return x / torch.sqrt(s + w.eps) * weight.view(x.shape[1], D)
        if w.norm:
            x = x / torch.sqrt((x * x).sum(-1, keepdim=True) / geo.dim + w.eps)
        return x * weight if w.norm == "head" else x
    q, k = norm(q, w.q_norm), norm(k, w.k_norm)
    if angles is not None:
        pos = batch.positions.long()
        q, k = rotate_stored(q, angles, pos), rotate_stored(k, angles, pos)
    if w.q_temp is not None:
        coef, every = w.q_temp
        q = q * (1.0 + coef * torch.log(torch.floor((batch.positions + 1).float() / every) + 1.0))[:, None, None]
    if first_values is not None:
        sl = batch.slots.long()
        first = torch.nn.functional.pad(first_values[sl // bs, :, sl % bs].float(), (0, max(0, D - first_values.shape[3])))
        v = (1.0 - w.vmix) * v + w.vmix * first[..., :D]
    return _attend_torch(q.to(proj.dtype), k.to(proj.dtype), v.to(proj.dtype), k_pool, v_pool, batch, w.form, gate, out)


def _attend_torch(q, keys, values, k_pool, v_pool, batch, form: ScoreForm, gate: OutputGate, out):
    """q [T, H, D], keys, values [T, G, D] -> out [T, H * D]; appends to the pools."""
    T, H, D = q.shape
    G, bs = keys.shape[1], k_pool.shape[2]
    window = form.mask.size if isinstance(form.mask, Window) else 0
    chunk = 0 if window else form.mask
    out[:, :H * D] = 0
    for i, (row0, n, slot, pos0) in enumerate(batch.spans()):
        if slot < 0:
            continue
        sl = batch.slots[row0:row0 + n].long()
        k_pool[sl // bs, :, sl % bs] = keys[row0:row0 + n]
        v_pool[sl // bs, :, sl % bs] = values[row0:row0 + n]
        total = pos0 + n
        k = _gather_request(k_pool, batch.tables[i], total).float().repeat_interleave(H // G, dim=0)
        v = _gather_request(v_pool, batch.tables[i], total).float().repeat_interleave(H // G, dim=0)
        s = (q[row0:row0 + n].float().transpose(0, 1) @ k.transpose(1, 2)) * form.scale
        if form.softcap:
            s = form.softcap * torch.tanh(s / form.softcap)
        qi, kj = torch.arange(pos0, total)[:, None], torch.arange(total)[None, :]
        if form.slopes is not None:
            s = s - form.slopes[:, None, None] * (qi - kj)
        hidden = kj > qi
        if chunk > 0:
            hidden |= (kj // chunk) != (qi // chunk)
        if window > 0:
            hidden |= qi - kj >= window
        s = s.masked_fill(hidden, float("-inf"))
        if form.sink is not None:                   # one more place, without a value
            s = torch.cat([s, form.sink[:, None, None].expand(H, n, 1)], dim=2)
        o = torch.softmax(s, dim=-1)[:, :, :total] @ v
        o = o.transpose(0, 1) * gate.scale
        if gate.gate is not None:
            g = torch.sigmoid(gate.gate[row0:row0 + n].float())
            o = o * (g[:, :H * D].view(n, H, D) if gate.per_element else g[:, :H, None])
        out[row0:row0 + n, :H * D] = o.reshape(n, H * D).to(out.dtype)
    return out
