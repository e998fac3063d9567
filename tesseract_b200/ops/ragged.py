"""Attention over paged pools for ragged batches: decoded rows (one token per sequence) first, then portions of prompts.

``ragged_attention`` takes a packed [q | k | v] projection, adds its biases, appends keys and values to the pool and
attends under an optional chunk mask (token i sees the tokens j <= i of its own run of ``chunk`` positions):

* decoded rows: the split-K paged kernel (``csrc/decode_attn_mma.cu``), which starts at the first key of the chunk;
* prompt rows: the tcgen05 kernel (``csrc/flash_attn_fwd.cu``) with every chunk of a portion as a sequence of its own; the
  keys that a portion needs from earlier ones are copied from the pool in front of its own;
* fp32 models and head sizes other than 64 / 128: one warp per (row, head) over the pool (``csrc/ragged_attn.cu``).

Query, key and value heads share one padded size ``D`` (zero columns change no score and no result).
"""
from __future__ import annotations

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr
from .paged import _decode_scratch, _gather_request, _scratch_floats

P, I, L, F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({
    "tsb_ragged_append": [P, L, P, P, P, P, P, P, P, I, I, I, I, I, I, I, P],
    "tsb_stage_gather": [P, P, P, P, P, I, I, I, I, P],
    "tsb_ragged_attn": [P, L, P, P, P, I, P, P, P, I, I, I, I, I, I, I, F, I, P],
    "tsb_paged_decode_chunked": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, F, I, I, I, P],
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


def ragged_attention(qkv: torch.Tensor, bias, k_pool: torch.Tensor, v_pool: torch.Tensor, batch, heads: int, kv_heads: int,
                     scale: float, chunk: int = 0) -> torch.Tensor:
    """qkv [T, (heads + 2 kv_heads) D] -> [T, heads * D]; pools [blocks, kv_heads, block, D]."""
    T, H, G, D = qkv.shape[0], heads, kv_heads, k_pool.shape[3]
    nb, _, bs, _ = k_pool.shape
    if T == 0:
        return qkv.new_empty((0, H * D))
    if not qkv.is_cuda:
        return _ragged_attention_torch(qkv, bias, k_pool, v_pool, batch, H, G, scale, chunk)
    st, dt = stream_ptr(qkv.device), dtype_code(qkv.dtype)
    nd, n = batch.n_decode, T - batch.n_decode
    fast = tensor_core_heads(D, qkv.dtype) and bs % 8 == 0
    q = torch.empty((T, H, D), device=qkv.device, dtype=qkv.dtype)
    seg = batch.segments(chunk) if fast and n else None
    stage = torch.empty((seg.keys, 2 * G, D), device=qkv.device, dtype=qkv.dtype) if seg is not None else None
    check(lib().tsb_ragged_append(qkv.data_ptr(), qkv.stride(0), bias.data_ptr() if bias is not None else None,
                                  batch.slots.data_ptr(), q.data_ptr(), k_pool.data_ptr(), v_pool.data_ptr(),
                                  stage.data_ptr() if stage is not None else None,
                                  seg.stage_rows.data_ptr() if seg is not None else None, nd, T, H, G, D, bs, dt, st),
          "tsb_ragged_append")
    o = torch.empty((T, H, D), device=qkv.device, dtype=qkv.dtype)
    tables = batch.tables
    if not fast:
        check(lib().tsb_ragged_attn(q.data_ptr(), H * D, k_pool.data_ptr(), v_pool.data_ptr(), tables.data_ptr(), tables.stride(0),
                                    batch.seq_of.data_ptr(), batch.positions.data_ptr(), o.data_ptr(), T, H, G, D, bs, nb,
                                    int(chunk), float(scale), dt, st), "tsb_ragged_attn")
        return o.view(T, H * D)
    if nd:
        # planned for the longest sequence the tables can hold, so that a captured launch serves every later step
        longest = batch.max_len
        span = min(longest, chunk) if chunk > 0 else longest
        scratch = _decode_scratch(qkv.device, _scratch_floats(nd, H, G, D, span, False))
        args = (q.data_ptr(), k_pool.data_ptr(), v_pool.data_ptr())
        if chunk > 0:
            check(lib().tsb_paged_decode_chunked(*args, tables.data_ptr(), batch.lens.data_ptr(), o.data_ptr(), scratch.data_ptr(),
                                                 nd, H, G, D, bs, nb, tables.stride(0), float(scale), longest, int(chunk), dt, st),
                  "tsb_paged_decode_chunked")
        else:
            check(lib().tsb_paged_decode(*args, None, None, tables.data_ptr(), batch.lens.data_ptr(), o.data_ptr(),
                                         scratch.data_ptr(), nd, H, G, D, bs, nb, tables.stride(0), float(scale), longest, dt, st),
                  "tsb_paged_decode")
    if n:
        if seg.n_gather:
            check(lib().tsb_stage_gather(k_pool.data_ptr(), v_pool.data_ptr(), stage.data_ptr(), seg.gather_dst.data_ptr(),
                                         seg.gather_src.data_ptr(), seg.n_gather, G, D, bs, st), "tsb_stage_gather")
        qp, op, vp = q[nd:], o[nd:], stage[:, G:]
        check(lib().tsb_flash_fwd_varlen_keys(qp.data_ptr(), stage.data_ptr(), vp.data_ptr(), op.data_ptr(), seg.cu_q.data_ptr(),
                                              seg.cu_k.data_ptr(), seg.n, seg.max_q, n, seg.keys, H, G, D, H * D, D, 2 * G * D, D,
                                              2 * G * D, D, H * D, D, float(scale), st), "tsb_flash_fwd_varlen_keys")
    return o.view(T, H * D)


def _ragged_attention_torch(qkv, bias, k_pool, v_pool, batch, H, G, scale, chunk):
    T, D, bs = qkv.shape[0], k_pool.shape[3], k_pool.shape[2]
    z = qkv.float() + bias if bias is not None else qkv.float()
    z = z.to(qkv.dtype).view(T, H + 2 * G, D)
    out = torch.zeros(T, H, D, dtype=qkv.dtype)
    for i, (row0, n, slot, pos0) in enumerate(batch.spans()):
        if slot < 0:
            continue
        sl = batch.slots[row0:row0 + n].long()
        k_pool[sl // bs, :, sl % bs] = z[row0:row0 + n, H:H + G]
        v_pool[sl // bs, :, sl % bs] = z[row0:row0 + n, H + G:]
        total = pos0 + n
        k = _gather_request(k_pool, batch.tables[i], total).float().repeat_interleave(H // G, dim=0)
        v = _gather_request(v_pool, batch.tables[i], total).float().repeat_interleave(H // G, dim=0)
        s = (z[row0:row0 + n, :H].float().transpose(0, 1) @ k.transpose(1, 2)) * scale
        qi, kj = torch.arange(pos0, total)[:, None], torch.arange(total)[None, :]
        hidden = kj > qi
        if chunk > 0:
            hidden |= (kj // chunk) != (qi // chunk)
        p = torch.softmax(s.masked_fill(hidden, float("-inf")), dim=-1)
        out[row0:row0 + n] = (p @ v).transpose(0, 1).to(qkv.dtype)
    return out.view(T, H * D)
