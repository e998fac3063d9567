"""Fused bandwidth-bound ops with autograd: RMSNorm (+ residual), SwiGLU, RoPE on packed QKV,
embedding, cross-entropy. CUDA tensors run the sm_100a kernels of ``csrc/fused_norm_act.cu`` and
``csrc/loss_optim.cu``; CPU tensors run the plain torch restatement of the reference's math, which is
also the oracle the kernels are tested against.

Reference semantics: RMSNorm composite (src/ops/cpu/RMSNorm.cpp:49-97), SwiGLU ``silu(gate) * up``
(src/ops/cpu/SwiGLU.cpp:106-115), adjacent-pair RoPE (src/ops/cpu/RotaryEmbedding.cpp,
src/nn/RotaryEmbedding.cpp:35-57), mean cross-entropy with int64 targets (src/ops/cpu/Loss.cpp:154).
"""
from __future__ import annotations

import math

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr

_NATIVE_DTYPES = (torch.float32, torch.bfloat16, torch.float16)


def _native_ok(t: torch.Tensor) -> bool:
    return t.is_cuda and t.dtype in _NATIVE_DTYPES


# --------------------------------------------------------------------------------------- RMSNorm
def rms_norm_ref(x, weight, eps):
    xf = x.float()
    rstd = torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (xf * rstd * weight.float()).to(x.dtype)


class _RMSNormFn(torch.autograd.Function):
    """y = rmsnorm(x [+ residual]) * w. Returns (y, h) where h = x + residual (or x itself)."""

    @staticmethod
    def forward(ctx, x, residual, weight, eps, wgrad_buf):
        ctx.set_materialize_grads(False)
        D = x.shape[-1]
        x2 = x.reshape(-1, D).contiguous()
        rows = x2.shape[0]
        y = torch.empty(x.shape, device=x.device, dtype=x.dtype)
        rstd = torch.empty(rows, device=x.device, dtype=torch.float32)
        if residual is not None:
            r2 = residual.reshape(-1, D).contiguous()
            h = torch.empty(x.shape, device=x.device, dtype=x.dtype)
            check(lib().tsb_rmsnorm_fwd(x2.data_ptr(), r2.data_ptr(), weight.data_ptr(), y.data_ptr(), h.data_ptr(),
                                        rstd.data_ptr(), rows, D, eps, dtype_code(x.dtype), stream_ptr(x.device)),
                  "tsb_rmsnorm_fwd")
        else:
            h = x2
            check(lib().tsb_rmsnorm_fwd(x2.data_ptr(), None, weight.data_ptr(), y.data_ptr(), None,
                                        rstd.data_ptr(), rows, D, eps, dtype_code(x.dtype), stream_ptr(x.device)),
                  "tsb_rmsnorm_fwd")
        ctx.save_for_backward(h, weight, rstd)
        ctx.has_res = residual is not None
        ctx.wgrad_buf = wgrad_buf
        ctx.shape = x.shape
        return y, (h if residual is not None else None)

    @staticmethod
    def backward(ctx, dy, dh):
        h, weight, rstd = ctx.saved_tensors
        D = h.shape[-1]
        h = h.reshape(-1, D)
        rows = h.shape[0]
        if dy is None:
            dy = torch.zeros(ctx.shape, device=h.device, dtype=h.dtype)
        dy2 = dy.reshape(-1, D).contiguous()
        dh2 = dh.reshape(-1, D).contiguous() if dh is not None else None
        dx = torch.empty_like(h)
        parts = lib().tsb_rmsnorm_bwd_parts(rows)
        partial = torch.empty((parts, D), device=h.device, dtype=torch.float32)
        buf = ctx.wgrad_buf
        if buf is not None and buf.dtype == weight.dtype:
            dw_t, acc, dw_ret = buf, 1, None
        else:
            dw_t = torch.empty_like(weight)
            acc, dw_ret = 0, dw_t
        check(lib().tsb_rmsnorm_bwd(dy2.data_ptr(), h.data_ptr(), weight.data_ptr(), rstd.data_ptr(),
                                    dh2.data_ptr() if dh2 is not None else None, dx.data_ptr(), dw_t.data_ptr(),
                                    partial.data_ptr(), rows, D, acc, dtype_code(h.dtype), stream_ptr(h.device)),
              "tsb_rmsnorm_bwd")
        _native.add_launches(1)
        if buf is not None and dw_ret is not None:
            buf.add_(dw_ret.to(buf.dtype))
            dw_ret = None
        dx = dx.view(ctx.shape)
        return dx, (dx if ctx.has_res else None), dw_ret, None, None


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float = 1e-5, residual: torch.Tensor | None = None,
             wgrad_buf: torch.Tensor | None = None):
    """RMSNorm over the last dimension. With ``residual`` returns ``(y, x + residual)``; else ``y``."""
    if _native_ok(x) and x.shape[-1] % 8 == 0 and x.shape[-1] <= 8192 and weight.dtype == x.dtype:
        y, h = _RMSNormFn.apply(x, residual, weight, float(eps), wgrad_buf)
        return (y, h) if residual is not None else y
    if residual is not None:
        h = x + residual
        return _ref_norm_with_buf(h, weight, eps, wgrad_buf), h
    return _ref_norm_with_buf(x, weight, eps, wgrad_buf)


class _GradToBuf(torch.autograd.Function):
    """Identity on a parameter whose gradient is added into ``buf`` instead of ``param.grad``."""

    @staticmethod
    def forward(ctx, w, buf):
        ctx.buf = buf
        return w.view_as(w)

    @staticmethod
    def backward(ctx, g):
        ctx.buf.add_(g.to(ctx.buf.dtype))
        return None, None


def grad_to_buf(w: torch.Tensor, buf: torch.Tensor | None) -> torch.Tensor:
    if buf is None or not (torch.is_grad_enabled() and w.requires_grad):
        return w
    return _GradToBuf.apply(w, buf)


def _ref_norm_with_buf(x, weight, eps, wgrad_buf):
    return rms_norm_ref(x, grad_to_buf(weight, wgrad_buf), eps)


# --------------------------------------------------------------------------------------- SwiGLU
def swiglu_ref(gate_up: torch.Tensor) -> torch.Tensor:
    F = gate_up.shape[-1] // 2
    g, u = gate_up[..., :F].float(), gate_up[..., F:].float()
    return (torch.nn.functional.silu(g) * u).to(gate_up.dtype)


class _SwiGLUFn(torch.autograd.Function):
    @staticmethod
    def forward(ctx, gate_up):
        F = gate_up.shape[-1] // 2
        gu = gate_up.reshape(-1, 2 * F).contiguous()
        out = torch.empty((gu.shape[0], F), device=gu.device, dtype=gu.dtype)
        check(lib().tsb_swiglu_fwd(gu.data_ptr(), out.data_ptr(), gu.shape[0], F, dtype_code(gu.dtype),
                                   stream_ptr(gu.device)), "tsb_swiglu_fwd")
        ctx.save_for_backward(gu)
        ctx.shape = gate_up.shape
        return out.view(*gate_up.shape[:-1], F)

    @staticmethod
    def backward(ctx, dout):
        (gu,) = ctx.saved_tensors
        F = gu.shape[-1] // 2
        d2 = dout.reshape(-1, F).contiguous()
        dgu = torch.empty_like(gu)
        check(lib().tsb_swiglu_bwd(d2.data_ptr(), gu.data_ptr(), dgu.data_ptr(), gu.shape[0], F,
                                   dtype_code(gu.dtype), stream_ptr(gu.device)), "tsb_swiglu_bwd")
        return dgu.view(ctx.shape)


def swiglu_backward(gate_up: torch.Tensor, dout: torch.Tensor) -> torch.Tensor:
    """Gradient of ``swiglu`` with respect to the packed [rows, 2F] input (CUDA kernel; no autograd)."""
    F = gate_up.shape[-1] // 2
    gu = gate_up.reshape(-1, 2 * F).contiguous()
    d2 = dout.reshape(-1, F).contiguous()
    dgu = torch.empty_like(gu)
    check(lib().tsb_swiglu_bwd(d2.data_ptr(), gu.data_ptr(), dgu.data_ptr(), gu.shape[0], F, dtype_code(gu.dtype),
                               stream_ptr(gu.device)), "tsb_swiglu_bwd")
    return dgu.view(gate_up.shape)


def swiglu(gate_up: torch.Tensor) -> torch.Tensor:
    """silu(gate) * up for a packed [..., 2F] tensor (gate = first half of the last dimension)."""
    F = gate_up.shape[-1] // 2
    if _native_ok(gate_up) and F % 8 == 0:
        return _SwiGLUFn.apply(gate_up)
    return swiglu_ref(gate_up)


def swiglu_silu_gate(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """Two-operand form of the reference API (``ops::swiglu_silu_gate``)."""
    if _native_ok(gate) and gate.shape[-1] % 8 == 0:
        return swiglu(torch.cat([gate, up], dim=-1))
    return (torch.nn.functional.silu(gate.float()) * up.float()).to(gate.dtype)


# --------------------------------------------------------------------------------------- RoPE
def rope_tables(max_pos: int, head_dim: int, theta: float, device=None) -> tuple[torch.Tensor, torch.Tensor]:
    """cos/sin tables [max_pos, head_dim/2] (fp32): angle(p, j) = p * theta^(-2j/d)."""
    j = torch.arange(0, head_dim, 2, dtype=torch.float64)
    inv = theta ** (-j / head_dim)
    ang = torch.arange(max_pos, dtype=torch.float64)[:, None] * inv[None, :]
    return ang.cos().float().to(device), ang.sin().float().to(device)


def rope_ref(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    """Adjacent-pair rotation of x [..., T, H, D] (positions [T] or broadcastable [..., T])."""
    c = cos[positions].unsqueeze(-2)  # [..., T, 1, D/2]
    s = sin[positions].unsqueeze(-2)
    xf = x.float()
    a, b = xf[..., 0::2], xf[..., 1::2]
    out = torch.stack((a * c - b * s, a * s + b * c), dim=-1).flatten(-2)
    return out.to(x.dtype)


class _RopeQKVFn(torch.autograd.Function):
    """In-place rotation of the query and key heads of a packed [T, (Hq + 2 Hkv) * D] buffer."""

    @staticmethod
    def forward(ctx, qkv, cos, sin, positions, seq_len, pos_offset, hq, hkv, D):
        assert qkv.is_contiguous()
        T = qkv.shape[0]
        check(lib().tsb_rope_qkv(qkv.data_ptr(), cos.data_ptr(), sin.data_ptr(),
                                 positions.data_ptr() if positions is not None else None, T, seq_len, pos_offset,
                                 hq + hkv, hq + 2 * hkv, D, 1.0, dtype_code(qkv.dtype), stream_ptr(qkv.device)),
              "tsb_rope_qkv")
        ctx.mark_dirty(qkv)
        ctx.save_for_backward(cos, sin, positions)
        ctx.args = (seq_len, pos_offset, hq, hkv, D)
        return qkv

    @staticmethod
    def backward(ctx, dqkv):
        cos, sin, positions = ctx.saved_tensors
        seq_len, pos_offset, hq, hkv, D = ctx.args
        d = dqkv.contiguous()
        if d.data_ptr() == dqkv.data_ptr():
            d = d.clone()
        check(lib().tsb_rope_qkv(d.data_ptr(), cos.data_ptr(), sin.data_ptr(),
                                 positions.data_ptr() if positions is not None else None, d.shape[0], seq_len,
                                 pos_offset, hq + hkv, hq + 2 * hkv, D, -1.0, dtype_code(d.dtype),
                                 stream_ptr(d.device)), "tsb_rope_qkv")
        return d, None, None, None, None, None, None, None, None


def rope_qkv(qkv: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, *, num_heads: int, num_kv_heads: int,
             head_dim: int, seq_len: int, pos_offset: int = 0, positions: torch.Tensor | None = None) -> torch.Tensor:
    """Rotate the Q and K heads of packed ``qkv`` [T, (Hq + 2 Hkv) * D]; token t sits at position
    ``positions[t]`` (int32) or ``pos_offset + t % seq_len``. V is left untouched."""
    T = qkv.shape[0]
    if _native_ok(qkv) and head_dim % 8 == 0:
        if positions is not None:
            positions = positions.to(torch.int32)
        return _RopeQKVFn.apply(qkv, cos, sin, positions, seq_len, pos_offset, num_heads, num_kv_heads, head_dim)
    if positions is None:
        positions = pos_offset + (torch.arange(T, device=qkv.device) % seq_len)
    x = qkv.view(T, num_heads + 2 * num_kv_heads, head_dim)
    rot = rope_ref(x[:, : num_heads + num_kv_heads], cos, sin, positions.long())
    return torch.cat([rot, x[:, num_heads + num_kv_heads:]], dim=1).reshape(T, -1)


# --------------------------------------------------------------------------------------- embedding
class _EmbeddingFn(torch.autograd.Function):
    @staticmethod
    def forward(ctx, ids, table, wgrad_buf):
        flat = ids.reshape(-1).contiguous()
        D = table.shape[1]
        out = torch.empty((flat.numel(), D), device=table.device, dtype=table.dtype)
        check(lib().tsb_embedding_fwd(flat.data_ptr(), table.data_ptr(), out.data_ptr(), flat.numel(), D,
                                      table.shape[0], dtype_code(table.dtype), stream_ptr(table.device)),
              "tsb_embedding_fwd")
        ctx.save_for_backward(flat)
        ctx.wgrad_buf = wgrad_buf
        ctx.tshape = table.shape
        ctx.tdtype = table.dtype
        return out.view(*ids.shape, D)

    @staticmethod
    def backward(ctx, dy):
        (flat,) = ctx.saved_tensors
        V, D = ctx.tshape
        d2 = dy.reshape(-1, D).contiguous()
        buf = ctx.wgrad_buf
        ret = None
        if buf is not None and buf.dtype in (torch.float32, torch.bfloat16):
            tgt = buf
        else:
            tgt = torch.zeros((V, D), device=dy.device, dtype=torch.float32)
            ret = tgt
        check(lib().tsb_embedding_bwd(flat.data_ptr(), d2.data_ptr(), tgt.data_ptr(), flat.numel(), D, V,
                                      dtype_code(d2.dtype), int(tgt.dtype == torch.float32), stream_ptr(dy.device)),
              "tsb_embedding_bwd")
        if ret is not None:
            ret = ret.to(ctx.tdtype)
            if buf is not None:
                buf.add_(ret.to(buf.dtype))
                ret = None
        return None, ret, None


def embedding(ids: torch.Tensor, table: torch.Tensor, wgrad_buf: torch.Tensor | None = None) -> torch.Tensor:
    """Row gather ``table[ids]`` for int64 ids (validated against the vocabulary size)."""
    if ids.dtype != torch.int64:
        raise TypeError("embedding: ids must be int64")
    if _native_ok(table) and table.shape[1] % 8 == 0 and ids.is_cuda:
        return _EmbeddingFn.apply(ids, table, wgrad_buf)
    return torch.nn.functional.embedding(ids, grad_to_buf(table, wgrad_buf))


# --------------------------------------------------------------------------------------- cross-entropy
def cross_entropy_ref(logits: torch.Tensor, targets: torch.Tensor) -> torch.Tensor:
    lf = logits.float()
    return (torch.logsumexp(lf, -1) - lf.gather(-1, targets[:, None]).squeeze(-1)).mean()


def ce_stats(logits: torch.Tensor, targets: torch.Tensor, vocab_start: int = 0) -> torch.Tensor:
    """Per-row {max, sum exp(x - max), target logit (0 if not in this shard)} -> fp32 [rows, 3]."""
    rows, V = logits.shape
    if _native_ok(logits):
        stats = torch.empty((rows, 3), device=logits.device, dtype=torch.float32)
        check(lib().tsb_ce_stats(logits.data_ptr(), targets.data_ptr(), stats.data_ptr(), rows, V, logits.stride(0),
                                 vocab_start, dtype_code(logits.dtype), stream_ptr(logits.device)), "tsb_ce_stats")
        return stats
    lf = logits.float()
    m = lf.max(-1).values
    s = (lf - m[:, None]).exp().sum(-1)
    loc = targets - vocab_start
    inside = (loc >= 0) & (loc < V)
    tl = torch.where(inside, lf.gather(-1, loc.clamp(0, V - 1)[:, None]).squeeze(-1), torch.zeros_like(m))
    return torch.stack([m, s, tl], dim=-1)


def merge_ce_stats(stats_list: list[torch.Tensor]) -> torch.Tensor:
    """Combine per-shard stats of the same rows (what a vocab-parallel all-reduce computes)."""
    m = torch.stack([s[:, 0] for s in stats_list]).max(0).values
    ssum = sum(s[:, 1] * (s[:, 0] - m).exp() for s in stats_list)
    tl = sum(s[:, 2] for s in stats_list)
    return torch.stack([m, ssum, tl], dim=-1)


def ce_loss_and_grad_(logits: torch.Tensor, targets: torch.Tensor, stats: torch.Tensor, grad_scale: float,
                      vocab_start: int = 0, write_grad: bool = True) -> torch.Tensor:
    """Per-row losses (fp32 [rows]); when ``write_grad`` the logits are overwritten IN PLACE with
    ``(softmax - onehot) * grad_scale``. Rows with a negative target contribute nothing."""
    rows, V = logits.shape
    if _native_ok(logits):
        loss_rows = torch.empty(rows, device=logits.device, dtype=torch.float32)
        check(lib().tsb_ce_loss_grad(logits.data_ptr(), targets.data_ptr(), stats.data_ptr(), loss_rows.data_ptr(),
                                     rows, V, logits.stride(0), vocab_start, float(grad_scale), int(write_grad),
                                     dtype_code(logits.dtype), stream_ptr(logits.device)), "tsb_ce_loss_grad")
        return loss_rows
    m, s, tl = stats[:, 0], stats[:, 1], stats[:, 2]
    ignored = targets < 0
    loss_rows = torch.where(ignored, torch.zeros_like(m), s.log() + m - tl)
    if write_grad:
        p = (logits.float() - m[:, None]).exp() / s[:, None]
        loc = targets - vocab_start
        inside = (loc >= 0) & (loc < V) & ~ignored
        rows_idx = torch.nonzero(inside).squeeze(-1)
        p[rows_idx, loc[rows_idx]] -= 1.0
        p = p * grad_scale
        p[ignored] = 0
        logits.copy_(p.to(logits.dtype))
    return loss_rows


class _CrossEntropyFn(torch.autograd.Function):
    @staticmethod
    def forward(ctx, logits, targets):
        work = logits.detach().clone()
        stats = ce_stats(work, targets)
        n = logits.shape[0]
        loss_rows = ce_loss_and_grad_(work, targets, stats, 1.0 / n)
        ctx.save_for_backward(work)
        return loss_rows.sum() / n

    @staticmethod
    def backward(ctx, g):
        (grad,) = ctx.saved_tensors
        return (grad.float() * g).to(grad.dtype), None


def cross_entropy(logits: torch.Tensor, targets: torch.Tensor) -> torch.Tensor:
    """Mean over rows of ``logsumexp(row) - row[target]``; ``logits`` [N, V], ``targets`` int64 [N]."""
    if logits.dim() != 2 or targets.dim() != 1 or targets.shape[0] != logits.shape[0]:
        raise ValueError("cross_entropy expects logits [N, V] and targets [N]")
    if targets.dtype != torch.int64:
        raise TypeError("cross_entropy: targets must be int64")
    if _native_ok(logits):
        return _CrossEntropyFn.apply(logits.contiguous(), targets.contiguous())
    return cross_entropy_ref(logits, targets)


# --------------------------------------------------------------------------------------- residual steps, clamped GLU
_P, _I, _L, _F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({
    "tsb_dyn_tanh_residual": [_P, _I, _I, _P, _L, _P, _F, _P, _P, _P, _P, _L, _F, _I, _I, _P, _F, _P, _P, _P, _L, _I, _I, _P],
    "tsb_clamped_glu": [_P, _L, _P, _P, _L, _I, _I, _F, _F, _F, _F, _F, _I, _P],
    "tsb_depth_residual": [_P, _P, _P, _L, _P, _I, _I, _P, _L, _F, _P, _P, _L, _I, _P, _L, _I, _I, _I, _F, _F, _I, _P],
})
_EMBED_MODES = {None: 0, "set": 1, "add": 2}


def _ptr(t):
    return t.data_ptr() if t is not None else None


def dyn_tanh_residual(x, y=None, y_bias=None, post=None, tokens=None, table=None, scale=1.0, embed=None, step=None,
                      next_norm=None, out_cols=0, out_dtype=None):
    """One step of an fp32 residual stream ``x`` [T, W] (updated in place) between two matrix products; norms are
    (alpha, weight, bias) triples meaning tanh(alpha z) * weight + bias, all in fp32:

        x  = table[tokens] * scale                 (embed="set")
        x += post(y + y_bias)                      (y given)
        x += table[tokens] * scale                 (embed="add")
        x += step                                  (step given)
        return next_norm(x)                        (next_norm given: [T, out_cols], zero past W, ``out_dtype``)
    """
    T, W = x.shape
    h = None
    if next_norm is not None:
        h = torch.empty((T, out_cols or W), device=x.device, dtype=out_dtype or (y.dtype if y is not None else table.dtype))
    if T == 0:
        return h
    if x.is_cuda:
        act = next(t for t in (h, y, table) if t is not None)
        for t in (y, table, h):
            if t is not None and (t.dtype != act.dtype or t.stride(-1) != 1):
                raise ValueError("dyn_tanh_residual: y, table and the result share one dtype and have contiguous rows")
        pa, pw, pb = post if post is not None else (0.0, None, None)
        na, nw, nb = next_norm if next_norm is not None else (0.0, None, None)
        check(lib().tsb_dyn_tanh_residual(
            x.data_ptr(), T, W, _ptr(y), y.stride(0) if y is not None else 0, _ptr(y_bias), float(pa), _ptr(pw), _ptr(pb),
            _ptr(tokens), _ptr(table), table.stride(0) if table is not None else 0, float(scale), _EMBED_MODES[embed],
            table.shape[0] if table is not None else 0, _ptr(step), float(na), _ptr(nw), _ptr(nb), _ptr(h),
            h.stride(0) if h is not None else 0, h.shape[1] if h is not None else 0, dtype_code(act.dtype),
            stream_ptr(x.device)), "tsb_dyn_tanh_residual")
        return h
    e = table[tokens.long(), :W].float() * scale if embed is not None else None
    if embed == "set":
        x.copy_(e)
    if y is not None:
        z = y[:, :W].float()
        if y_bias is not None:
            z = z + y_bias
        x.add_(torch.tanh(post[0] * z) * post[1] + post[2])
    if embed == "add":
        x.add_(e)
    if step is not None:
        x.add_(step)
    if h is not None:
        h[:, W:] = 0
        h[:, :W] = torch.tanh(next_norm[0] * x) * next_norm[1] + next_norm[2]
    return h


def clamped_glu(gate_up, bias, limit, slope=1.702, shift=1.0, in_scale=1.0, out=None, cubic=0.0):
    """gate_up [T, 2 F] (gate, then up; times ``in_scale``, plus ``bias`` fp32 [2 F] if given) ->
    g sigmoid(slope (g + cubic g^3)) (u + shift) with g = min(gate, limit), u = clamp(up, -limit, limit). ``out`` may be columns of a wider matrix."""
    T, F2 = gate_up.shape
    F = F2 // 2
    if out is None:
        out = torch.empty((T, F), device=gate_up.device, dtype=gate_up.dtype)
    if T == 0:
        return out
    if gate_up.is_cuda:
        check(lib().tsb_clamped_glu(gate_up.data_ptr(), gate_up.stride(0), _ptr(bias), out.data_ptr(), out.stride(0), T, F,
                                    float(limit), float(slope), float(shift), float(in_scale), float(cubic), dtype_code(gate_up.dtype),
                                    stream_ptr(gate_up.device)), "tsb_clamped_glu")
        return out
    z = gate_up.float() * in_scale
    if bias is not None:
        z = z + bias
    g, u = z[:, :F].clamp(max=limit), z[:, F:].clamp(-limit, limit)
    return out.copy_(g * torch.sigmoid(slope * (g + cubic * g ** 3)) * (u + shift))


def silu_glu(gate_up, in_scale=1.0, out=None):
    """SiLU(gate) * up of the two halves of a row, both times ``in_scale`` first."""
    return clamped_glu(gate_up, None, math.inf, 1.0, 0.0, in_scale, out)


def gelu_glu(gate_up, in_scale=1.0, out=None):
    """The tanh form of GELU(gate) * up: (1 + tanh z) / 2 = sigmoid(2 z)."""
    return clamped_glu(gate_up, None, math.inf, 2.0 * math.sqrt(2.0 / math.pi), 0.0, in_scale, out, 0.044715)


def depth_residual(x_in=None, y=None, mult=1.0, tokens=None, table=None, width=0, history=None, depth=0, average=None, store=True,
                   gain=1.0, eps=0.0, out_cols=0, out_dtype=None, want_h=True):
    """One step of an fp32 residual stream between two matrix products, with depth averaging and an RMS norm of one gain:

        X = table[tokens]  or  x_in + mult * y
        x = sum_j average[j] history[j] + average[depth] X, j < depth    (average given; else x = X)
        h = x / sqrt(mean(x^2) + eps) * gain

    ``history`` [entries, T, width] (fp32) receives X as entry ``depth`` when ``store``. Returns (x, h [T, out_cols] in
    ``out_dtype`` with zeros past the width, or None); at the start of the model x is the stored entry itself."""
    start = tokens is not None
    T, W = (tokens.shape[0], width) if start else x_in.shape
    dev = table.device if start else x_in.device
    src = table if start else y
    h = torch.empty((T, out_cols or W), device=dev, dtype=out_dtype or src.dtype) if want_h else None
    store = store and history is not None
    alias = start and store and average is None
    x = history[depth] if alias else torch.empty((T, W), device=dev, dtype=torch.float32)
    if T == 0:
        return x, h
    if x.is_cuda:
        if h is not None and h.dtype != src.dtype:
            raise ValueError("depth_residual: the input and the result share one dtype")
        check(lib().tsb_depth_residual(_ptr(x_in), None if alias else x.data_ptr(), _ptr(history),
                                       history.stride(0) if history is not None else 0, _ptr(average), depth, int(store),
                                       _ptr(y), y.stride(0) if y is not None else 0, float(mult), _ptr(tokens), _ptr(table),
                                       table.stride(0) if start else 0, table.shape[0] if start else 0, _ptr(h),
                                       h.stride(0) if h is not None else 0, h.shape[1] if h is not None else 0, T, W, float(gain), float(eps),
                                       dtype_code(src.dtype), stream_ptr(dev)), "tsb_depth_residual")
        return x, h
    new = table[tokens.long(), :W].float() if start else x_in + mult * y[:, :W].float()
    if store:
        history[depth].copy_(new)
    if average is not None:
        new = average[depth] * new + (average[:depth, None, None] * history[:depth]).sum(0)
    if not alias:
        x.copy_(new)
    if h is not None:
        h[:, W:] = 0
        h[:, :W] = new / torch.sqrt((new * new).mean(-1, keepdim=True) + eps) * gain
    return x, h


_native.register_signatures({
    "tsb_post_norm_step": [_P, _P, _L, _P, _P, _F, _P, _P, _L, _I, _F, _P, _L, _I, _I, _I, _I, _P],
    "tsb_gelu_lookup": [_P, _L, _P, _P, _L, _I, _I, _P, _L, _I, _I, _I, _I, _P],
})


def post_norm_step(x, y=None, gain=None, eps=0.0, tokens=None, table=None, scale=1.0, final=None, out_cols=0, out_dtype=None, out=None):
    """One step of an fp32 residual stream ``x`` [T, W] (updated in place) whose sublayers are normed on their way in:

        x  = table[tokens] * scale                          (tokens given)
        x += y / sqrt(mean(y^2) + eps) * gain               (y given; gain fp32 [W])
        return x, or x / sqrt(mean(x^2) + eps) * final      (final fp32 [W]; [T, out_cols], zero past W, ``out_dtype``)

    ``out``: receives the result when given."""
    T, W = x.shape
    h = out if out is not None else torch.empty((T, out_cols or W), device=x.device,
                                                dtype=out_dtype or (y.dtype if y is not None else table.dtype))
    if T == 0:
        return h
    if x.is_cuda:
        start = tokens is not None
        if y is not None and y.dtype != h.dtype or start and table.dtype != h.dtype:
            raise ValueError("post_norm_step: the inputs and the result share one dtype")
        check(lib().tsb_post_norm_step(x.data_ptr(), _ptr(y), y.stride(0) if y is not None else 0, _ptr(gain), _ptr(final),
                                       float(eps), _ptr(tokens), _ptr(table) if start else None, table.stride(0) if start else 0,
                                       table.shape[0] if start else 0, float(scale), h.data_ptr(), h.stride(0), h.shape[1], T, W,
                                       dtype_code(h.dtype), stream_ptr(x.device)), "tsb_post_norm_step")
        return h
    if tokens is not None:
        x.copy_(table[tokens.long(), :W].float() * scale)
    if y is not None:
        z = y[:, :W].float()
        x += z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps) * gain
    h[:, W:] = 0
    h[:, :W] = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * final if final is not None else x
    return h


def gelu_lookup(g, tokens, table, first, dim):
    """gelu_tanh(g[:, :dim]) * table[tokens, first:first + dim] as [T, cols of g] (zero past ``dim``)."""
    T = g.shape[0]
    out = torch.empty_like(g)
    if T == 0:
        return out
    if g.is_cuda:
        check(lib().tsb_gelu_lookup(g.data_ptr(), g.stride(0), tokens.data_ptr(), table.data_ptr(), table.stride(0), table.shape[0],
                                    first, out.data_ptr(), out.stride(0), out.shape[1], T, dim, dtype_code(g.dtype),
                                    stream_ptr(g.device)), "tsb_gelu_lookup")
        return out
    out[:, dim:] = 0
    e = table[tokens.long(), first:first + dim].float()
    out[:, :dim] = torch.nn.functional.gelu(g[:, :dim].float(), approximate="tanh") * e
    return out
