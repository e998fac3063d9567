"""Residual step of models that norm what their sublayers read (``csrc/pre_norm.cu``): an fp32 stream, norms in equal parts of the row, a
sinusoid of the position at the start, a scale per channel on what is added, and the token shift of a mixer's input."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr
from .moe import Mixed
from .timemix import token_shift

P, I, F = _native.P, _native.I, _native.F
_native.register_signatures({"tsb_pre_norm_step": [P, P, P, F, I, P]})
NORM_UNITS, NORM_UNIT = 128, (32, 128)      # a row is at most so many runs of 32 columns (128 where parts are multiples of 4) inside parts
SHIFT_ROWS = 1024            # prompt rows of a step up to which the shift is part of it


def _ptr(t):
    return t.data_ptr() if t is not None else None


@dataclass
class Moved:
    """Last rows of a step's portions that the next ``pre_norm_step`` puts into their slots."""
    tail: torch.Tensor
    last: torch.Tensor
    slots: torch.Tensor


@dataclass
class Shift:
    """h + (h' - h) mu with h' of the token before, rounded to the type of h: ``mu`` fp32 [columns of h]; ``last`` [slots, 1, columns of h]
    carries the last row of every sequence."""
    mu: torch.Tensor
    last: torch.Tensor


def sinusoid_frequencies(width):
    """[ceil(width / 2), 2]: 10000^(-2 i / width) as a sum of two fp32 numbers."""
    f = 10000.0 ** (-torch.arange(0, width, 2, dtype=torch.float64) / width)
    hi = f.float()
    return torch.stack([hi, (f - hi.double()).float()], dim=1).contiguous()


def _part_norm(x, gain, parts, eps):
    z = x.view(x.shape[0], parts, -1)
    return (z / torch.sqrt((z * z).mean(-1, keepdim=True) + eps)).reshape(x.shape) * gain


def pre_norm_step(batch, width, gain, parts, eps, x=None, y=None, bias=None, scale=None, table=None, freq=None, embed_gain=None, shift=None,
                  moved=None, out_cols=0, out_dtype=None):
    """One step of an fp32 residual stream whose sublayers read it through norms in ``parts`` (every part over its own root mean
    square), for the rows of ``batch``:

        x = norm(table[tokens] + sinusoid(positions)) embed_gain    (table given; the sinusoid with ``freq``, the norm with a gain)
        x = x + scale (y + bias)                                    (y given, also a ``moe.Mixed``; scale, bias fp32 [W] or None)
        h = norm(x) gain, and with ``shift`` h + (h' - h) mu

    Returns (x [T, W] -- a new tensor, h [T, out_cols] in ``out_dtype`` with zeros past W, Moved or None). What a shift of this step
    leaves for the slots of its portions is passed to the next step as ``moved``."""
    T, W = batch.tokens.shape[0], width
    start = table is not None
    dev = table.device if start else x.device
    h = torch.empty((T, out_cols or W), device=dev, dtype=out_dtype or (table.dtype if start else torch.float32))
    if shift is not None and h.is_cuda and T - batch.n_decode > SHIFT_ROWS:      # (many rows: cheaper than to work out most of them twice)
        new, h, _ = pre_norm_step(batch, W, gain, parts, eps, x, y, bias, scale, table, freq, embed_gain, None, moved, out_cols, out_dtype)
        return new, token_shift(h, shift.mu[None], shift.last, batch)[0], None
    new = torch.empty((T, W), device=dev, dtype=torch.float32)
    prompts = shift is not None and batch.n_prompts > 0
    after = (Moved(torch.empty((batch.n_prompts, h.shape[1]), device=dev, dtype=h.dtype), shift.last, batch.state_slots[batch.n_decode:])
             if prompts else None)
    if T == 0:
        return new, h, after
    mixed = y if isinstance(y, Mixed) else None
    rows = mixed.rows if mixed is not None else y
    if not h.is_cuda:
        return _pre_norm_torch(batch, W, gain, parts, eps, x, mixed.sum() if mixed is not None else y, bias, scale, table, freq, embed_gain,
                               shift, moved, new, h, after)
    for t in (rows, table):
        if t is not None and t.dtype != h.dtype:
            raise ValueError("pre_norm_step: the inputs and the result share one dtype")
    ints = (ctypes.c_int * 8)(mixed.pos.shape[1] if mixed is not None else 0, table.shape[0] if start else 0, parts, batch.n_decode,
                              moved.slots.shape[0] if moved is not None else 0, h.shape[1], T, W)
    lds = (ctypes.c_longlong * 3)(rows.stride(0) if rows is not None else 0, table.stride(0) if start else 0, h.stride(0))
    ptrs = (ctypes.c_void_p * 24)(
        _ptr(x), new.data_ptr(), _ptr(rows), *((_ptr(mixed.pos), _ptr(mixed.weight)) if mixed is not None else (None, None)), _ptr(bias),
        _ptr(scale), _ptr(batch.tokens) if start else None, _ptr(table), _ptr(freq), _ptr(embed_gain), _ptr(batch.positions), _ptr(gain),
        *((_ptr(shift.mu), _ptr(shift.last)) if shift is not None else (None, None)), after.tail.data_ptr() if after is not None else None,
        _ptr(batch.seq_of), _ptr(batch.state_slots), *((_ptr(batch.cu), _ptr(batch.pos0)) if prompts else (None, None)),
        *((_ptr(moved.tail), _ptr(moved.last), _ptr(moved.slots)) if moved is not None else (None, None, None)), h.data_ptr())
    check(lib().tsb_pre_norm_step(ints, lds, ptrs, float(eps), dtype_code(h.dtype), stream_ptr(dev)), "tsb_pre_norm_step")
    return new, h, after


def _pre_norm_torch(batch, W, gain, parts, eps, x, y, bias, scale, table, freq, embed_gain, shift, moved, new, h, after):
    if moved is not None:
        moved.last[moved.slots.long(), 0] = moved.tail
    if table is not None:
        new.copy_(table[batch.tokens.long(), :W])
        if freq is not None:
            a = (batch.positions[:, None].double() * freq.double().sum(1)[None, :])
            new += torch.stack([torch.sin(a), torch.cos(a)], dim=2).reshape(new.shape[0], -1)[:, :W].float()
        if embed_gain is not None:
            new.copy_(_part_norm(new, embed_gain, parts, eps))
    else:
        new.copy_(x)
    if y is not None:
        z = y[:, :W].float()
        z = z + bias if bias is not None else z
        new += z * scale if scale is not None else z
    n = _part_norm(new, gain, parts, eps)
    if shift is not None:
        out = n.clone()
        for i, (row0, rows, slot, pos0) in enumerate(batch.spans()):
            z = n[row0:row0 + rows]
            kept = torch.nn.functional.pad(z, (0, h.shape[1] - W)).to(h.dtype)
            first = shift.last[slot] if pos0 > 0 and slot >= 0 else torch.zeros(1, h.shape[1])
            out[row0:row0 + rows] = z + (torch.cat([first, kept[:-1]])[:, :W].float() - z) * shift.mu[:W]
            if i >= batch.n_decode:
                after.tail[i - batch.n_decode] = kept[-1]
            elif slot >= 0:
                shift.last[slot] = kept[-1]
        n = out
    h[:, W:] = 0
    h[:, :W] = n
    return new, h, after
