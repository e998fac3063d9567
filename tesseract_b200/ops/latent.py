"""Latent attention over ragged batches (``csrc/latent_attn.cu``): keys and values of all heads are products of one normed
vector c per token, plus one rotated key part that all heads share; the pool keeps only these two.

``latent_attention`` takes a packed projection [q: nope, rot per head | c, rot | gate per head] and attends

* decoded rows (and every row of an fp32 model, or of head sizes that the next form does not take) in the latent space:
  W_uk^T q against the pool rows, W_uv on the read-out. One pool row serves all heads as key and value;
* prompt rows in written-out form: keys and values of the portion and of what earlier portions left are products of the
  gathered pool rows with one matrix (which also copies the rotated part into every head), attended by the tcgen05 kernel
  (``csrc/flash_attn_fwd.cu``).

Heads come out times sigmoid(gate).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from .. import _native
from .._native import check, dtype_code, lib, stream_ptr
from .gemm import project
from .rotary import Rotary, rotate_stored

P, I, L, F = _native.P, _native.I, _native.L, _native.F
_native.register_signatures({
    "tsb_latent_append": [P, P, L, F, P, F] + [P] * 8 + [I, P],
    "tsb_latent_gather": [P, P, P, P, I, I, P],
    "tsb_head_linear": [P, L, I, P, L, I, P, L, I, P, L, F, I, I, I, I, I, P],
    "tsb_gate_heads": [P, I, P, L, F, P, L, I, I, I, I, P],
    "tsb_latent_attn": [P, P, P, I, P, P, P, P, P, P, I, I, I, I, I, I, I, F, I, P],
})

MAX_ROW = 1024


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class LatentGeometry:
    heads: int
    dim: int             # unrotated query / key coordinates of a head
    rot_dim: int         # rotated ones
    vdim: int
    kv_rank: int
    rotary: Rotary

    def __post_init__(self):
        if min(self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank) < 1 or self.rotary.dims != self.rot_dim:
            raise ValueError("latent attention: positive sizes, and rot_dim rotated dims")
        if self.row > MAX_ROW:
            raise ValueError(f"latent attention: a cached row takes at most {MAX_ROW} columns")

    # padded sections of a head and of a cached row
    @property
    def np(self) -> int:
        return _up(self.dim, 8)

    @property
    def q_cols(self) -> int:
        return self.np + 2 * self.rotary.hp

    @property
    def vp(self) -> int:
        return _up(self.vdim, 8)

    @property
    def cp(self) -> int:
        return _up(self.kv_rank, 64)

    @property
    def rp(self) -> int:
        return _up(2 * self.rotary.hp, 32)

    @property
    def row(self) -> int:
        return self.cp + self.rp

    # packed projection
    @property
    def off_c(self) -> int:
        return self.heads * self.q_cols

    @property
    def off_gate(self) -> int:
        return self.off_c + _up(self.kv_rank, 8) + 2 * self.rotary.hp

    @property
    def cols(self) -> int:
        return self.off_gate + self.heads * self.vp

    @property
    def out_cols(self) -> int:
        return _up(self.heads * self.vp, 16)

    @property
    def D(self) -> int:
        """Common size of query, key and value heads in written-out form."""
        d = max(self.q_cols, self.vp, _up(self.np, 16))
        return 64 if d <= 64 else 128 if d <= 128 else _up(d, 16)

    def written_out(self, dtype) -> bool:
        return dtype == torch.bfloat16 and self.D <= 128

    def tensor_cores(self, dtype, block: int) -> bool:
        """Whether single rows run on ``latent_decode_kernel`` (its sums, scores and queries fit in tensor memory)."""
        return dtype == torch.bfloat16 and self.cp <= 512 and self.row <= 640 and block % 8 == 0


@dataclass
class LatentWeights:
    """norm fp32 [cp]; w_up [2 heads D, row]: for every head D rows that turn a pool row into its key (unrotated rows, then
    ones that copy the rotated part), then for every head D rows that turn it into its value; w_absorb [heads, cp, k]
    (W_uk of a head transposed, k = its unrotated coordinates rounded up to 16)."""
    norm: torch.Tensor
    w_up: torch.Tensor
    w_absorb: torch.Tensor
    eps: float
    scale: float


def _splits(rows: int, geo: LatentGeometry, max_len: int) -> int:
    """Key splits of the decode kernel (one CTA per SM): fewest waves times the tiles of a split, plus what a CTA spends before
    and after its tiles."""
    ctas, tiles = rows * ((geo.heads + 31) // 32), (max_len + 63) // 64
    most = max(1, min((tiles + 1) // 2, 64, 4 * 148 // ctas + 4))
    return min(range(1, most + 1), key=lambda s: -(-ctas * s // 148) * (-(-tiles // s) + 2))


def latent_attention(proj: torch.Tensor, geo: LatentGeometry, w: LatentWeights, pool: torch.Tensor, table: torch.Tensor, batch,
                     in_scale: float = 1.0, out: torch.Tensor | None = None) -> torch.Tensor:
    """proj [T, geo.cols] -> [T, geo.out_cols] (``out`` may be columns of a wider matrix); pool [blocks, block, geo.row]."""
    T, H, dev = proj.shape[0], geo.heads, proj.device
    if out is None:
        out = torch.empty((T, geo.out_cols), device=dev, dtype=proj.dtype)
    if T == 0:
        return out
    if geo.out_cols > H * geo.vp:
        out[:, H * geo.vp:] = 0
    if not proj.is_cuda:
        return _latent_torch(proj, geo, w, pool, table, batch, in_scale, out)
    dt, st = dtype_code(proj.dtype), stream_ptr(dev)
    nb, bs, row = pool.shape
    D, new = geo.D, dict(device=dev, dtype=proj.dtype)
    written = geo.written_out(proj.dtype)
    nl = batch.n_decode if written else T              # rows attended in the latent space come first
    n = T - nl
    seg = batch.segments(0) if n else None
    q = torch.empty((T, H, D), **new)
    q_cat = torch.empty((nl, H, row), **new) if nl else None
    stage = torch.empty((seg.keys, row), **new) if n else None
    ptr = lambda t: t.data_ptr() if t is not None else None   # noqa: E731
    v = (H, geo.np, geo.rotary.hp, D, geo.off_c, geo.kv_rank, geo.cp, geo.rp, nl, nl, T)
    check(lib().tsb_latent_append((ctypes.c_int * len(v))(*v), proj.data_ptr(), proj.stride(0), float(in_scale), w.norm.data_ptr(),
                                  float(w.eps), table.data_ptr(), batch.positions.data_ptr(), batch.slots.data_ptr(), q.data_ptr(),
                                  ptr(q_cat), pool.data_ptr(), ptr(stage), seg.stage_rows.data_ptr() if n else None, dt, st),
          "tsb_latent_append")
    gate = proj[:, geo.off_gate:]
    if nl:
        k = w.w_absorb.shape[2]
        check(lib().tsb_head_linear(q.data_ptr(), H * D, D, w.w_absorb.data_ptr(), geo.cp * k, k, q_cat.data_ptr(), H * row, row, None, 0,
                                    0.0, nl, H, geo.cp, k, dt, st), "tsb_head_linear")
        lat = torch.empty((nl, H, geo.cp), **new)
        tables = batch.tables
        single = nl == batch.n_decode                   # row i is sequence i, lengths are at hand
        fast = geo.tensor_cores(proj.dtype, bs)
        splits = _splits(nl, geo, batch.max_len) if fast else 0
        part_o = torch.empty((nl, H, splits, geo.cp), device=dev, dtype=torch.float32) if splits > 1 else None
        part_ml = torch.empty((nl, H, splits, 2), device=dev, dtype=torch.float32) if splits > 1 else None
        check(lib().tsb_latent_attn(q_cat.data_ptr(), pool.data_ptr(), tables.data_ptr(), tables.stride(0),
                                    None if single else batch.seq_of.data_ptr(), batch.lens.data_ptr() if single else None,
                                    batch.positions.data_ptr(), lat.data_ptr(), ptr(part_o), ptr(part_ml), nl, H, geo.cp, geo.rp, bs, nb,
                                    splits, float(w.scale), dt, st), "tsb_latent_attn")
        wv = w.w_up[H * D:]                              # a head's value rows; their last rp columns are zero and not read
        check(lib().tsb_head_linear(lat.data_ptr(), H * geo.cp, geo.cp, wv.data_ptr(), D * row, row, out.data_ptr(), out.stride(0),
                                    geo.vp, gate.data_ptr(), gate.stride(0), float(in_scale), nl, H, geo.vp, geo.cp, dt, st),
              "tsb_head_linear")
        _native.add_launches(1 if splits > 1 else 0)
    if n:
        if seg.n_gather:
            check(lib().tsb_latent_gather(pool.data_ptr(), stage.data_ptr(), seg.gather_dst.data_ptr(), seg.gather_src.data_ptr(),
                                          seg.n_gather, row, st), "tsb_latent_gather")
        kv = project(stage, w.w_up).view(seg.keys, 2 * H, D)
        o = torch.empty((n, H, D), **new)
        qp, vp = q[nl:], kv[:, H:]
        check(lib().tsb_flash_fwd_varlen_keys(qp.data_ptr(), kv.data_ptr(), vp.data_ptr(), o.data_ptr(), seg.cu_q.data_ptr(),
                                              seg.cu_k.data_ptr(), seg.n, seg.max_q, n, seg.keys, H, H, D, H * D, D, 2 * H * D, D,
                                              2 * H * D, D, H * D, D, float(w.scale), st), "tsb_flash_fwd_varlen_keys")
        go, oo = gate[nl:], out[nl:]
        check(lib().tsb_gate_heads(o.data_ptr(), D, go.data_ptr(), go.stride(0), float(in_scale), oo.data_ptr(), oo.stride(0), n, H,
                                   geo.vp, dt, st), "tsb_gate_heads")
    return out


def _latent_torch(proj, geo, w, pool, table, batch, in_scale, out):
    """Written-out form in fp32 from the pool rows."""
    H, D, np_, hp = geo.heads, geo.D, geo.np, geo.rotary.hp
    bs, rank = pool.shape[1], geo.kv_rank
    flat = pool.view(-1, geo.row)
    up = w.w_up.float()
    for i, (row0, n, slot, pos0) in enumerate(batch.spans()):
        if slot < 0:
            out[row0:row0 + n] = 0
            continue
        p = proj[row0:row0 + n].float() * in_scale
        pos = torch.arange(pos0, pos0 + n)
        c = p[:, geo.off_c:geo.off_c + rank]
        at = geo.off_c + (rank + 7) // 8 * 8
        sl = batch.slots[row0:row0 + n].long()
        flat[sl, :rank] = (c / torch.sqrt((c * c).mean(-1, keepdim=True) + w.eps) * w.norm[:rank]).to(pool.dtype)
        flat[sl, geo.cp:geo.cp + 2 * hp] = rotate_stored(p[:, at:at + 2 * hp], table, pos).to(pool.dtype)
        total = pos0 + n
        seen = torch.arange(total)
        rows = flat[batch.tables[i][seen // bs].long() * bs + seen % bs].float()
        kv = (rows @ up.t()).view(total, 2 * H, D)
        q = torch.zeros(n, H, D)
        head = p[:, :geo.off_c].view(n, H, geo.q_cols)
        q[..., :np_] = head[..., :np_]
        q[..., np_:geo.q_cols] = rotate_stored(head[..., np_:], table, pos)
        q = q.to(proj.dtype).float()
        s = torch.einsum("thd,shd->hts", q, kv[:, :H]) * w.scale
        s = s.masked_fill(seen[None, :] > pos[:, None], float("-inf"))
        o = torch.einsum("hts,shd->thd", torch.softmax(s, dim=-1), kv[:, H:])[..., :geo.vp]
        gate = p[:, geo.off_gate:geo.cols].view(n, H, geo.vp)
        out[row0:row0 + n, :H * geo.vp] = (o * torch.sigmoid(gate)).reshape(n, -1).to(out.dtype)
    return out
