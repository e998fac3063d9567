// Latent attention for ragged batches: keys and values of all heads are products of one normed vector c per token (the
// latent), plus one rotated key part that all heads share; only these two are cached, as one row [c: cp | rotated: rp] of a
// paged pool [blocks, block, cp + rp] (padding columns are zero).
//
// A packed projection row holds [q of every head: nope | rot] [c | rot] [gate of every head]; "rot" is stored as
// [u: hp | v: hp], the pairs that turn together hp columns apart.
//
//   latent_append_kernel  scales the row, norms c, rotates, stores the pool row (and, for prompt rows that are attended in
//                         written-out form, the row of the key axis), and writes q: `q_out` [rows, H, D] = [nope | rot | 0]
//                         and, for rows attended in the latent space, the rotated part of `q_cat` [rows, H, cp + rp].
//   head_linear_kernel    one small product per head: W_uk^T q into q_cat's first cp columns before the attention in the
//                         latent space, W_uv o after it, times the output gate.
//   latent_decode_kernel  attention of single rows in the latent space on the tensor cores (bf16), split over keys; the pool
//                         row serves as key and, its first cp columns, as value, so it is read once for all heads.
//   latent_merge_kernel   merges the splits.
//   latent_rows_kernel    the same attention with one warp per (row, head) in fp32: fp32 models and sizes the other does not take.
//   latent_gather_kernel  pool rows of earlier portions -> key axis.
//   gate_heads_kernel     o * sigmoid(gate) for the written-out form.
#include "head_tile.cuh"

#include <algorithm>

namespace tsb {
namespace {

struct LatentAppendParams {
  const void* proj;          // [rows, ldp]
  long long ldp;
  int H, np, hp, D;          // query head in the projection: np + 2 hp columns; in q_out: D
  int off_c, rank, cp, rp;   // c section: rank columns (padded to 8), then the rotated part
  float in_scale;
  const float* norm;         // [cp], zero past rank
  float eps;
  const float2* table;       // [positions, hp] cos, sin
  const int* positions;      // [rows]
  const int* slots;          // [rows] pool row, -1: none
  void* q_out;               // [rows, H, D]
  void* q_cat;               // [cat_rows, H, cp + rp] or null
  int cat_rows;
  void* pool;
  void* stage;               // [keys, cp + rp] or null
  const int* stage_rows;     // [rows - stage_from]
  int stage_from, rows;
};

template <typename T>
__global__ void __launch_bounds__(256)
latent_append_kernel(LatentAppendParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>;
  __shared__ float red[8];
  const int row = blockIdx.x, tid = threadIdx.x, L = p.cp + p.rp;
  const T* x = static_cast<const T*>(p.proj) + row * p.ldp;
  const int pos = max(p.positions[row], 0);
  const float2* table = p.table + static_cast<long long>(pos) * p.hp;
  const float s = p.in_scale;
  // the latent's sum of squares
  float ss = 0.f;
  for (int i = tid * V; i < p.rank; i += 256 * V) {
    float f[V];
    ld16<T>(x + p.off_c + i, f);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(f[e] * s, f[e] * s, ss);         // (columns past rank are zero)
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  // queries
  const int qs = p.np + 2 * p.hp, vph = p.D / V;
  const bool cat = row < p.cat_rows;
  for (int i = tid; i < p.H * vph; i += 256) {
    const int h = i / vph, d = (i % vph) * V;
    const T* head = x + h * qs;
    float f[V] = {};
    if (d < p.np) ld16<T>(head + d, f);
    else if (d < qs) rotated_piece<T>(head + p.np, d - p.np, p.hp, table, f);
#pragma unroll
    for (int e = 0; e < V; ++e) f[e] *= s;
    st16<T>(static_cast<T*>(p.q_out) + (static_cast<long long>(row) * p.H + h) * p.D + d, f);
  }
  if (cat) {
    const int vpr = p.rp / V;
    for (int i = tid; i < p.H * vpr; i += 256) {
      const int h = i / vpr, d = (i % vpr) * V;
      float f[V] = {};
      if (d < 2 * p.hp) rotated_piece<T>(x + h * qs + p.np, d, p.hp, table, f);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] *= s;
      st16<T>(static_cast<T*>(p.q_cat) + (static_cast<long long>(row) * p.H + h) * L + p.cp + d, f);
    }
  }
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) ss += red[w];
  const float r = s / sqrtf(ss / static_cast<float>(p.rank) + p.eps);
  const int slot = p.slots[row];
  T* pool = slot >= 0 ? static_cast<T*>(p.pool) + static_cast<long long>(slot) * L : nullptr;
  T* stage = p.stage && row >= p.stage_from ? static_cast<T*>(p.stage) + static_cast<long long>(p.stage_rows[row - p.stage_from]) * L : nullptr;
  const int rank8 = (p.rank + 7) / 8 * 8;
  for (int d = tid * V; d < L; d += 256 * V) {
    float f[V] = {};
    if (d < p.cp) {
      if (d < rank8) {
        ld16<T>(x + p.off_c + d, f);
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] *= r * p.norm[d + e];
      }
    } else if (d - p.cp < 2 * p.hp) {
      rotated_piece<T>(x + p.off_c + rank8, d - p.cp, p.hp, table, f);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] *= s;
    }
    if (pool) st16<T>(pool + d, f);
    if (stage) st16<T>(stage + d, f);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
latent_gather_kernel(const T* pool, T* stage, const int* dst_rows, const int* src_slots, int n, int L) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>;
  const int vpr = L / V;
  const unsigned idx = blockIdx.x * 256u + threadIdx.x;
  const int i = static_cast<int>(idx / vpr), d = static_cast<int>(idx % vpr) * V;
  if (i >= n) return;
  *reinterpret_cast<uint4*>(stage + static_cast<long long>(dst_rows[i]) * L + d) =
      *reinterpret_cast<const uint4*>(pool + static_cast<long long>(src_slots[i]) * L + d);
}

// ------------------------------------------------------------------ one product per head
struct HeadLinearParams {
  const void* x;             // [rows, ldx], head h at h * xh
  long long ldx;
  int xh;
  const void* w;             // head h at h * wh, rows ldw apart
  long long wh;
  int ldw;
  void* out;                 // [rows, ldo], head h at h * oh
  long long ldo;
  int oh;
  const void* gate;          // [rows, ldg], head h at h * oh: out *= sigmoid(gate_scale * gate); or null
  long long ldg;
  float gate_scale;
  int rows, N, K;
};

template <typename T, int BM>
__global__ void __launch_bounds__(128)
head_linear_kernel(HeadLinearParams p) {
  using Tile = HeadTile<T, BM, 1>;
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  const int n0 = blockIdx.x * 64, h = blockIdx.y, m0 = blockIdx.z * BM;
  const int rows = min(BM, p.rows - m0), cols = min(64, p.N - n0);
  const T* const w[1] = {static_cast<const T*>(p.w) + h * p.wh + static_cast<long long>(n0) * p.ldw};
  const float* acc = Tile::run(smem, static_cast<const T*>(p.x) + m0 * p.ldx + h * p.xh, p.ldx, rows, w, p.ldw, cols, p.K);
  for (int i = threadIdx.x; i < rows * 32; i += 128) {
    const int m = i >> 5, n = (i & 31) * 2;
    if (n >= cols) continue;                       // (N is even)
    const long long row = m0 + m;
    float a = acc[m * Tile::kLdC + n], b = acc[m * Tile::kLdC + n + 1];
    if (p.gate) {
      const T* g = static_cast<const T*>(p.gate) + row * p.ldg + h * p.oh + n0 + n;
      a *= sigmoid_f32(p.gate_scale * to_f32<T>(g[0]));
      b *= sigmoid_f32(p.gate_scale * to_f32<T>(g[1]));
    }
    T* o = static_cast<T*>(p.out) + row * p.ldo + h * p.oh + n0 + n;
    if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(o) = pack_bf16x2(a, b);
    else *reinterpret_cast<float2*>(o) = make_float2(a, b);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
gate_heads_kernel(const T* o, int D, const T* gate, long long ldg, float scale, T* out, long long ldo, int rows, int H, int vp) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>;
  const unsigned vpr = H * vp / V, idx = blockIdx.x * 256u + threadIdx.x;
  const int row = static_cast<int>(idx / vpr), c = static_cast<int>(idx % vpr) * V;
  if (row >= rows) return;
  const int h = c / vp, d = c % vp;
  float f[V], g[V];
  ld16<T>(o + (static_cast<long long>(row) * H + h) * D + d, f);
  ld16<T>(gate + row * ldg + c, g);
#pragma unroll
  for (int i = 0; i < V; ++i) f[i] *= sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-scale * g[i])) : sigmoid_f32(scale * g[i]);
  st16<T>(out + row * ldo + c, f);
}

// ------------------------------------------------------------------ attention in the latent space
struct LatentAttnParams {
  const void* q;             // [rows, H, L]
  const void* pool;          // [blocks, bs, L]
  const int* tables;         // [sequences, table_ld]
  const int* seq_of;         // [rows] or null: row i is sequence i
  const int* lens;           // [rows] keys of a row, or
  const int* pos;            // [rows] keys - 1
  void* out;                 // [rows, H, cp]
  float* part_o;             // [rows, H, splits, cp]
  float* part_ml;            // [rows, H, splits, 2]
  int rows, H, cp, rp, bs, nb, table_ld, splits;
  float scale;
  int* status;
};

constexpr int kKeys = 64;          // keys of a tile

// One CTA per (key split, 16 heads, row), eight warps. Per tile: warp w scores keys 8 w .. 8 w + 7 for the 16 heads; the
// weights go through shared memory; then every warp adds the tile to its own cp / 8 columns of the read-out.
template <int CT>
__global__ void __launch_bounds__(256)
latent_decode_kernel(LatentAttnParams p) {
  using T = __nv_bfloat16;
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int kLdP = kKeys + 8;
  const int L = p.cp + p.rp, ld = L + 8;
  T* sq = reinterpret_cast<T*>(smem);                 // [16][ld]
  T* sk = sq + 16 * ld;                               // [2][kKeys][ld]
  T* sp = sk + 2 * kKeys * ld;                        // [16][kLdP]
  float* smax = reinterpret_cast<float*>(sp + 16 * kLdP);      // [8][16]
  float* ssum = smax + 8 * 16;                        // [8][16]
  const int split = blockIdx.x, h0 = blockIdx.y * 16, row = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int len = p.lens ? p.lens[row] : p.pos[row] + 1;
  const int share = ((len + p.splits - 1) / p.splits + kKeys - 1) / kKeys * kKeys;
  const int t_begin = split * share, t_end = min(len, t_begin + share);
  const int n_tiles = t_end > t_begin ? (t_end - t_begin + kKeys - 1) / kKeys : 0;
  const int* table = p.tables + static_cast<long long>(p.seq_of ? p.seq_of[row] : row) * p.table_ld;
  const int pieces = L / 8;

  auto issue = [&](int j) {
    T* dst = sk + (j & 1) * kKeys * ld;
    for (int i = 0; i < 8; ++i) {
      const int r = warp * 8 + i, t = t_begin + j * kKeys + r;
      const bool ok = t < t_end;
      int blk = ok ? table[t / p.bs] : 0;
      if (blk < 0 || blk >= p.nb) {        // never read outside the pool: block 0 instead, and the host hears of it
        if (lane == 0 && p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
        blk = 0;
      }
      const T* src = static_cast<const T*>(p.pool) + (static_cast<long long>(blk) * p.bs + (ok ? t % p.bs : 0)) * L;
      for (int v = lane; v < pieces; v += 32) cp_async_16(smem_u32(dst + r * ld + v * 8), src + v * 8, ok ? 16 : 0);
    }
  };
  for (int i = tid; i < 16 * pieces; i += 256) {
    const int h = i / pieces, v = i % pieces;
    const bool ok = h0 + h < p.H;
    cp_async_16(smem_u32(sq + h * ld + v * 8),
                static_cast<const T*>(p.q) + (static_cast<long long>(row) * p.H + (ok ? h0 + h : 0)) * L + v * 8, ok ? 16 : 0);
  }
  if (n_tiles > 0) issue(0);
  cp_commit();

  float o[CT][4];
#pragma unroll
  for (int i = 0; i < CT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_part[2] = {0.f, 0.f};      // rows g and g + 8
  const float scale_log2 = p.scale * 1.4426950408889634f;
  const uint32_t q_addr = smem_u32(sq), p_addr = smem_u32(sp);
  for (int j = 0; j < n_tiles; ++j) {
    if (j + 1 < n_tiles) issue(j + 1);
    cp_commit();
    cp_wait<1>();
    __syncthreads();
    const uint32_t k_addr = smem_u32(sk + (j & 1) * kKeys * ld);
    // scores: four independent sums over interleaved slices of the row
    float s[4][4];
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e][0] = s[e][1] = s[e][2] = s[e][3] = 0.f;
    for (int k0 = 0; k0 < L; k0 += 64) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int k = k0 + half * 32;
        if (k >= L) break;
        uint32_t b[4], a0[4], a1[4];
        ldmat_x4(b, k_addr + static_cast<uint32_t>((warp * 8 + (lane & 7)) * ld + k + (lane >> 3) * 8) * 2);
        ldmat_x4(a0, q_addr + frag_a(lane, 0, k, ld));
        ldmat_x4(a1, q_addr + frag_a(lane, 0, k + 16, ld));
        mma_bf16(s[2 * half], a0, b[0], b[1]);
        mma_bf16(s[2 * half + 1], a1, b[2], b[3]);
      }
    }
    const int key = t_begin + j * kKeys + warp * 8 + 2 * t4;
    float sc[4];
#pragma unroll
    for (int e = 0; e < 4; ++e)
      sc[e] = key + (e & 1) < t_end ? (s[0][e] + s[1][e] + s[2][e] + s[3][e]) * scale_log2 : -INFINITY;
    float mx[2] = {fmaxf(sc[0], sc[1]), fmaxf(sc[2], sc[3])};
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
      mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
    }
    if (t4 == 0) {
      smax[warp * 16 + g] = mx[0];
      smax[warp * 16 + g + 8] = mx[1];
    }
    __syncthreads();
    float corr[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      float mn = m_run[i];
#pragma unroll
      for (int w = 0; w < 8; ++w) mn = fmaxf(mn, smax[w * 16 + g + 8 * i]);     // (every tile has a key in it: finite)
      corr[i] = m_run[i] == -INFINITY ? 0.f : exp2f(m_run[i] - mn);
      m_run[i] = mn;
      const float p0 = exp2f(sc[2 * i] - mn), p1 = exp2f(sc[2 * i + 1] - mn);
      l_part[i] = l_part[i] * corr[i] + p0 + p1;
      *reinterpret_cast<uint32_t*>(sp + (g + 8 * i) * kLdP + warp * 8 + 2 * t4) = pack_bf16x2(p0, p1);
    }
    __syncthreads();
    uint32_t pa[4][4];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) ldmat_x4(pa[kk], p_addr + frag_a(lane, 0, kk * 16, kLdP));
#pragma unroll
    for (int i = 0; i < CT; ++i) {
      const int col = (warp * CT + i) * 8;
      o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1];
#pragma unroll
      for (int kk = 0; kk < 2; ++kk) {               // 32 keys x 8 columns per load
        uint32_t b[4];
        ldmat_x4_trans(b, k_addr + static_cast<uint32_t>((kk * 32 + lane) * ld + col) * 2);
        mma_bf16(o[i], pa[2 * kk], b[0], b[1]);
        mma_bf16(o[i], pa[2 * kk + 1], b[2], b[3]);
      }
    }
    __syncthreads();
  }
  cp_wait<0>();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l_part[i] += __shfl_xor_sync(0xffffffffu, l_part[i], 1);
    l_part[i] += __shfl_xor_sync(0xffffffffu, l_part[i], 2);
    if (t4 == 0) ssum[warp * 16 + g + 8 * i] = l_part[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int h = h0 + g + 8 * i;
    if (h >= p.H) continue;
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) l += ssum[w * 16 + g + 8 * i];
    const long long at = static_cast<long long>(row) * p.H + h;
    if (p.splits == 1) {
      const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
      for (int c = 0; c < CT; ++c)
        *reinterpret_cast<uint32_t*>(static_cast<T*>(p.out) + at * p.cp + (warp * CT + c) * 8 + 2 * t4) =
            pack_bf16x2(o[c][2 * i] * inv, o[c][2 * i + 1] * inv);
    } else {
      const long long pi = at * p.splits + split;
#pragma unroll
      for (int c = 0; c < CT; ++c)
        *reinterpret_cast<float2*>(p.part_o + pi * p.cp + (warp * CT + c) * 8 + 2 * t4) = make_float2(o[c][2 * i], o[c][2 * i + 1]);
      if (warp == 0 && t4 == 0) {
        p.part_ml[pi * 2] = m_run[i];
        p.part_ml[pi * 2 + 1] = l;
      }
    }
  }
}

__global__ void __launch_bounds__(128)
latent_merge_kernel(LatentAttnParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const long long at = blockIdx.x;
  const float* ml = p.part_ml + at * p.splits * 2;
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < p.splits; ++s) m = fmaxf(m, ml[2 * s]);
  for (int s = 0; s < p.splits; ++s) l += ml[2 * s] == -INFINITY ? 0.f : exp2f(ml[2 * s] - m) * ml[2 * s + 1];
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int c = threadIdx.x * 2; c < p.cp; c += 256) {
    float a = 0.f, b = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      if (ml[2 * s] == -INFINITY) continue;
      const float w = exp2f(ml[2 * s] - m) * inv;
      const float2 v = *reinterpret_cast<const float2*>(p.part_o + (at * p.splits + s) * p.cp + c);
      a = fmaf(w, v.x, a);
      b = fmaf(w, v.y, b);
    }
    *reinterpret_cast<uint32_t*>(static_cast<__nv_bfloat16*>(p.out) + at * p.cp + c) = pack_bf16x2(a, b);
  }
}

// QN columns of a pool row per lane, the first CN of them columns of c (lane + 32 i). Keys four at a time.
template <typename T, int QN>
__global__ void __launch_bounds__(128)
latent_rows_kernel(LatentAttnParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const long long w = blockIdx.x * 4ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, L = p.cp + p.rp;
  if (w >= static_cast<long long>(p.rows) * p.H) return;
  const int row = static_cast<int>(w / p.H), h = static_cast<int>(w % p.H);
  const int* table = p.tables + static_cast<long long>(p.seq_of ? p.seq_of[row] : row) * p.table_ld;
  const T* qr = static_cast<const T*>(p.q) + (static_cast<long long>(row) * p.H + h) * L;
  float q[QN], o[QN];
#pragma unroll
  for (int i = 0; i < QN; ++i) {
    q[i] = lane + 32 * i < L ? to_f32<T>(qr[lane + 32 * i]) : 0.f;
    o[i] = 0.f;
  }
  const int len = p.lens ? p.lens[row] : p.pos[row] + 1;
  float m = -INFINITY, l = 0.f;
  constexpr int kAt = QN <= 12 ? 4 : 2;
  for (int t = 0; t < len; t += kAt) {
    float s[kAt], k[kAt][QN];
#pragma unroll
    for (int j = 0; j < kAt; ++j) {
      const int tt = min(t + j, len - 1);
      int blk = table[tt / p.bs];
      if (blk < 0 || blk >= p.nb) {
        if (p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
        blk = 0;
      }
      const T* kr = static_cast<const T*>(p.pool) + (static_cast<long long>(blk) * p.bs + tt % p.bs) * L;
      s[j] = 0.f;
#pragma unroll
      for (int i = 0; i < QN; ++i) {
        k[j][i] = lane + 32 * i < L ? to_f32<T>(kr[lane + 32 * i]) : 0.f;
        s[j] = fmaf(q[i], k[j][i], s[j]);
      }
    }
    float mn = m;
#pragma unroll
    for (int j = 0; j < kAt; ++j) {
      s[j] = t + j < len ? warp_sum(s[j]) * p.scale : -INFINITY;
      mn = fmaxf(mn, s[j]);
    }
    const float corr = m == -INFINITY ? 0.f : expf(m - mn);
    l *= corr;
#pragma unroll
    for (int i = 0; i < QN; ++i) o[i] *= corr;
#pragma unroll
    for (int j = 0; j < kAt; ++j) {
      const float e = s[j] == -INFINITY ? 0.f : expf(s[j] - mn);
      l += e;
#pragma unroll
      for (int i = 0; i < QN; ++i) o[i] = fmaf(e, k[j][i], o[i]);
    }
    m = mn;
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  T* out = static_cast<T*>(p.out) + (static_cast<long long>(row) * p.H + h) * p.cp;
#pragma unroll
  for (int i = 0; i < QN; ++i)
    if (lane + 32 * i < p.cp) out[lane + 32 * i] = from_f32<T>(o[i] * inv);
}

template <int CT>
int launch_latent_decode(const LatentAttnParams& p, cudaStream_t s) {
  const int ld = p.cp + p.rp + 8;
  const int smem = (16 * ld + 2 * kKeys * ld + 16 * (kKeys + 8)) * 2 + 2 * 8 * 16 * 4;
  if (smem > 227 * 1024) return -2;
  auto kern = latent_decode_kernel<CT>;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  launch_pdl(kern, dim3(p.splits, (p.H + 15) / 16, p.rows), dim3(256), smem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int launch_latent_rows(const LatentAttnParams& p, cudaStream_t s) {
  const unsigned blocks = static_cast<unsigned>((static_cast<long long>(p.rows) * p.H + 3) / 4);
  const bool pdl = pdl_all_enabled();
  const int n = (p.cp + p.rp + 31) / 32;
#define TSB_LR(N) launch_pdl(latent_rows_kernel<T, N>, dim3(blocks), dim3(128), 0, s, pdl, p)
  if (n <= 2) TSB_LR(2);
  else if (n <= 4) TSB_LR(4);
  else if (n <= 8) TSB_LR(8);
  else if (n <= 12) TSB_LR(12);
  else if (n <= 18) TSB_LR(18);
  else if (n <= 32) TSB_LR(32);
  else return -2;
#undef TSB_LR
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int BM>
int launch_head_linear(const HeadLinearParams& p, int H, cudaStream_t s) {
  using Tile = HeadTile<T, BM, 1>;
  auto kern = head_linear_kernel<T, BM>;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Tile::kSmem);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  launch_pdl(kern, dim3((p.N + 63) / 64, H, (p.rows + BM - 1) / BM), dim3(128), Tile::kSmem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace
}  // namespace tsb

// ints: H, np, hp, D, off_c, rank, cp, rp, cat_rows, stage_from, rows. D, cp and rp are multiples of 8, np and hp too. See
// LatentAppendParams.
TSB_EXPORT int tsb_latent_append(const int* ints, const void* proj, long long ldp, float in_scale, const float* norm, float eps,
                                 const float* table, const int* positions, const int* slots, void* q_out, void* q_cat, void* pool,
                                 void* stage, const int* stage_rows, int dtype, void* stream) {
  using namespace tsb;
  LatentAppendParams p{};
  p.proj = proj; p.ldp = ldp; p.in_scale = in_scale; p.norm = norm; p.eps = eps;
  p.table = reinterpret_cast<const float2*>(table); p.positions = positions; p.slots = slots; p.q_out = q_out; p.q_cat = q_cat;
  p.pool = pool; p.stage = stage; p.stage_rows = stage_rows;
  p.H = ints[0]; p.np = ints[1]; p.hp = ints[2]; p.D = ints[3]; p.off_c = ints[4]; p.rank = ints[5]; p.cp = ints[6]; p.rp = ints[7];
  p.cat_rows = q_cat ? ints[8] : 0; p.stage_from = ints[9]; p.rows = ints[10];
  if (p.rows <= 0 || p.H <= 0 || p.np % 8 || p.hp % 8 || p.D % 8 || p.D < p.np + 2 * p.hp || p.off_c % 8 || p.rank <= 0 ||
      p.cp < p.rank || p.cp % 8 || p.rp % 8 || p.rp < 2 * p.hp || ldp % 8 || (stage && !stage_rows))
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) launch_pdl(latent_append_kernel<__nv_bfloat16>, dim3(p.rows), dim3(256), 0, s, pdl_all_enabled(), p);
  else if (dtype == 0) launch_pdl(latent_append_kernel<float>, dim3(p.rows), dim3(256), 0, s, pdl_all_enabled(), p);
  else return -2;
  return static_cast<int>(cudaGetLastError());
}

// stage[dst_rows[i]] = pool row src_slots[i], i < n (bf16, L columns).
TSB_EXPORT int tsb_latent_gather(const void* pool, void* stage, const int* dst_rows, const int* src_slots, int n, int L, void* stream) {
  using namespace tsb;
  const long long vecs = static_cast<long long>(n) * L / 8;
  if (n <= 0 || L <= 0 || L % 8 || vecs > 0x7fffffffLL) return -2;
  launch_pdl(latent_gather_kernel<__nv_bfloat16>, dim3(static_cast<unsigned>((vecs + 255) / 256)), dim3(256), 0,
             static_cast<cudaStream_t>(stream), pdl_all_enabled(), static_cast<const __nv_bfloat16*>(pool),
             static_cast<__nv_bfloat16*>(stage), dst_rows, src_slots, n, L);
  return static_cast<int>(cudaGetLastError());
}

// out[row, h * oh + n] = sum_k x[row, h * xh + k] w[h, n, k] (times sigmoid(gate_scale * gate[row, h * oh + n])), n < N (even),
// K a multiple of 16; rows of w are ldw apart, heads wh. bf16 (dtype 1) or fp32 (0).
TSB_EXPORT int tsb_head_linear(const void* x, long long ldx, int xh, const void* w, long long wh, int ldw, void* out, long long ldo, int oh,
                               const void* gate, long long ldg, float gate_scale, int rows, int H, int N, int K, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || H <= 0 || H > 65535 || N <= 0 || N % 2 || K <= 0 || K % 16 || ldx % 8 || xh % 8 || wh % 8 || ldw % 8 || ldw < K || ldo % 2 || oh % 2) return -2;
  HeadLinearParams p{x, ldx, xh, w, wh, ldw, out, ldo, oh, gate, ldg, gate_scale, rows, N, K};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool few = rows <= 32;
  if (!few && (rows + 63) / 64 > 65535) return -2;
  if (dtype == 1) return few ? launch_head_linear<__nv_bfloat16, 16>(p, H, s) : launch_head_linear<__nv_bfloat16, 64>(p, H, s);
  if (dtype == 0) return few ? launch_head_linear<float, 16>(p, H, s) : launch_head_linear<float, 64>(p, H, s);
  return -2;
}

// out[row, c] = o[row, h, d] sigmoid(scale * gate[row, c]) with c = h * vp + d, d < vp; o rows are [H, D]. vp % 8 == 0.
TSB_EXPORT int tsb_gate_heads(const void* o, int D, const void* gate, long long ldg, float scale, void* out, long long ldo, int rows,
                              int H, int vp, int dtype, void* stream) {
  using namespace tsb;
  const long long vecs = static_cast<long long>(rows) * H * vp / (dtype == 1 ? 8 : 4);
  if (rows <= 0 || H <= 0 || vp <= 0 || vp % 8 || D % 8 || D < vp || ldg % 8 || ldo % 8 || vecs > 0x7fffff00LL) return -2;
  const dim3 grid(static_cast<unsigned>((vecs + 255) / 256));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1)
    launch_pdl(gate_heads_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const __nv_bfloat16*>(o), D,
               static_cast<const __nv_bfloat16*>(gate), ldg, scale, static_cast<__nv_bfloat16*>(out), ldo, rows, H, vp);
  else if (dtype == 0)
    launch_pdl(gate_heads_kernel<float>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const float*>(o), D,
               static_cast<const float*>(gate), ldg, scale, static_cast<float*>(out), ldo, rows, H, vp);
  else
    return -2;
  return static_cast<int>(cudaGetLastError());
}

// Attention of single rows in the latent space: q [rows, H, cp + rp], pool [nb, bs, cp + rp] -> out [rows, H, cp]. Row i sees the
// first lens[i] keys (or pos[i] + 1 when lens is null) of sequence seq_of[i] (null: i). splits > 0: tensor cores, bf16, cp a
// multiple of 64 up to 512, rp a multiple of 32; part_o and part_ml are scratch of rows * H * splits * cp and * 2 floats when
// splits > 1. splits = 0: one warp per (row, head), any type, cp + rp <= 1024.
TSB_EXPORT int tsb_latent_attn(const void* q, const void* pool, const int* tables, int table_ld, const int* seq_of, const int* lens,
                               const int* pos, void* out, float* part_o, float* part_ml, int rows, int H, int cp, int rp, int bs, int nb,
                               int splits, float scale, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || H <= 0 || cp <= 0 || rp < 0 || bs <= 0 || nb <= 0 || splits < 0 || (!lens && !pos)) return -2;
  LatentAttnParams p{q, pool, tables, seq_of, lens, pos, out, part_o, part_ml, rows, H, cp, rp, bs, nb, table_ld, splits, scale,
                     device_status_word()};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (splits == 0) {
    if (dtype == 1) return launch_latent_rows<__nv_bfloat16>(p, s);
    return dtype == 0 ? launch_latent_rows<float>(p, s) : -2;
  }
  if (dtype != 1 || cp % 64 || cp > 512 || rp % 32 || rows > 65535 || (splits > 1 && (!part_o || !part_ml))) return -2;
  int rc;
  switch (cp / 64) {
    case 1: rc = launch_latent_decode<1>(p, s); break;
    case 2: rc = launch_latent_decode<2>(p, s); break;
    case 3: rc = launch_latent_decode<3>(p, s); break;
    case 4: rc = launch_latent_decode<4>(p, s); break;
    case 5: rc = launch_latent_decode<5>(p, s); break;
    case 6: rc = launch_latent_decode<6>(p, s); break;
    case 7: rc = launch_latent_decode<7>(p, s); break;
    default: rc = launch_latent_decode<8>(p, s); break;
  }
  if (rc || splits == 1) return rc;
  launch_pdl(latent_merge_kernel, dim3(static_cast<unsigned>(rows * H)), dim3(128), 0, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}
