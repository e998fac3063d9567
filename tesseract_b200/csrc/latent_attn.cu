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
//   latent_decode_kernel  attention of single rows in the latent space on tcgen05 (bf16), split over keys; the pool row serves
//                         as key and, its first cp columns, as value, so it is read once for 32 heads.
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
  const int n = (threadIdx.x & 31) * 2;
  if (n >= cols) return;                           // (N is even)
  const T* gate = p.gate ? static_cast<const T*>(p.gate) + h * p.oh + n0 + n : nullptr;
  T* out = static_cast<T*>(p.out) + h * p.oh + n0 + n;
  struct alignas(2 * sizeof(T)) Two { T v[2]; };
  constexpr int kPer = BM / 4 < 8 ? BM / 4 : 8;    // rows whose gates are requested together
#pragma unroll
  for (int r0 = threadIdx.x >> 5; r0 < BM; r0 += 4 * kPer) {
    Two g[kPer];
#pragma unroll
    for (int i = 0; i < kPer; ++i)
      if (gate) g[i] = *reinterpret_cast<const Two*>(gate + static_cast<long long>(m0 + min(r0 + 4 * i, rows - 1)) * p.ldg);
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int m = r0 + 4 * i;
      if (m >= rows) break;
      float2 a = *reinterpret_cast<const float2*>(acc + m * Tile::kLdC + n);
      if (gate) {
        const float x = p.gate_scale * to_f32<T>(g[i].v[0]), y = p.gate_scale * to_f32<T>(g[i].v[1]);
        a.x *= sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-x)) : sigmoid_f32(x);
        a.y *= sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-y)) : sigmoid_f32(y);
      }
      T* o = out + static_cast<long long>(m0 + m) * p.ldo;
      if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(o) = pack_bf16x2(a.x, a.y);
      else *reinterpret_cast<float2*>(o) = a;
    }
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
constexpr int kHeads = 32;         // heads of a CTA
constexpr int kBlockBytes = kKeys * 128;      // 64 keys x 64 columns, 128-byte swizzle

// One CTA per (key split, 32 heads, row); a tile of 64 pool rows is brought in once (TMA, one box per run of rows of a page and
// 64 columns) and is the B operand of the scores and the A operand of the read-out:
//   S[head, key]   = q[head, :] . row[key, :]       A = q in tensor memory, the 32 heads once in every quarter of the lanes
//   O[col, head]  += row[key, col] P[head, key]     M = 128 columns a time, N = heads: no row of the product is padding
// Warps 0 .. 3 turn scores into weights: lane = head, each warp reads its own quarter of the lanes and takes 16 of the keys. The
// reference maximum is lazy as in flash_attn_fwd.cu: O is rescaled only when a head's maximum has grown by more than 2^8. Warp 4
// loads, warp 5 issues the products.
struct LatentPlan {
  int blocks, stages, m_tiles, tmem_cols, smem;
  __host__ __device__ LatentPlan(int cp, int L) {
    blocks = (L + 63) / 64;
    m_tiles = (cp + 127) / 128;
    const int tile = blocks * kBlockBytes, room = 227 * 1024 - 4096 - kHeads * 128;
    stages = room / tile < 4 ? room / tile : 4;
    smem = 1024 + kHeads * 128 + stages * tile;
    const int cols = m_tiles * kHeads + kKeys + blocks * 32;
    tmem_cols = cols <= 128 ? 128 : cols <= 256 ? 256 : 512;
    if (cols > 512) stages = 0;
  }
};

__global__ void __launch_bounds__(192, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_pool, LatentAttnParams p) {
  pdl_grid_wait();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int L = p.cp + p.rp;
  const LatentPlan plan(p.cp, L);
  const int NB = plan.blocks, stages = plan.stages, m_tiles = plan.m_tiles;
  uint8_t* sp = smem;                                  // [32 heads][128 B]
  uint8_t* sk = sp + kHeads * 128;                     // [stages][NB][64 keys][128 B]
  __shared__ __align__(8) uint64_t q_in, q_full, k_full[4], k_empty[4], s_full, s_free, p_full, o_full;
  __shared__ uint32_t tmem_base_smem;
  __shared__ volatile int cta_abort;
  __shared__ float smax[2][4][kHeads], lsum[4][kHeads], corr[kHeads];
  const int split = blockIdx.z, h0 = blockIdx.y * kHeads, row = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int len = p.lens ? p.lens[row] : p.pos[row] + 1;
  const int share = ((len + p.splits - 1) / p.splits + kKeys - 1) / kKeys * kKeys;
  const int t_begin = split * share, t_end = min(len, t_begin + share);
  const int n_tiles = t_end > t_begin ? (t_end - t_begin + kKeys - 1) / kKeys : 0;

  if (threadIdx.x == 0) {
    cta_abort = 0;
    mbar_init(&q_in, 1);
    mbar_init(&q_full, 128);
    for (int i = 0; i < 4; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
    }
    mbar_init(&s_full, 1);
    mbar_init(&s_free, 128);
    mbar_init(&p_full, 128);
    mbar_init(&o_full, 1);
    mbar_fence_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_pool);
  }
  if (warp == 5) {
    tmem_alloc(&tmem_base_smem, plan.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // Only now may successors start: one that allocates tensor memory ahead of its own wait must not take it from a CTA of this
  // grid, on whose end it depends.
  pdl_trigger();
  const uint32_t tmem = tmem_base_smem, tmem_s = tmem + m_tiles * kHeads, tmem_q = tmem_s + kKeys;

  if (warp == 4) {
    // ---------------------------------------------------------------- loads: a lane per run of rows inside a page
    if (n_tiles > 0) {
      // the queries land in the last stage on their way to tensor memory
      if (lane == 0) mbar_expect_tx(&q_in, NB * kHeads * 128);
      __syncwarp();
      if (lane < NB) tma_load_2d(sk + (stages - 1) * NB * kBlockBytes + lane * kHeads * 128, &tm_q, &q_in, lane * 64, row * p.H + h0);
      const int* table = p.tables + static_cast<long long>(p.seq_of ? p.seq_of[row] : row) * p.table_ld;
      int run = 64;
      while (p.bs % run) run >>= 1;                    // rows that are neighbours in the pool: 64, 32, 16 or 8
      const int runs = kKeys / run;
      auto pool_row = [&](int j) {                     // first pool row of this lane's run; past the keys: past the pool (zeros)
        const int t = t_begin + j * kKeys + lane * run;
        if (lane >= runs || t >= t_end) return p.nb * p.bs;
        int blk = table[t / p.bs];
        if (blk < 0 || blk >= p.nb) {                  // never read another page: zeros instead, and the host hears of it
          if (p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
          return p.nb * p.bs;
        }
        return blk * p.bs + t % p.bs;
      };
      int next = pool_row(0);
      for (int j = 0; j < n_tiles; ++j) {
        const int st = j % stages, y = next;
        if (j + 1 < n_tiles) next = pool_row(j + 1);
        bool ok = mbar_wait(&k_empty[st], ((j / stages) & 1) ^ 1u, &cta_abort, p.status);
        if (j == stages - 1) ok = ok && mbar_wait(&q_full, 0, &cta_abort, p.status);
        if (!__all_sync(0xffffffffu, ok ? 1 : 0)) break;
        if (lane == 0) mbar_expect_tx(&k_full[st], NB * kBlockBytes);
        __syncwarp();
        if (lane < runs) {
          uint8_t* dst = sk + st * NB * kBlockBytes + lane * run * 128;
          for (int b = 0; b < NB; ++b) tma_load_2d(dst + b * kBlockBytes, &tm_pool, &k_full[st], b * 64, y);
        }
      }
    }
  } else if (warp == 5) {
    // ---------------------------------------------------------------- products
    // The products are small (16 - 32 cycles each), so what surrounds them counts: the whole warp walks the loop and works out the
    // descriptors, which keeps them uniform, and lane 0 alone is predicated on for the instruction itself.
    if (n_tiles > 0) {
      constexpr uint32_t idesc_s = umma_idesc(128, kKeys, 1, 1, 0, 0);       // both K-major
      constexpr uint32_t idesc_o = umma_idesc(128, kHeads, 1, 1, 1, 0);      // pool rows: columns contiguous (M-major)
      const uint32_t leader = lane == 0;
      const uint64_t k_desc = umma_smem_desc_sw128(smem_u32(sk), 16, 1024), v_desc = umma_smem_desc_sw128(smem_u32(sk), kBlockBytes, 1024),
                     p_desc = umma_smem_desc_sw128(smem_u32(sp), 16, 1024);
      const uint32_t tile16 = NB * kBlockBytes / 16;                         // descriptors count 16-byte units
      bool ok = __all_sync(0xffffffffu, mbar_wait(&q_full, 0, &cta_abort, p.status) ? 1 : 0) != 0;
      // scores of tile j and the read-out of tile j - 1, whichever can start first: the load of a later tile waits for the
      // read-out, so a read-out must not wait for a tile that is still on its way
      uint32_t st = 0, sv = 0;                                               // stages of tiles j and j - 1
      for (int j = 0; ok && j <= n_tiles; ++j) {
        bool score = j < n_tiles, read = j > 0;
        const long long since = clock64();
        while (score || read) {
          if (score && __all_sync(0xffffffffu, mbar_test_wait(&k_full[st], (j / stages) & 1) && mbar_test_wait(&s_free, (j & 1) ^ 1u))) {
            tc_fence_after();
            uint64_t d = k_desc + st * tile16;
            uint32_t a = tmem_q;
            umma_f16_ts_if(leader, tmem_s, a, d, idesc_s, 0);
            umma_f16_ts_if(leader, tmem_s, a + 8, d + 2, idesc_s, 1);
            umma_f16_ts_if(leader, tmem_s, a + 16, d + 4, idesc_s, 1);
            umma_f16_ts_if(leader, tmem_s, a + 24, d + 6, idesc_s, 1);
            for (int b = 1; b < NB; ++b) {
              a += 32;
              d += kBlockBytes / 16;
              umma_f16_ts_if(leader, tmem_s, a, d, idesc_s, 1);
              umma_f16_ts_if(leader, tmem_s, a + 8, d + 2, idesc_s, 1);
              umma_f16_ts_if(leader, tmem_s, a + 16, d + 4, idesc_s, 1);
              umma_f16_ts_if(leader, tmem_s, a + 24, d + 6, idesc_s, 1);
            }
            if (leader) umma_commit(&s_full);
            score = false;
          }
          if (read && __all_sync(0xffffffffu, mbar_test_wait(&p_full, (j - 1) & 1))) {
            tc_fence_after();
            uint64_t d = v_desc + sv * tile16;
            for (int m = 0; m < m_tiles; ++m) {
              umma_f16_if(leader, tmem + m * kHeads, d, p_desc, idesc_o, j > 1);
              umma_f16_if(leader, tmem + m * kHeads, d + 128, p_desc + 2, idesc_o, 1);
              umma_f16_if(leader, tmem + m * kHeads, d + 256, p_desc + 4, idesc_o, 1);
              umma_f16_if(leader, tmem + m * kHeads, d + 384, p_desc + 6, idesc_o, 1);
              d += 2 * kBlockBytes / 16;
            }
            if (leader) {
              umma_commit(&o_full);
              umma_commit(&k_empty[sv]);
            }
            read = false;
          }
          if (cta_abort) ok = false;
          if (clock64() - since > kWaitCycleLimit) {
            cta_abort = 1;
            if (p.status) atomicCAS(p.status, kStatusOk, kStatusMbarTimeout);
            ok = false;
          }
          ok = __all_sync(0xffffffffu, ok ? 1 : 0) != 0;
          if (!ok) break;
        }
        sv = st;
        st = st + 1 == static_cast<uint32_t>(stages) ? 0 : st + 1;
      }
    }
  } else {
    // ---------------------------------------------------------------- queries, weights, rescaling and output
    const uint32_t lanes = static_cast<uint32_t>(warp * 32) << 16;
    const float scale_log2 = p.scale * 1.4426950408889634f;
    if (n_tiles > 0) {
      const bool ok = mbar_wait(&q_in, 0, &cta_abort, p.status);
      if (__all_sync(0xffffffffu, ok ? 1 : 0)) {
        const uint8_t* sq = sk + (stages - 1) * NB * kBlockBytes + lane * 128;
        for (int b = 0; b < NB; ++b) {
          uint32_t r[32];
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            const uint4 v = *reinterpret_cast<const uint4*>(sq + b * kHeads * 128 + (i ^ (lane & 7)) * 16);
            r[4 * i] = v.x; r[4 * i + 1] = v.y; r[4 * i + 2] = v.z; r[4 * i + 3] = v.w;
          }
          tmem_st_32x32(tmem_q + lanes + b * 32, r);
        }
        tmem_st_wait();
        tc_fence_before();
        fence_proxy_async_smem();                      // (the last stage's next writer is the asynchronous proxy)
        mbar_arrive(&q_full);
      }
    }
    float m_ref = -INFINITY, l = 0.f;
    bool good = true;
    for (int j = 0; j < n_tiles; ++j) {
      // (every warp passes each barrier below once per tile whether its waits succeed or not; a failure is told through smax)
      bool ok = mbar_wait(&s_full, j & 1, &cta_abort, p.status);
      ok = __all_sync(0xffffffffu, ok ? 1 : 0) != 0;
      uint32_t s[16];
      float m_own = -INFINITY;
      const int vis = t_end - (t_begin + j * kKeys + warp * 16);
      if (ok) {
        tc_fence_after();
        tmem_ld_32x16(tmem_s + lanes + warp * 16, s);
        tmem_ld_wait();
        tc_fence_before();
        mbar_arrive(&s_free);
#pragma unroll
        for (int i = 0; i < 16; ++i)
          if (i < vis) m_own = fmaxf(m_own, __uint_as_float(s[i]));
      }
      smax[j & 1][warp][lane] = ok ? m_own : INFINITY;
      asm volatile("bar.sync 1, 128;" ::: "memory");
      float m_tile = -INFINITY;
#pragma unroll
      for (int w = 0; w < 4; ++w) m_tile = fmaxf(m_tile, smax[j & 1][w][lane]);
      if (__any_sync(0xffffffffu, m_tile == INFINITY)) {      // the same answer in all four warps
        good = false;
        break;
      }
      float factor = 1.f;
      bool grow = false;
      if (j == 0) {
        m_ref = m_tile;
      } else if ((m_tile - m_ref) * scale_log2 > 8.f) {
        factor = exp2f((m_ref - m_tile) * scale_log2);
        m_ref = m_tile;
        grow = true;
      }
      l *= factor;
      const float mneg = -m_ref * scale_log2;
      uint32_t w8[8];
      // weights as the tensor core will read them; the denominator sums those
#pragma unroll
      for (int i = 0; i < 16; i += 2) {
        const float p0 = i < vis ? exp2f(fmaf(__uint_as_float(s[i]), scale_log2, mneg)) : 0.f;
        const float p1 = i + 1 < vis ? exp2f(fmaf(__uint_as_float(s[i + 1]), scale_log2, mneg)) : 0.f;
        const __nv_bfloat162 pb = __floats2bfloat162_rn(p0, p1);
        l += __low2float(pb) + __high2float(pb);
        w8[i >> 1] = *reinterpret_cast<const uint32_t*>(&pb);
      }
      // the read-out before must be finished: it reads the weights in shared memory, and rescaling rewrites its result
      if (j > 0) {
        ok = mbar_wait(&o_full, (j - 1) & 1, &cta_abort, p.status);
        ok = __all_sync(0xffffffffu, ok ? 1 : 0) != 0;
        if (__any_sync(0xffffffffu, grow)) {           // (the same in all four warps)
          tc_fence_after();
          if (warp == 0) corr[lane] = factor;
          asm volatile("bar.sync 2, 128;" ::: "memory");
          for (int m = 0; ok && m < m_tiles; ++m) {
            uint32_t r[32];
            tmem_ld_32x32(tmem + lanes + m * kHeads, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * corr[i]);
            tmem_st_32x32(tmem + lanes + m * kHeads, r);
          }
          tmem_st_wait();
        }
      }
      uint8_t* prow = sp + lane * 128;
#pragma unroll
      for (int c = 0; c < 2; ++c)
        *reinterpret_cast<uint4*>(prow + ((2 * warp + c) ^ (lane & 7)) * 16) = make_uint4(w8[4 * c], w8[4 * c + 1], w8[4 * c + 2], w8[4 * c + 3]);
      fence_proxy_async_smem();
      tc_fence_before();
      if (ok) mbar_arrive(&p_full);
    }
    lsum[warp][lane] = l;
    asm volatile("bar.sync 1, 128;" ::: "memory");
    const float sum = lsum[0][lane] + lsum[1][lane] + lsum[2][lane] + lsum[3][lane];
    if (warp == 0) {
      corr[lane] = p.splits > 1 ? 1.f : sum > 0.f ? 1.f / sum : 0.f;
      if (p.splits > 1 && h0 + lane < p.H) {
        float* ml = p.part_ml + ((static_cast<long long>(row) * p.H + h0 + lane) * p.splits + split) * 2;
        ml[0] = n_tiles > 0 ? m_ref * scale_log2 : -INFINITY;
        ml[1] = sum;
      }
    }
    asm volatile("bar.sync 1, 128;" ::: "memory");
    bool have = false;
    if (good && n_tiles > 0) have = mbar_wait(&o_full, (n_tiles - 1) & 1, &cta_abort, p.status);
    have = __all_sync(0xffffffffu, have ? 1 : 0) != 0;
    if (have) tc_fence_after();
    for (int m = 0; m < m_tiles; ++m) {
      uint32_t r[32];
      if (have) {
        tmem_ld_32x32(tmem + lanes + m * kHeads, r);
        tmem_ld_wait();
      } else {
#pragma unroll
        for (int i = 0; i < 32; ++i) r[i] = 0u;
      }
      const int c = m * 128 + warp * 32 + lane;
      const long long at = static_cast<long long>(row) * p.H + h0;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        if (h0 + i >= p.H || c >= p.cp) break;
        const float v = __uint_as_float(r[i]);
        if (p.splits == 1) static_cast<__nv_bfloat16*>(p.out)[(at + i) * p.cp + c] = __float2bfloat16_rn(v * corr[i]);
        else p.part_o[((at + i) * p.splits + split) * p.cp + c] = v;
      }
      __syncwarp();
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem, plan.tmem_cols);
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

int launch_latent_decode(const LatentAttnParams& p, cudaStream_t s) {
  const int L = p.cp + p.rp;
  const LatentPlan plan(p.cp, L);
  if (plan.stages < 2) return -2;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - 3072);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  int run = 64;
  while (p.bs % run) run >>= 1;
  CUtensorMap tm_q, tm_pool;
  if (!make_tmap_2d(&tm_q, p.q, 2, static_cast<uint64_t>(p.rows) * p.H, L, L * 2ull, kHeads, 64, true) ||
      !make_tmap_2d(&tm_pool, p.pool, 2, static_cast<uint64_t>(p.nb) * p.bs, L, L * 2ull, run, 64, true)) return -3;
  launch_pdl(latent_decode_kernel, dim3(p.rows, (p.H + kHeads - 1) / kHeads, p.splits), dim3(192), plan.smem, s, pdl_all_enabled(), tm_q,
             tm_pool, p);
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
  if (rows <= 0 || H <= 0 || H > 65535 || N <= 0 || N % 2 || K <= 0 || K % 16 || ldx % 8 || xh % 8 || wh % 8 || ldw % 8 || ldw < K || ldo % 2 || oh % 2 || (gate && ldg % 2)) return -2;
  HeadLinearParams p{x, ldx, xh, w, wh, ldw, out, ldo, oh, gate, ldg, gate_scale, rows, N, K};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool few = rows <= 64;
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
  if (dtype != 1 || cp % 64 || cp > 512 || rp % 32 || rp <= 0 || bs % 8 || splits > 65535 || (splits > 1 && (!part_o || !part_ml))) return -2;
  const int rc = launch_latent_decode(p, s);
  if (rc || splits == 1) return rc;
  launch_pdl(latent_merge_kernel, dim3(static_cast<unsigned>(rows * H)), dim3(128), 0, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}
