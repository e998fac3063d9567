// Mixture-of-experts feed-forward for serving: which experts a token takes, and W_down relu(W_up h)^2 of every one.
//
//   s = sigmoid(z), c = s + correction       (z: router logits, fp32)
//   a group of neighbours is worth the sum of its two largest c; the experts of the `keep` best groups stay
//   the `top` largest c among them are taken, with weights s / (sum s + 1e-20) * scale
//
// One warp chooses for one token. Assignments are then laid out expert by expert, every expert's rows padded to a multiple of `pad`
// (`offsets` [E + 1], `assign` [row] = token * top + place or -1, `pos` [token * top + place] = row). Up to kPlanTokens tokens one CTA
// does all of that. Few rows per expert: expert_tile_kernel, tiles of 16 or 64 rows, which picks the rows by `assign` on the way in;
// many (bf16): expert_gather_kernel and the grouped tcgen05 GEMM. The weighted sum over a token's experts is left to the residual
// step, which takes `pos` and the weights.
#include "head_tile.cuh"

#include <algorithm>

namespace tsb {
namespace {

constexpr int kMaxExperts = 256, kMaxTop = 32, kPlanTokens = 64, kPlanWarps = 32, kRouteWarps = 8;

struct RouteParams {
  const float* logits;       // [slices, T, ld]: the sum over slices
  long long ld;
  int slices;
  const float* correction;   // [E]
  int T, E, top, groups, keep, pad;
  float scale;
  int* idx;                  // [T, top]
  float* weight;             // [T, top]
  int* counts;               // [E], then E cursors (zero)
  int* offsets;              // [E + 1]
  int* pos;                  // [T, top]
  int* assign;               // [rows]
};

// The warp's choice for one token: lane r < top returns its r-th expert and weight. SL experts a lane; sm: 3 E floats of the warp's own.
template <int SL>
__device__ __forceinline__ void choose(const RouteParams& p, int token, float* sm, int* expert, float* weight) {
  const int lane = threadIdx.x & 31, size = p.E / p.groups;
  const float* z = p.logits + token * p.ld;
  float *choice = sm, *worth = sm + p.E, *score = worth + p.E;
  float c[SL];
#pragma unroll
  for (int i = 0; i < SL; ++i) {
    const int e = lane + 32 * i;
    c[i] = -INFINITY;
    if (e >= p.E) continue;
    float sum = 0.f;
    for (int k = 0; k < p.slices; ++k) sum += z[k * p.T * p.ld + e];
    score[e] = sigmoid_f32(sum);
    choice[e] = c[i] = score[e] + p.correction[e];
  }
  __syncwarp();
  if (p.keep < p.groups) {
    for (int g = lane; g < p.groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;
      for (int j = 0; j < size; ++j) {
        const float v = choice[g * size + j];
        b = fmaxf(b, fminf(a, v));
        a = fmaxf(a, v);
      }
      worth[g] = size > 1 ? a + b : a;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < SL; ++i) {
      const int e = lane + 32 * i;
      if (e >= p.E) continue;
      const int g = e / size;
      int better = 0;
      for (int o = 0; o < p.groups; ++o) better += worth[o] > worth[g] || (worth[o] == worth[g] && o < g);
      if (better >= p.keep) c[i] = -INFINITY;
    }
  }
  int mine = 0;
  for (int r = 0; r < p.top; ++r) {
    float bv = -INFINITY;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < SL; ++i)
      if (c[i] > bv) {
        bv = c[i];
        bi = lane + 32 * i;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) {
        bv = ov;
        bi = oi;
      }
    }
    bi = min(bi, p.E - 1);                             // (nothing compares with a NaN)
    if (lane == r) mine = bi;
#pragma unroll
    for (int i = 0; i < SL; ++i)
      if (lane + 32 * i == bi) c[i] = -INFINITY;
  }
  const float s = lane < p.top ? score[mine] : 0.f;
  *weight = s / (warp_sum(s) + 1e-20f) * p.scale;
  *expert = mine;
  __syncwarp();
}

// offsets of all experts' padded rows from their counts, by the whole CTA into shared memory [E + 1].
__device__ __forceinline__ void padded_offsets(const int* counts, int E, int pad, int* off) {
  for (int e = threadIdx.x; e < E; e += blockDim.x) off[e + 1] = (counts[e] + pad - 1) / pad * pad;
  __syncthreads();
  if (threadIdx.x < 32) {                              // eight experts a lane
    const int first = threadIdx.x * 8;
    int sum = 0;
    for (int i = 0; i < 8; ++i) sum += first + i < E ? off[first + i + 1] : 0;
    int before = sum;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, before, o);
      if (static_cast<int>(threadIdx.x) >= o) before += v;
    }
    before -= sum;
    if (threadIdx.x == 0) off[0] = 0;
    for (int i = 0; i < 8; ++i)
      if (first + i < E) off[first + i + 1] = before += off[first + i + 1];
  }
  __syncthreads();
}

// Up to kPlanTokens tokens: choice, counts, layout.
template <int SL>
__global__ void __launch_bounds__(kPlanWarps * 32)
expert_plan_kernel(RouteParams p) {
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ float choice_sm[];
  __shared__ int counts[kMaxExperts], cursor[kMaxExperts], off[kMaxExperts + 1];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int e = tid; e < p.E; e += blockDim.x) counts[e] = cursor[e] = 0;
  __syncthreads();
  for (int t = warp; t < p.T; t += kPlanWarps) {
    int e;
    float w;
    choose<SL>(p, t, choice_sm + warp * 3 * p.E, &e, &w);
    if (lane < p.top) {
      p.idx[t * p.top + lane] = e;
      p.weight[t * p.top + lane] = w;
      atomicAdd(&counts[e], 1);
    }
  }
  __syncthreads();
  padded_offsets(counts, p.E, p.pad, off);
  for (int e = tid; e <= p.E; e += blockDim.x) p.offsets[e] = off[e];
  for (int r = tid; r < off[p.E]; r += blockDim.x) p.assign[r] = -1;
  __syncthreads();
  for (int i = tid; i < p.T * p.top; i += blockDim.x) {
    const int e = p.idx[i], row = off[e] + atomicAdd(&cursor[e], 1);
    p.pos[i] = row;
    p.assign[row] = i;
  }
}

template <int SL>
__global__ void __launch_bounds__(kRouteWarps * 32)
expert_route_kernel(RouteParams p) {
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ float choice_sm[];
  __shared__ int counts[kMaxExperts];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int e = tid; e < p.E; e += blockDim.x) counts[e] = 0;
  __syncthreads();
  for (int t = blockIdx.x * kRouteWarps + warp; t < p.T; t += gridDim.x * kRouteWarps) {
    int e;
    float w;
    choose<SL>(p, t, choice_sm + warp * 3 * p.E, &e, &w);
    if (lane < p.top) {
      p.idx[static_cast<long long>(t) * p.top + lane] = e;
      p.weight[static_cast<long long>(t) * p.top + lane] = w;
      atomicAdd(&counts[e], 1);
    }
  }
  __syncthreads();
  for (int e = tid; e < p.E; e += blockDim.x)
    if (counts[e]) atomicAdd(&p.counts[e], counts[e]);
}

// A CTA places 1024 assignments: one global claim per expert, places inside it in shared memory.
__global__ void __launch_bounds__(256)
expert_place_kernel(RouteParams p) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ int off[kMaxExperts + 1], mine[kMaxExperts], base[kMaxExperts];
  const int tid = threadIdx.x;
  padded_offsets(p.counts, p.E, p.pad, off);
  if (blockIdx.x == 0)
    for (int e = tid; e <= p.E; e += blockDim.x) p.offsets[e] = off[e];
  for (int e = blockIdx.x; e < p.E; e += gridDim.x)    // padding rows
    for (int r = off[e] + p.counts[e] + tid; r < off[e + 1]; r += blockDim.x) p.assign[r] = -1;
  for (int e = tid; e < p.E; e += blockDim.x) mine[e] = 0;
  __syncthreads();
  const long long n = static_cast<long long>(p.T) * p.top, first = blockIdx.x * 1024ll;
  int e[4], at[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const long long i = first + k * 256 + tid;
    e[k] = i < n ? p.idx[i] : -1;
    if (e[k] >= 0) at[k] = atomicAdd(&mine[e[k]], 1);
  }
  __syncthreads();
  for (int x = tid; x < p.E; x += blockDim.x) base[x] = mine[x] ? off[x] + atomicAdd(&p.counts[p.E + x], mine[x]) : 0;
  __syncthreads();
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const long long i = first + k * 256 + tid;
    if (e[k] < 0) continue;
    const int row = base[e[k]] + at[k];
    p.pos[i] = row;
    p.assign[row] = static_cast<int>(i);
  }
}

// dst[row] = src[assign[row] / top] (zeros on padding), 16 bytes a thread.
__global__ void __launch_bounds__(256)
expert_gather_kernel(const uint4* src, long long lds, const int* assign, const int* total, uint4* dst, int vecs, int top) {
  pdl_trigger();
  pdl_grid_wait();
  const int rows = *total;
  const long long n = static_cast<long long>(rows) * vecs, step = gridDim.x * 256ll;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < n; i += 4 * step) {
    uint4 v[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const long long j = i + k * step;
      v[k] = make_uint4(0u, 0u, 0u, 0u);
      if (j >= n) continue;
      const int row = static_cast<int>(j / vecs), a = assign[row];
      if (a >= 0) v[k] = src[(a / top) * lds + (j - static_cast<long long>(row) * vecs)];
    }
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (i + k * step < n) dst[i + k * step] = v[k];
  }
}

// logits[slice] [T, ld] = x W^T over the slice's columns: one tile of 16 tokens and 64 experts a CTA. Few tokens against a narrow matrix:
// the columns are cut so that the whole is not one CTA's walk; whoever reads the logits sums the slices.
template <typename T>
__global__ void __launch_bounds__(128)
expert_logits_kernel(const T* x, long long ldx, const T* w, long long ldw, float* out, long long ld, int rows, int N, int K, int step) {
  pdl_trigger();
  pdl_grid_wait();
  using Tile = HeadTile<T, 16, 1>;
  extern __shared__ __align__(16) uint8_t smem[];
  const int n0 = blockIdx.x * 64, row0 = blockIdx.y * 16, k0 = blockIdx.z * step, cols = min(64, N - n0);
  const T* const wp[1] = {w + n0 * ldw + k0};
  auto row = [&](int r) -> const T* { return row0 + r < rows ? x + (row0 + r) * ldx + k0 : nullptr; };
  const float* c = Tile::run_rows(smem, row, wp, ldw, cols, min(step, K - k0));
  for (int i = threadIdx.x; i < 16 * 64; i += 128) {
    const int r = i >> 6, n = i & 63;
    if (row0 + r < rows && n < cols) out[(static_cast<long long>(blockIdx.z) * rows + row0 + r) * ld + n0 + n] = c[r * Tile::kLdC + n];
  }
}

template <typename T>
int run_logits(const T* x, long long ldx, const T* w, long long ldw, float* out, long long ld, int rows, int N, int K, int slices, cudaStream_t s) {
  auto kern = expert_logits_kernel<T>;
  constexpr int smem = HeadTile<T, 16, 1>::kSmem;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  const int step = ((K + slices - 1) / slices + 15) / 16 * 16;
  if ((slices - 1) * step >= K) return -2;                   // (a slice without columns)
  launch_pdl(kern, dim3((N + 63) / 64, (rows + 15) / 16, slices), dim3(128), smem, s, pdl_all_enabled(), x, ldx, w, ldw, out, ld, rows, N, K, step);
  return static_cast<int>(cudaGetLastError());
}

template <int SL>
int run_route(const RouteParams& p, cudaStream_t s) {
  const bool pdl = pdl_all_enabled();
  if (p.T <= kPlanTokens) {
    static PerDeviceFlag attr;
    auto kern = expert_plan_kernel<SL>;
    if (attr.unset()) {
      const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kPlanWarps * 3 * 32 * SL * 4);
      if (e != cudaSuccess) return static_cast<int>(e);
      attr.set();
    }
    launch_pdl(kern, dim3(1), dim3(kPlanWarps * 32), kPlanWarps * 3 * p.E * 4, s, pdl, p);
    return static_cast<int>(cudaGetLastError());
  }
  const cudaError_t e = cudaMemsetAsync(p.counts, 0, 2 * p.E * sizeof(int), s);
  if (e != cudaSuccess) return static_cast<int>(e);
  const int ctas = std::min((p.T + kRouteWarps - 1) / kRouteWarps, sm_count() * 8);
  launch_pdl(expert_route_kernel<SL>, dim3(ctas), dim3(kRouteWarps * 32), kRouteWarps * 3 * p.E * 4, s, false, p);
  const long long n = static_cast<long long>(p.T) * p.top;
  launch_pdl(expert_place_kernel, dim3(static_cast<unsigned>((n + 1023) / 1024)), dim3(256), 0, s, pdl, p);
  return static_cast<int>(cudaGetLastError());
}

struct ExpertParams {
  const void* x;             // UP: [T, ldx] rows of tokens; else [rows, ldx]
  long long ldx;
  const void* w;             // [E, N, ldw]
  long long ldw;
  void* y;                   // [rows, ldy]
  long long ldy;
  const int *offsets, *assign;
  int E, N, K, top;
};

// One tile of BM rows of one expert and 64 result columns. UP: rows by `assign`, relu(..)^2.
template <typename T, int BM, bool UP>
__global__ void __launch_bounds__(128)
expert_tile_kernel(ExpertParams p) {
  pdl_trigger();
  pdl_grid_wait();
  using Tile = HeadTile<T, BM, 1>;
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ int expert, row_of[BM];
  const int row0 = blockIdx.y * BM, n0 = blockIdx.x * 64, tid = threadIdx.x;
  if (row0 >= p.offsets[p.E]) return;
  for (int e = tid; e < p.E; e += 128)
    if (p.offsets[e] <= row0 && row0 < p.offsets[e + 1]) expert = e;
  if (UP && tid < BM) {
    const int a = p.assign[row0 + tid];
    row_of[tid] = a < 0 ? -1 : a / p.top;
  }
  __syncthreads();
  const T* const w[1] = {static_cast<const T*>(p.w) + (static_cast<long long>(expert) * p.N + n0) * p.ldw};
  const T* x = static_cast<const T*>(p.x);
  auto row = [&](int r) -> const T* {
    if (!UP) return x + (row0 + r) * p.ldx;
    return row_of[r] < 0 ? nullptr : x + row_of[r] * p.ldx;
  };
  const float* c = Tile::run_rows(smem, row, w, p.ldw, min(64, p.N - n0), p.K);
  const bool vec = p.ldy % 4 == 0 && n0 + 64 <= p.N;
  for (int i = tid; i < BM * 16; i += 128) {
    const int r = i >> 4, n = (i & 15) * 4;
    const float4 v = *reinterpret_cast<const float4*>(c + r * Tile::kLdC + n);
    float f[4] = {v.x, v.y, v.z, v.w};
    if (UP) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        f[j] = fmaxf(f[j], 0.f);
        f[j] *= f[j];
      }
    }
    T* y = static_cast<T*>(p.y) + (row0 + r) * p.ldy + n0 + n;
    if (vec) {
      if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(y) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
      else *reinterpret_cast<float4*>(y) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (n0 + n + j < p.N) y[j] = from_f32<T>(f[j]);
    }
  }
}

template <typename T, int BM, bool UP>
int launch_tile(const ExpertParams& p, int tiles, cudaStream_t s) {
  auto kern = expert_tile_kernel<T, BM, UP>;
  constexpr int smem = HeadTile<T, BM, 1>::kSmem;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  launch_pdl(kern, dim3((p.N + 63) / 64, tiles), dim3(128), smem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int run_tile(const ExpertParams& p, int tiles, int bm, int up, cudaStream_t s) {
  if (bm == 16) return up ? launch_tile<T, 16, true>(p, tiles, s) : launch_tile<T, 16, false>(p, tiles, s);
  return up ? launch_tile<T, 64, true>(p, tiles, s) : launch_tile<T, 64, false>(p, tiles, s);
}

}  // namespace
}  // namespace tsb

// out [slices, rows, ld] fp32, summed over slices: x [rows, K] times w [N, K]^T. K is a multiple of 16, rows start on 16 bytes.
TSB_EXPORT int tsb_expert_logits(const void* x, long long ldx, const void* w, long long ldw, float* out, long long ld, int rows, int N, int K,
                                 int slices, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || N <= 0 || K <= 0 || K % 16 || ld < N || slices < 1 || slices > 64 || ldx % 8 || ldw % 8 || (reinterpret_cast<uintptr_t>(x) & 15) ||
      (reinterpret_cast<uintptr_t>(w) & 15))
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1)
    return run_logits(static_cast<const __nv_bfloat16*>(x), ldx, static_cast<const __nv_bfloat16*>(w), ldw, out, ld, rows, N, K, slices, s);
  if (dtype == 0) return run_logits(static_cast<const float*>(x), ldx, static_cast<const float*>(w), ldw, out, ld, rows, N, K, slices, s);
  return -2;
}

// ints: T, E, top, groups, keep, pad, slices; ptrs: logits, correction, idx, weight, counts, offsets, pos, assign (see RouteParams). counts
// has 2 E places; assign as many as T * top assignments of E experts may take with padding. Returns in offsets[E] (on the device) the rows
// in use.
TSB_EXPORT int tsb_expert_route(const int* v, long long ld, void* const* q, float scale, void* stream) {
  using namespace tsb;
  RouteParams p{static_cast<const float*>(q[0]), ld, v[6], static_cast<const float*>(q[1]), v[0], v[1], v[2], v[3], v[4], v[5], scale,
                static_cast<int*>(q[2]), static_cast<float*>(q[3]), static_cast<int*>(q[4]), static_cast<int*>(q[5]), static_cast<int*>(q[6]),
                static_cast<int*>(q[7])};
  if (p.T <= 0 || p.E <= 0 || p.E > kMaxExperts || p.top <= 0 || p.top > kMaxTop || p.groups <= 0 || p.E % p.groups || p.keep <= 0 ||
      p.keep > p.groups || p.top > p.E / p.groups * p.keep || p.pad <= 0 || p.ld < p.E || p.slices < 1 ||
      static_cast<long long>(p.T) * p.top > 0x3fffffff)
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (p.E <= 32) return run_route<1>(p, s);
  if (p.E <= 64) return run_route<2>(p, s);
  if (p.E <= 128) return run_route<4>(p, s);
  return run_route<8>(p, s);
}

// dst [rows_cap, cols] bf16: the first offsets[E] rows (`total` points at that number) are gathered. cols, lds: multiples of 8.
TSB_EXPORT int tsb_expert_gather(const void* src, long long lds, const int* assign, const int* total, void* dst, int rows_cap, int cols, int top,
                                 void* stream) {
  using namespace tsb;
  if (rows_cap <= 0 || cols <= 0 || cols % 8 || lds % 8 || top <= 0 || (reinterpret_cast<uintptr_t>(src) & 15)) return -2;
  const long long n = static_cast<long long>(rows_cap) * (cols / 8);
  const int grid = static_cast<int>(std::min<long long>((n + 1023) / 1024, sm_count() * 16));
  launch_pdl(expert_gather_kernel, dim3(grid), dim3(256), 0, static_cast<cudaStream_t>(stream), pdl_all_enabled(), static_cast<const uint4*>(src),
             lds / 8, assign, total, static_cast<uint4*>(dst), cols / 8, top);
  return static_cast<int>(cudaGetLastError());
}

// ints: E, N, K, top, tiles, bm (16 or 64, the padding of the rows), up; lds: x, w, y; ptrs: x, w, y, offsets, assign (see ExpertParams).
// K is a multiple of 16; rows of x and w start on 16 bytes.
TSB_EXPORT int tsb_expert_tiles(const int* v, const long long* ld, void* const* q, int dtype, void* stream) {
  using namespace tsb;
  ExpertParams p{q[0], ld[0], q[1], ld[1], q[2], ld[2], static_cast<const int*>(q[3]), static_cast<const int*>(q[4]), v[0], v[1], v[2], v[3]};
  const int tiles = v[4], bm = v[5];
  if (p.E <= 0 || p.E > kMaxExperts || p.N <= 0 || p.K <= 0 || p.K % 16 || p.top <= 0 || tiles <= 0 || tiles > 65535 || (bm != 16 && bm != 64) ||
      p.ldx % 8 || p.ldw % 8 || p.ldw > (1 << 24) || (reinterpret_cast<uintptr_t>(p.x) & 15) || (reinterpret_cast<uintptr_t>(p.w) & 15) ||
      (reinterpret_cast<uintptr_t>(p.y) & 15) || !p.offsets || (v[6] && !p.assign))
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) return run_tile<__nv_bfloat16>(p, tiles, bm, v[6], s);
  if (dtype == 0) return run_tile<float>(p, tiles, bm, v[6], s);
  return -2;
}
