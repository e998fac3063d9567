// Residual step of blocks whose sublayers run side by side, with depth averaging and an RMS norm of one gain, in one pass
// over the row; the residual stream and everything it is made of are fp32.
//
//   X   = E[token]                        (start of the model)   or   X = x + mult * y     (y: sum of the sublayers)
//   x   = sum_j avg[j] hist[j] + avg[n] X  (avg given: hist[0 .. n - 1] are the earlier X; X becomes hist[n])  or   x = X
//   h   = x / sqrt(mean(x^2) + eps) * gain  (input of the next product, in its type, zero up to a padded width)
//
// One CTA per row: the row's columns stay in registers between the sums and the norm. Per element: 4 bytes of every earlier
// X, x in and out, X out, y in, h out; bound by memory.
#include "common.cuh"

#include <algorithm>

namespace tsb {
namespace {

struct DepthParams {
  const float* x_in;      // [rows, W]; unused at the start of the model
  float* x_out;           // [rows, W] or null (nothing reads it: at the start x is hist[0])
  float* hist;            // [.., rows, W] or null
  long long hist_ld;      // elements between two entries of hist
  const float* avg;       // [n_hist + 1] or null
  int n_hist;             // earlier entries
  int store;              // X is stored as hist[n_hist]
  const void* y;
  long long ldy;
  float mult;
  const int* tokens;      // start of the model
  const void* table;
  long long ld_table;
  int vocab;
  void* h;                // or null
  long long ldh;
  int h_cols, rows, W;
  float gain, eps;
  int* status;
};

template <typename T, int V>
__device__ __forceinline__ void load_n(const T* p, float (&f)[V]) {
  if constexpr (V == 1) {
    f[0] = to_f32<T>(*p);
  } else if constexpr (sizeof(T) == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  } else {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const T* e = reinterpret_cast<const T*>(&a);
#pragma unroll
    for (int i = 0; i < 4; ++i) f[i] = to_f32<T>(e[i]);
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_n(T* p, const float (&f)[V]) {
  if constexpr (V == 1) {
    *p = from_f32<T>(f[0]);
  } else if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  }
}

// KEEP groups of V columns per thread stay in registers; rows wider than that are read back from x_out for the norm
// (KEEP = 0).
template <typename T, int V, int KEEP>
__global__ void __launch_bounds__(256)
depth_residual_kernel(DepthParams p) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ float red[8];
  const int row = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  const long long base = static_cast<long long>(row) * p.W;
  const T* src;
  if (p.tokens) {
    int tok = p.tokens[row];
    if (tok < 0 || tok >= p.vocab) {
      if (tid == 0 && p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
      tok = 0;
    }
    src = static_cast<const T*>(p.table) + tok * p.ld_table;
  } else {
    src = static_cast<const T*>(p.y) + row * p.ldy;
  }
  constexpr int N = KEEP > 0 ? KEEP : 1;
  float keep[N][V];
  float ss = 0.f;
  auto column = [&](int c, float (&x)[V]) {
    load_n<T, V>(src + c, x);
    if (!p.tokens) {
      float r[V];
      load_n<float, V>(p.x_in + base + c, r);
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] = fmaf(p.mult, x[i], r[i]);
    }
    if (p.store) store_n<float, V>(p.hist + p.n_hist * p.hist_ld + base + c, x);
    if (p.avg) {
      const float w = p.avg[p.n_hist];
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] *= w;
      const float* past = p.hist + base + c;
#pragma unroll 4
      for (int j = 0; j < p.n_hist; ++j) {
        float r[V];
        load_n<float, V>(past + j * p.hist_ld, r);
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] = fmaf(p.avg[j], r[i], x[i]);
      }
    }
    if (p.x_out) store_n<float, V>(p.x_out + base + c, x);
#pragma unroll
    for (int i = 0; i < V; ++i) ss = fmaf(x[i], x[i], ss);
  };
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = (k * nt + tid) * V;
      if (c < p.W) column(c, keep[k]);
    }
  } else {
    for (int c = tid * V; c < p.W; c += nt * V) column(c, keep[0]);
  }
  if (!p.h) return;
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < nt / 32; ++w) ss += red[w];
  const float r = p.gain / sqrtf(ss / static_cast<float>(p.W) + p.eps);
  T* h = static_cast<T*>(p.h) + row * p.ldh;
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = (k * nt + tid) * V;
      if (c >= p.W) break;
#pragma unroll
      for (int i = 0; i < V; ++i) keep[k][i] *= r;
      store_n<T, V>(h + c, keep[k]);
    }
  } else {
    const float* x = p.x_out ? p.x_out : p.hist + p.n_hist * p.hist_ld;
    for (int c = tid * V; c < p.W; c += nt * V) {
      load_n<float, V>(x + base + c, keep[0]);
#pragma unroll
      for (int i = 0; i < V; ++i) keep[0][i] *= r;
      store_n<T, V>(h + c, keep[0]);
    }
  }
  for (int c = p.W + tid; c < p.h_cols; c += nt) h[c] = from_f32<T>(0.f);
}

template <typename T, int V>
void launch_depth(const DepthParams& p, cudaStream_t s) {
  const int groups = (p.W + V - 1) / V;
  const int nt = std::min(256, (groups + 31) / 32 * 32);
  const int keep = (groups + nt - 1) / nt;
  const bool pdl = pdl_all_enabled();
#define TSB_DR(K) launch_pdl(depth_residual_kernel<T, V, K>, dim3(p.rows), dim3(nt), 0, s, pdl, p)
  if (keep == 1) TSB_DR(1);
  else if (keep == 2) TSB_DR(2);
  else if (keep <= 4) TSB_DR(4);
  else if (keep <= 8) TSB_DR(8);
  else TSB_DR(0);
#undef TSB_DR
}

}  // namespace
}  // namespace tsb

// See the head of this file. Exactly one of (x_in, y) and (tokens, table) is given; y, the table and h are bf16 (dtype 1) or
// fp32 (0). `avg` holds n_hist + 1 weights. When `h` is asked for, x has to be kept in x_out or stored.
TSB_EXPORT int tsb_depth_residual(const float* x_in, float* x_out, float* hist, long long hist_ld, const float* avg, int n_hist,
                                  int store, const void* y, long long ldy, float mult, const int* tokens, const void* table,
                                  long long ld_table, int vocab, void* h, long long ldh, int h_cols, int rows, int W, float gain,
                                  float eps, int dtype, void* stream) {
  using namespace tsb;
  const bool start = tokens && table;
  if (rows <= 0 || W <= 0 || (dtype != 0 && dtype != 1) || start == (x_in && y) || n_hist < 0 || ((avg || store) && !hist) ||
      (h && h_cols < W) || !(x_out || store))
    return -2;
  DepthParams p{x_in, x_out, hist, hist_ld, avg, n_hist, store, y, ldy, mult, start ? tokens : nullptr, table, ld_table, vocab, h, ldh,
                h_cols, rows, W, gain, eps, device_status_word()};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto off = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) != 0; };
  const long long ld_src = start ? ld_table : ldy;
  const bool vec = W % 4 == 0 && ld_src % 4 == 0 && !off(start ? table : y) && hist_ld % 4 == 0 && !off(hist) && !off(x_in) &&
                   !off(x_out) && (!h || (ldh % 4 == 0 && !off(h)));
  if (dtype == 1) {
    if (vec) launch_depth<__nv_bfloat16, 4>(p, s);
    else launch_depth<__nv_bfloat16, 1>(p, s);
  } else {
    if (vec) launch_depth<float, 4>(p, s);
    else launch_depth<float, 1>(p, s);
  }
  return static_cast<int>(cudaGetLastError());
}
