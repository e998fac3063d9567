// Elementwise steps of blocks normed by Dynamic Tanh (tanh(alpha x) * w + b: no statistics, so nothing to reduce) and
// the clamped gated unit of their feed-forward.
//
// `tsb_dyn_tanh_residual` is everything between two matrix products of such a block in one pass over the row, with the
// residual stream in fp32:
//   x  = E[token] * scale                      (mode "set": start of the model)
//   x += norm_post(y + y_bias)                 (y: output of the sublayer before, bias of its projection folded in)
//   x += E[token] * scale                      (mode "add": a repeated pass gets the embedding again)
//   x += step                                  (vector of the pass)
//   h  = norm_next(x)                          (input of the next product, in its type, zero up to a padded width)
// each line optional. Per element 4 + 4 bytes of x, the y read and the h write: bound by memory.
#include "common.cuh"

#include <algorithm>

namespace tsb {
namespace {

struct DynTanhParams {
  float* x;
  int rows, W;
  const void* y;
  long long ldy;
  const float* y_bias;
  float post_alpha;
  const float* post_w;
  const float* post_b;
  const int* tokens;
  const void* table;
  long long ld_table;
  float scale;
  int embed_mode;      // 0: none, 1: set, 2: add
  int vocab;
  const float* step;
  float next_alpha;
  const float* next_w;
  const float* next_b;
  void* h;
  long long ldh;
  int h_cols;
  int* status;
};

template <typename T, int V>
__device__ __forceinline__ void load_v(const T* p, float (&f)[V]) {
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
__device__ __forceinline__ void store_v(T* p, const float (&f)[V]) {
  if constexpr (V == 1) {
    *p = from_f32<T>(f[0]);
  } else if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    uint2 a;
    T* e = reinterpret_cast<T*>(&a);
#pragma unroll
    for (int i = 0; i < 4; ++i) e[i] = from_f32<T>(f[i]);
    *reinterpret_cast<uint2*>(p) = a;
  }
}

// A thread keeps V columns (their norm weights stay in registers) and walks the rows; the loads of the next row are
// issued before the current one is computed.
template <typename T, int V>
__global__ void __launch_bounds__(256)
dyn_tanh_residual_kernel(DynTanhParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  const int stride = gridDim.y;
  if (c >= p.W) {
    if (p.h && c < p.h_cols) {
      const float z[V] = {};
      for (int r = blockIdx.y; r < p.rows; r += stride) store_v<T, V>(static_cast<T*>(p.h) + r * p.ldh + c, z);
    }
    return;
  }
  float yb[V] = {}, pw[V], pb[V], nw[V], nb[V], st[V] = {};
  if (p.y) {
    if (p.y_bias) load_v<float, V>(p.y_bias + c, yb);
    load_v<float, V>(p.post_w + c, pw);
    load_v<float, V>(p.post_b + c, pb);
  }
  if (p.step) load_v<float, V>(p.step + c, st);
  if (p.h) {
    load_v<float, V>(p.next_w + c, nw);
    load_v<float, V>(p.next_b + c, nb);
  }
  float xn[V] = {}, yn[V] = {}, en[V] = {};
  auto fetch = [&](int r) {
    if (p.embed_mode != 1) load_v<float, V>(p.x + static_cast<long long>(r) * p.W + c, xn);
    if (p.y) load_v<T, V>(static_cast<const T*>(p.y) + r * p.ldy + c, yn);
    if (p.embed_mode) {
      int tok = p.tokens[r];
      if (tok < 0 || tok >= p.vocab) {
        if (p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
        tok = 0;
      }
      load_v<T, V>(static_cast<const T*>(p.table) + tok * p.ld_table + c, en);
    }
  };
  int r = blockIdx.y;
  if (r < p.rows) fetch(r);
  for (; r < p.rows; r += stride) {
    float x[V], y[V], e[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      x[i] = xn[i];
      y[i] = yn[i];
      e[i] = en[i] * p.scale;
    }
    if (r + stride < p.rows) fetch(r + stride);
    float h[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      if (p.embed_mode == 1) x[i] = e[i];
      if (p.y) x[i] += fmaf(tanhf(p.post_alpha * (y[i] + yb[i])), pw[i], pb[i]);
      if (p.embed_mode == 2) x[i] += e[i];
      x[i] += st[i];
      if (p.h) h[i] = fmaf(tanhf(p.next_alpha * x[i]), nw[i], nb[i]);
    }
    store_v<float, V>(p.x + static_cast<long long>(r) * p.W + c, x);
    if (p.h) store_v<T, V>(static_cast<T*>(p.h) + r * p.ldh + c, h);
  }
}

// out[r, c] = g sigmoid(slope g) (u + 1), g = min(gate + bias, limit), u = clamp(up + bias, -limit, limit); gate and up
// are the two halves of a row.
template <typename T>
__global__ void __launch_bounds__(256)
clamped_glu_kernel(const T* gu, long long ldg, const float* bias, T* out, long long ldo, int rows, int F, float limit, float slope) {
  pdl_trigger();
  pdl_grid_wait();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (c >= F) return;
  float gb[4] = {}, ub[4] = {};
  if (bias) {
    load_v<float, 4>(bias + c, gb);
    load_v<float, 4>(bias + F + c, ub);
  }
  const int stride = gridDim.y;
  float gn[4], un[4];
  int r = blockIdx.y;
  if (r < rows) {
    load_v<T, 4>(gu + r * ldg + c, gn);
    load_v<T, 4>(gu + r * ldg + F + c, un);
  }
  for (; r < rows; r += stride) {
    float g[4], u[4], y[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      g[i] = gn[i] + gb[i];
      u[i] = un[i] + ub[i];
    }
    if (r + stride < rows) {
      load_v<T, 4>(gu + (r + stride) * ldg + c, gn);
      load_v<T, 4>(gu + (r + stride) * ldg + F + c, un);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float gg = fminf(g[i], limit), uu = fminf(fmaxf(u[i], -limit), limit);
      y[i] = gg / (1.f + expf(-slope * gg)) * (uu + 1.f);
    }
    store_v<T, 4>(out + r * ldo + c, y);
  }
}

dim3 row_grid(int cols, int v, int rows) {
  const int gx = (cols + 256 * v - 1) / (256 * v);
  int gy = (sm_count() * 8 + gx - 1) / gx;
  gy = std::min(gy, std::min(rows, 65535));
  return dim3(gx, gy);
}

}  // namespace
}  // namespace tsb

// See the head of this file. Null pointers switch a line off: y (with y_bias, post_*), step, h (with next_*);
// embed_mode 0 / 1 / 2 = none / set / add. x is fp32 [rows, W] (contiguous); y, the table and h are bf16 (dtype 1) or
// fp32 (dtype 0); norm weights, the bias and the step vector are fp32. h is written up to h_cols >= W (zeros past W).
TSB_EXPORT int tsb_dyn_tanh_residual(float* x, int rows, int W, const void* y, long long ldy, const float* y_bias,
                                     float post_alpha, const float* post_w, const float* post_b, const int* tokens,
                                     const void* table, long long ld_table, float scale, int embed_mode, int vocab,
                                     const float* step, float next_alpha, const float* next_w, const float* next_b, void* h,
                                     long long ldh, int h_cols, int dtype, void* stream) {
  using namespace tsb;
  if (!x || rows <= 0 || W <= 0 || (dtype != 0 && dtype != 1) || embed_mode < 0 || embed_mode > 2 ||
      (embed_mode && (!tokens || !table)) || (y && (!post_w || !post_b)) || (h && (!next_w || !next_b || h_cols < W)))
    return -2;
  DynTanhParams p{x, rows, W, y, ldy, y_bias, post_alpha, post_w, post_b, tokens, table, ld_table, scale, embed_mode, vocab,
                  step, next_alpha, next_w, next_b, h, ldh, h_cols, device_status_word()};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int cols = h ? std::max(W, h_cols) : W;
  const bool pdl = pdl_all_enabled();
  auto misaligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) != 0; };
  const bool vec = W % 4 == 0 && (!y || (ldy % 4 == 0 && !misaligned(y))) && (!embed_mode || (ld_table % 4 == 0 && !misaligned(table))) &&
                   (!h || (ldh % 4 == 0 && h_cols % 4 == 0 && !misaligned(h))) && !misaligned(x) && !misaligned(y_bias) &&
                   !misaligned(post_w) && !misaligned(post_b) && !misaligned(step) && !misaligned(next_w) && !misaligned(next_b);
  const dim3 grid = row_grid(cols, vec ? 4 : 1, rows);
  if (dtype == 1) {
    if (vec) launch_pdl(dyn_tanh_residual_kernel<__nv_bfloat16, 4>, grid, dim3(256), 0, s, pdl, p);
    else launch_pdl(dyn_tanh_residual_kernel<__nv_bfloat16, 1>, grid, dim3(256), 0, s, pdl, p);
  } else {
    if (vec) launch_pdl(dyn_tanh_residual_kernel<float, 4>, grid, dim3(256), 0, s, pdl, p);
    else launch_pdl(dyn_tanh_residual_kernel<float, 1>, grid, dim3(256), 0, s, pdl, p);
  }
  return static_cast<int>(cudaGetLastError());
}

// gate_up [rows, 2 F] (row stride ldg), bias fp32 [2 F] or null, out [rows, F] (row stride ldo); F and the strides are
// multiples of 4 and the bases 16-byte aligned.
TSB_EXPORT int tsb_clamped_glu(const void* gate_up, long long ldg, const float* bias, void* out, long long ldo, int rows, int F,
                               float limit, float slope, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || F <= 0 || F % 4 || ldg % 4 || ldo % 4 || (dtype != 0 && dtype != 1)) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid = row_grid(F, 4, rows);
  if (dtype == 1)
    launch_pdl(clamped_glu_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl_all_enabled(),
               static_cast<const __nv_bfloat16*>(gate_up), ldg, bias, static_cast<__nv_bfloat16*>(out), ldo, rows, F, limit, slope);
  else
    launch_pdl(clamped_glu_kernel<float>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const float*>(gate_up), ldg, bias,
               static_cast<float*>(out), ldo, rows, F, limit, slope);
  return static_cast<int>(cudaGetLastError());
}
