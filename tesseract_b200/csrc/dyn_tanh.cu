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

// tanh within a few fp32 roundings: 1 - 2 / (exp(2 x) + 1), and its Taylor series where that would cancel (|x| < 1/4: the
// first dropped term is 1382 / 155925 x^11, below 1e-8 of x).
__device__ __forceinline__ float tanh_f32(float x) {
  const float z = x * x;
  const float series = fmaf(x * z, fmaf(z, fmaf(z, fmaf(z, 62.f / 2835.f, -17.f / 315.f), 2.f / 15.f), -1.f / 3.f), x);
  const float quotient = 1.f - __fdividef(2.f, __expf(2.f * x) + 1.f);
  return fabsf(x) < 0.25f ? series : quotient;
}

// V consecutive elements as stored, in registers.
template <typename T, int V>
struct alignas(V * sizeof(T)) Packed {
  T v[V];
};

// A thread keeps V columns (their norm weights stay in registers) and walks the rows, kRows at a time; the loads of the next
// rows are issued before the current ones are computed.
template <typename T, int V, int EMBED, bool HAS_Y>
__global__ void __launch_bounds__(256)
dyn_tanh_residual_kernel(DynTanhParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int kRows = 2;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  const int stride = gridDim.y * kRows;
  if (c >= p.W) {
    if (p.h && c < p.h_cols) {
      const float z[V] = {};
      for (int r = blockIdx.y; r < p.rows; r += gridDim.y) store_v<T, V>(static_cast<T*>(p.h) + r * p.ldh + c, z);
    }
    return;
  }
  float yb[V] = {}, pw[V], pb[V], nw[V], nb[V], st[V] = {};
  if constexpr (HAS_Y) {
    if (p.y_bias) load_v<float, V>(p.y_bias + c, yb);
    load_v<float, V>(p.post_w + c, pw);
    load_v<float, V>(p.post_b + c, pb);
  }
  if (p.step) load_v<float, V>(p.step + c, st);
  if (p.h) {
    load_v<float, V>(p.next_w + c, nw);
    load_v<float, V>(p.next_b + c, nb);
  }
  Packed<float, V> xn[kRows];
  Packed<T, V> yn[kRows], en[kRows];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int r = min(r0 + i, p.rows - 1);
      if constexpr (EMBED != 1) xn[i] = *reinterpret_cast<const Packed<float, V>*>(p.x + static_cast<long long>(r) * p.W + c);
      if constexpr (HAS_Y) yn[i] = *reinterpret_cast<const Packed<T, V>*>(static_cast<const T*>(p.y) + r * p.ldy + c);
      if constexpr (EMBED != 0) {
        int tok = p.tokens[r];
        if (tok < 0 || tok >= p.vocab) {
          if (p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
          tok = 0;
        }
        en[i] = *reinterpret_cast<const Packed<T, V>*>(static_cast<const T*>(p.table) + tok * p.ld_table + c);
      }
    }
  };
  int r0 = blockIdx.y * kRows;
  if (r0 < p.rows) fetch(r0);
  for (; r0 < p.rows; r0 += stride) {
    Packed<float, V> xc[kRows];
    Packed<T, V> yc[kRows], ec[kRows];
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      if constexpr (EMBED != 1) xc[i] = xn[i];
      if constexpr (HAS_Y) yc[i] = yn[i];
      if constexpr (EMBED != 0) ec[i] = en[i];
    }
    if (r0 + stride < p.rows) fetch(r0 + stride);
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int r = r0 + i;
      if (r >= p.rows) break;
      float x[V], h[V];
#pragma unroll
      for (int k = 0; k < V; ++k) {
        if constexpr (EMBED == 1) x[k] = to_f32<T>(ec[i].v[k]) * p.scale;
        else x[k] = xc[i].v[k];
        if constexpr (HAS_Y) x[k] += fmaf(tanh_f32(p.post_alpha * (to_f32<T>(yc[i].v[k]) + yb[k])), pw[k], pb[k]);
        if constexpr (EMBED == 2) x[k] = fmaf(to_f32<T>(ec[i].v[k]), p.scale, x[k]);
        x[k] += st[k];
        if (p.h) h[k] = fmaf(tanh_f32(p.next_alpha * x[k]), nw[k], nb[k]);
      }
      store_v<float, V>(p.x + static_cast<long long>(r) * p.W + c, x);
      if (p.h) store_v<T, V>(static_cast<T*>(p.h) + r * p.ldh + c, h);
    }
  }
}

template <typename T, int V>
void launch_residual(const DynTanhParams& p, dim3 grid, cudaStream_t s) {
  const bool pdl = pdl_all_enabled();
#define TSB_DT(E, Y) launch_pdl(dyn_tanh_residual_kernel<T, V, E, Y>, grid, dim3(256), 0, s, pdl, p)
  switch (p.embed_mode * 2 + (p.y ? 1 : 0)) {
    case 0: TSB_DT(0, false); break;
    case 1: TSB_DT(0, true); break;
    case 2: TSB_DT(1, false); break;
    case 3: TSB_DT(1, true); break;
    case 4: TSB_DT(2, false); break;
    default: TSB_DT(2, true); break;
  }
#undef TSB_DT
}

// out[r, c] = g sigmoid(slope g) (u + shift), g = min(scale * gate + bias, limit), u = clamp(scale * up + bias, -limit, limit);
// gate and up are the two halves of a row; sigmoid(slope (g + cubic g^3)) with a cubic. (limit = infinity, shift 0: SiLU(g) u for
// slope 1, the tanh form of GELU(g) u for slope 2 sqrt(2 / pi) and cubic 0.044715.)
template <typename T>
__global__ void __launch_bounds__(256)
clamped_glu_kernel(const T* gu, long long ldg, const float* bias, T* out, long long ldo, int rows, int F, float limit, float slope,
                   float shift, float scale, float cubic) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = 16 / sizeof(T);
  using Vec = Packed<T, V>;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (c >= F) return;
  float gb[V] = {}, ub[V] = {};
  if (bias) {
#pragma unroll
    for (int i = 0; i < V; ++i) {
      gb[i] = bias[c + i];
      ub[i] = bias[F + c + i];
    }
  }
  constexpr int kRows = 2;               // rows in flight next to the two being computed
  const int stride = gridDim.y * kRows;
  Vec gn[kRows], un[kRows];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const T* src = gu + min(r0 + i, rows - 1) * ldg + c;
      gn[i] = *reinterpret_cast<const Vec*>(src);
      un[i] = *reinterpret_cast<const Vec*>(src + F);
    }
  };
  int r0 = blockIdx.y * kRows;
  if (r0 < rows) fetch(r0);
  for (; r0 < rows; r0 += stride) {
    Vec g[kRows], u[kRows];
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      g[i] = gn[i];
      u[i] = un[i];
    }
    if (r0 + stride < rows) fetch(r0 + stride);
#pragma unroll
    for (int k = 0; k < kRows; ++k) {
      if (r0 + k >= rows) break;
      Vec y;
#pragma unroll
      for (int i = 0; i < V; ++i) {
        const float gg = fminf(fmaf(to_f32<T>(g[k].v[i]), scale, gb[i]), limit);
        const float uu = fminf(fmaxf(fmaf(to_f32<T>(u[k].v[i]), scale, ub[i]), -limit), limit);
        const float a = -slope * fmaf(cubic * gg * gg, gg, gg);
        const float q = sizeof(T) == 2 ? __fdividef(gg, 1.f + __expf(a)) : gg / (1.f + expf(a));
        y.v[i] = from_f32<T>(q * (uu + shift));
      }
      *reinterpret_cast<Vec*>(out + static_cast<long long>(r0 + k) * ldo + c) = y;
    }
  }
}

dim3 row_grid(int cols, int v, int rows) {
  const int gx = (cols + 256 * v - 1) / (256 * v);
  int gy = (sm_count() * 8 + gx - 1) / gx;
  gy = std::min(gy, std::min((rows + 1) / 2, 65535));
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
  auto misaligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) != 0; };
  const bool vec = W % 4 == 0 && (!y || (ldy % 4 == 0 && !misaligned(y))) && (!embed_mode || (ld_table % 4 == 0 && !misaligned(table))) &&
                   (!h || (ldh % 4 == 0 && h_cols % 4 == 0 && !misaligned(h))) && !misaligned(x) && !misaligned(y_bias) &&
                   !misaligned(post_w) && !misaligned(post_b) && !misaligned(step) && !misaligned(next_w) && !misaligned(next_b);
  const dim3 grid = row_grid(cols, vec ? 4 : 1, rows);
  if (dtype == 1) {
    if (vec) launch_residual<__nv_bfloat16, 4>(p, grid, s);
    else launch_residual<__nv_bfloat16, 1>(p, grid, s);
  } else {
    if (vec) launch_residual<float, 4>(p, grid, s);
    else launch_residual<float, 1>(p, grid, s);
  }
  return static_cast<int>(cudaGetLastError());
}

// gate_up [rows, 2 F] (row stride ldg), bias fp32 [2 F] or null, out [rows, F] (row stride ldo); F and the strides are
// multiples of 8 and the bases 16-byte aligned.
TSB_EXPORT int tsb_clamped_glu(const void* gate_up, long long ldg, const float* bias, void* out, long long ldo, int rows, int F,
                               float limit, float slope, float shift, float scale, float cubic, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || F <= 0 || F % 8 || ldg % 8 || ldo % 8 || (dtype != 0 && dtype != 1)) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid = row_grid(F, dtype == 1 ? 8 : 4, rows);
  if (dtype == 1)
    launch_pdl(clamped_glu_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl_all_enabled(),
               static_cast<const __nv_bfloat16*>(gate_up), ldg, bias, static_cast<__nv_bfloat16*>(out), ldo, rows, F, limit, slope,
               shift, scale, cubic);
  else
    launch_pdl(clamped_glu_kernel<float>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const float*>(gate_up), ldg, bias,
               static_cast<float*>(out), ldo, rows, F, limit, slope, shift, scale, cubic);
  return static_cast<int>(cudaGetLastError());
}
