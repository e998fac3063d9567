// Residual step of blocks that norm what their sublayers return, and the side input per token.
//
//   x  = E[token] * scale                               (start of the model)
//   x += y / sqrt(mean(y^2) + eps) * gain               (y: a sublayer's result, gain per channel)
//   h  = x  or, behind the last layer, x / sqrt(mean(x^2) + eps) * final     (input of the next product, in its type)
//
// One CTA per row; y and x stay in registers between the sums and the stores. The stream and both norms are fp32.
#include "warp_mma.cuh"

#include <algorithm>

namespace tsb {
namespace {

struct PostParams {
  float* x;               // [rows, W]
  const void* y;          // [rows, ldy] or null
  long long ldy;
  const float* gain;      // [W]
  const float* final_gain;// [W] or null
  float eps;
  const int* tokens;      // or null
  const void* table;
  long long ld_table;
  int vocab;
  float scale;
  void* h;
  long long ldh;
  int h_cols, rows, W;
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
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  }
}

// Sum over the CTA; `red` has a place per warp and may be used again after the next barrier.
__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x) / 32; ++w) v += red[w];
  return v;
}

// KEEP groups of V columns per thread stay in registers; wider rows (KEEP = 0) are read again.
template <typename T, int V, int KEEP>
__global__ void __launch_bounds__(256)
post_norm_kernel(PostParams p) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ float red[2][8];
  constexpr int N = KEEP > 0 ? KEEP : 1;
  const int row = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  float* x = p.x + static_cast<long long>(row) * p.W;
  const T* y = p.y ? static_cast<const T*>(p.y) + row * p.ldy : nullptr;
  T* h = static_cast<T*>(p.h) + row * p.ldh;
  const T* emb = nullptr;
  if (p.tokens) {
    int tok = p.tokens[row];
    if (tok < 0 || tok >= p.vocab) {
      if (tid == 0 && p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
      tok = 0;
    }
    emb = static_cast<const T*>(p.table) + tok * p.ld_table;
  }
  float kx[N][V], ky[N][V];
  auto residual = [&](int c, float (&a)[V]) {
    if (emb) {
      load_v<T, V>(emb + c, a);
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] *= p.scale;
    } else {
      load_v<float, V>(x + c, a);
    }
  };
  float ss = 0.f, r = 0.f;
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = (k * nt + tid) * V;
      if (c >= p.W) break;
      residual(c, kx[k]);
      if (!y) continue;
      load_v<T, V>(y + c, ky[k]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(ky[k][i], ky[k][i], ss);
    }
  } else if (y) {
    for (int c = tid * V; c < p.W; c += nt * V) {
      load_v<T, V>(y + c, ky[0]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(ky[0][i], ky[0][i], ss);
    }
  }
  if (y) r = 1.f / sqrtf(cta_sum(ss, red[0]) / static_cast<float>(p.W) + p.eps);
  ss = 0.f;
  auto add = [&](int c, float (&a)[V], const float (&b)[V]) {
    if (y) {
      float g[V];
      load_v<float, V>(p.gain + c, g);
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] = fmaf(b[i] * r, g[i], a[i]);
    }
    if (y || emb) store_v<float, V>(x + c, a);
    if (!p.final_gain) store_v<T, V>(h + c, a);
#pragma unroll
    for (int i = 0; i < V; ++i) ss = fmaf(a[i], a[i], ss);
  };
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = (k * nt + tid) * V;
      if (c < p.W) add(c, kx[k], ky[k]);
    }
  } else {
    for (int c = tid * V; c < p.W; c += nt * V) {
      residual(c, kx[0]);
      if (y) load_v<T, V>(y + c, ky[0]);
      add(c, kx[0], ky[0]);
    }
  }
  if (p.final_gain) {
    r = 1.f / sqrtf(cta_sum(ss, red[1]) / static_cast<float>(p.W) + p.eps);
    auto out = [&](int c, float (&a)[V]) {
      float g[V];
      load_v<float, V>(p.final_gain + c, g);
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] = a[i] * r * g[i];
      store_v<T, V>(h + c, a);
    };
    if constexpr (KEEP > 0) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int c = (k * nt + tid) * V;
        if (c < p.W) out(c, kx[k]);
      }
    } else {
      for (int c = tid * V; c < p.W; c += nt * V) {
        load_v<float, V>(x + c, kx[0]);
        out(c, kx[0]);
      }
    }
  }
  for (int c = p.W + tid; c < p.h_cols; c += nt) h[c] = from_f32<T>(0.f);
}

template <typename T, int V>
void launch_post(const PostParams& p, cudaStream_t s) {
  const int groups = (p.W + V - 1) / V;
  const int nt = std::min(256, (groups + 31) / 32 * 32);
  const int keep = (groups + nt - 1) / nt;
  const bool pdl = pdl_all_enabled();
#define TSB_PN(K) launch_pdl(post_norm_kernel<T, V, K>, dim3(p.rows), dim3(nt), 0, s, pdl, p)
  if (keep == 1) TSB_PN(1);
  else if (keep == 2) TSB_PN(2);
  else if (keep <= 4) TSB_PN(4);
  else if (keep <= 8) TSB_PN(8);
  else TSB_PN(0);
#undef TSB_PN
}

__device__ __forceinline__ float gelu_tanh_f32(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// out[row, c] = gelu(g[row, c]) * table[token, first + c] for c < dim, zero up to out_cols.
template <typename T>
__global__ void __launch_bounds__(256)
gelu_lookup_kernel(const T* g, long long ldg, const int* tokens, const T* table, long long ld_table, int vocab, int first, T* out,
                   long long ldo, int out_cols, int rows, int dim, int* status) {
  pdl_trigger();
  pdl_grid_wait();
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  const long long row = i / out_cols;
  const int c = static_cast<int>(i % out_cols);
  if (row >= rows) return;
  float v = 0.f;
  if (c < dim) {
    int tok = tokens[row];
    if (tok < 0 || tok >= vocab) {
      if (status) atomicCAS(status, kStatusOk, kStatusBadIndex);
      tok = 0;
    }
    v = gelu_tanh_f32(to_f32<T>(g[row * ldg + c])) * to_f32<T>(table[tok * ld_table + first + c]);
  }
  out[row * ldo + c] = from_f32<T>(v);
}

}  // namespace
}  // namespace tsb

// See the head of this file. y, the table and h are bf16 (dtype 1) or fp32 (0).
TSB_EXPORT int tsb_post_norm_step(float* x, const void* y, long long ldy, const float* gain, const float* final_gain, float eps,
                                  const int* tokens, const void* table, long long ld_table, int vocab, float scale, void* h,
                                  long long ldh, int h_cols, int rows, int W, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || W <= 0 || !x || !h || h_cols < W || (y && !gain) || (tokens && !table) || (dtype != 0 && dtype != 1)) return -2;
  PostParams p{x, y, ldy, gain, final_gain, eps, tokens, table, ld_table, vocab, scale, h, ldh, h_cols, rows, W, device_status_word()};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto off = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) != 0; };
  const bool vec = W % 4 == 0 && !off(x) && !off(h) && ldh % 4 == 0 && (!y || (!off(y) && ldy % 4 == 0 && !off(gain))) &&
                   (!tokens || (!off(table) && ld_table % 4 == 0)) && !off(final_gain);
  if (dtype == 1) {
    if (vec) launch_post<__nv_bfloat16, 4>(p, s);
    else launch_post<__nv_bfloat16, 1>(p, s);
  } else {
    if (vec) launch_post<float, 4>(p, s);
    else launch_post<float, 1>(p, s);
  }
  return static_cast<int>(cudaGetLastError());
}

TSB_EXPORT int tsb_gelu_lookup(const void* g, long long ldg, const int* tokens, const void* table, long long ld_table, int vocab, int first,
                               void* out, long long ldo, int out_cols, int rows, int dim, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || dim <= 0 || out_cols < dim || first < 0 || first + dim > ld_table || (dtype != 0 && dtype != 1)) return -2;
  const long long n = static_cast<long long>(rows) * out_cols;
  const dim3 grid(static_cast<unsigned>((n + 255) / 256));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1)
    launch_pdl(gelu_lookup_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const __nv_bfloat16*>(g), ldg, tokens,
               static_cast<const __nv_bfloat16*>(table), ld_table, vocab, first, static_cast<__nv_bfloat16*>(out), ldo, out_cols, rows, dim,
               device_status_word());
  else
    launch_pdl(gelu_lookup_kernel<float>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const float*>(g), ldg, tokens,
               static_cast<const float*>(table), ld_table, vocab, first, static_cast<float*>(out), ldo, out_cols, rows, dim,
               device_status_word());
  return static_cast<int>(cudaGetLastError());
}
