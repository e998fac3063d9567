// What attention kernels of ragged batches take besides q, k and v: the mask, what becomes of the scores, and what the result
// is multiplied with on its way out.
//
//   s = scale (q . k);  s = softcap tanh(s / softcap) (softcap > 0);  s -= slopes[h] (i - j) (slopes given)
//   p_j = exp(s_j) / (sum exp(s) + exp(sink[h]))  (sink given)
//   out = o * scale_out * sigmoid(gate)           (gate kind 1: one per head, 2: one per element)
#pragma once

#include "common.cuh"

namespace tsb {

constexpr float kLog2e = 1.4426950408889634f;

struct AttnForm {
  int chunk;               // > 0: token i sees the tokens j <= i of its own run of `chunk` positions
  int window;              // > 0: token i sees the tokens j with 0 <= i - j < window
  float scale, softcap;
  const float* slopes;     // [H] or null
  const float* sink;       // [H] or null

  __host__ __device__ bool plain() const { return window == 0 && softcap == 0.f && !slopes && !sink; }
  // first position that position `pos` sees
  __device__ __forceinline__ int first(int pos) const {
    return chunk > 0 ? pos / chunk * chunk : window > 0 ? max(0, pos - window + 1) : 0;
  }
};

struct AttnGate {
  int kind;
  const void* gate;        // [rows, ld]
  long long ld;
  float scale;
  long long ldo;           // elements between two rows of the result

  __host__ __device__ bool plain() const { return kind == 0 && scale == 1.f; }
  template <typename T>
  __device__ __forceinline__ float factor(long long row, int h, int D, int d) const {
    if (kind == 0) return scale;
    const T* g = static_cast<const T*>(gate) + row * ld;
    return scale / (1.f + expf(-to_f32<T>(g[kind == 1 ? h : h * D + d])));
  }
};

// ints: chunk, window, gate kind, gate row stride, result row stride; floats: scale, softcap, result scale; pointers: slopes, sink, gate.
inline bool read_attn_form(const long long* ints, const float* floats, const void* const* ptrs, AttnForm* f, AttnGate* g) {
  f->chunk = static_cast<int>(ints[0]); f->window = static_cast<int>(ints[1]);
  f->scale = floats[0]; f->softcap = floats[1];
  f->slopes = static_cast<const float*>(ptrs[0]); f->sink = static_cast<const float*>(ptrs[1]);
  g->kind = static_cast<int>(ints[2]); g->ld = ints[3]; g->ldo = ints[4]; g->scale = floats[2]; g->gate = ptrs[2];
  return f->chunk >= 0 && f->window >= 0 && !(f->chunk && f->window) && f->softcap >= 0.f && g->kind >= 0 && g->kind <= 2 &&
         (g->kind == 0 || g->gate);
}

// tanh to about 1e-7 absolute.
__device__ __forceinline__ float tanh_abs(float x) { return 1.f - __fdividef(2.f, 1.f + exp2f(2.f * kLog2e * x)); }

// The score in units of log 2, from the product and the distance i - j. `slope` is slopes[h] * log2 e.
struct ScoreLog2 {
  float mul, cap, slope;    // cap = 0: mul is scale * log2 e; else mul = scale / softcap and cap = softcap * log2 e
  __device__ __forceinline__ ScoreLog2(const AttnForm& f, int h) {
    mul = f.softcap > 0.f ? f.scale / f.softcap : f.scale * kLog2e;
    cap = f.softcap * kLog2e;
    slope = f.slopes ? f.slopes[h] * kLog2e : 0.f;
  }
  __device__ __forceinline__ float operator()(float qk, int distance) const {
    float s = qk * mul;
    if (cap > 0.f) s = cap * tanh_abs(s);
    return fmaf(-slope, static_cast<float>(distance), s);
  }
};

}  // namespace tsb
