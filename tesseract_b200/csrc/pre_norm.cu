// Residual step of blocks that norm what their sublayers read, with the token shift of the mixer's input.
//
//   x  = pnorm(E[token] + sinusoid(position)) * embed_gain     (start of the model)
//   x += scale * (y + bias)                                    (y: a sublayer's result, or the weighted sum of experts' rows;
//                                                               scale and bias per channel)
//   n  = pnorm(x) * gain
//   h  = n + (n' - n) * mu                                     (mu given; n' the n of the token before, zeros at the first)
//
// pnorm splits a row into equal parts, each over its own root mean square. Stream, norms and shift are fp32.
//
// A CTA takes a row; a warp owns units of 32 V columns that lie inside one part, and keeps them in registers. With a shift the row of the
// token before is worked out once more where it is part of the launch (x is not updated in place, so it still can be), which suits few
// rows; many are shifted by a pass of their own (token_shift_kernel). What the next step of a sequence needs of its last row goes to the
// slot at once for single tokens, and for portions to `tail`: another CTA may still have to read the slot. The next launch moves `tail`
// into the slots. n' is rounded to h's type wherever it comes from.
#include "warp_mma.cuh"

#include <algorithm>

namespace tsb {
namespace {

constexpr int kMaxWarps = 16;

struct PreParams {
  const float* x;           // [rows, W], or null at the start
  float* x_out;             // [rows, W]
  const void* y;            // [rows, ldy], or the experts' rows
  long long ldy;
  const int* pos;           // [rows, top] rows of y, or null
  const float* weight;      // [rows, top]
  int top;
  const float* bias;        // [W] or null
  const float* scale;       // [W] or null
  const int* tokens;        // start
  const void* table;
  long long ld_table;
  int vocab;
  const float2* freq;       // [ceil(W / 2)] angle per position in two parts, or null: no sinusoid
  const float* embed_gain;  // [W] or null: no norm of the start
  const int* positions;     // [rows]
  const float* gain;        // [W]
  int parts;
  float eps;
  const float* mu;          // [W] or null: no shift
  void* last;               // [slots, h_cols]
  void* tail;               // [prompts, h_cols]
  const int *seq_of, *slots, *cu, *pos0;
  int n_decode;
  const void* moved;        // [n_moved, h_cols]: what the launch before left in its tail
  void* moved_to;           // [slots, h_cols]
  const int* moved_slots;
  int n_moved;
  void* h;                  // [rows, ldh]
  long long ldh;
  int h_cols, rows, W;
  int* status;
};

template <typename T, int V>
__device__ __forceinline__ void ld_v(const T* p, float (&f)[V]) {
  if constexpr (V == 1) {
    f[0] = to_f32<T>(*p);
  } else if constexpr (sizeof(T) == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  } else {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const T* e = reinterpret_cast<const T*>(&a);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = to_f32<T>(e[i]);
  }
}
template <typename T, int V>
__device__ __forceinline__ void st_v(T* p, const float (&f)[V]) {
  if constexpr (V == 1) {
    *p = from_f32<T>(f[0]);
  } else if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  }
}

// sin and cos of p * (f.x + f.y): the product's rounding is carried along.
__device__ __forceinline__ float2 sin_cos(float p, float2 f) {
  const float a = p * f.x, e = fmaf(p, f.x, -a) + p * f.y;
  float s, c;
  sincosf(a, &s, &c);
  return make_float2(fmaf(c, e, s), fmaf(-s, e, c));
}

enum StepMode { kStart, kAdd, kMixed };      // where x comes from: the embedding, x + y, x + a weighted sum of rows

template <typename T, int V, int KEEP, int MODE, bool SHIFT>
__global__ void __launch_bounds__(kMaxWarps * 32)
pre_norm_kernel(PreParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int N = SHIFT ? 2 : 1;                     // rows held: the one before, then the CTA's own
  extern __shared__ float red[];                       // two turns of a sum per row and unit
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = blockDim.x >> 5, row = blockIdx.x;
  if (row >= p.rows) {
    const int i = row - p.rows, slot = p.moved_slots[i];
    if (slot < 0) return;
    const T* from = static_cast<const T*>(p.moved) + static_cast<long long>(i) * p.h_cols;
    T* to = static_cast<T*>(p.moved_to) + static_cast<long long>(slot) * p.h_cols;
    for (int c = tid; c < p.h_cols; c += blockDim.x) to[c] = from[c];
    return;
  }
  const int gs = p.W / p.parts, pieces = (gs + 32 * V - 1) / (32 * V), units = p.parts * pieces;
  int col[KEEP], part[KEEP];                           // first column of this lane's share of a unit (-1: none)
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int u = warp + k * nw;
    part[k] = u / pieces;
    const int c = (u - part[k] * pieces) * 32 * V + lane * V;
    col[k] = u < units && c < gs ? part[k] * gs + c : -1;
  }
  // (whether the row in front belongs to the sequence is only known later; its loads do not wait)
  const bool look_back = SHIFT && row > p.n_decode;
  auto used = [&](int n) { return n == N - 1 || look_back; };
  float a[N][KEEP][V];
  int turn = 0;
  // a -> a / rms of its part * w
  auto norm = [&](const float* w) {
    float* r = red + (turn ^= 1) * N * units;
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        float ss = 0.f;
        if (col[k] >= 0 && used(n)) {
#pragma unroll
          for (int i = 0; i < V; ++i) ss = fmaf(a[n][k][i], a[n][k][i], ss);
        }
        ss = warp_sum(ss);
        if (lane == 0 && warp + k * nw < units) r[n * units + warp + k * nw] = ss;
      }
    __syncthreads();
    float sums[N][KEEP];                               // of the parts that this warp's units lie in
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const float* z = r + n * units + min(part[k], p.parts - 1) * pieces;
        float ss = 0.f;
        if (pieces <= 2) {
          ss = z[0] + (pieces > 1 ? z[1] : 0.f);
        } else {
          for (int j = lane; j < pieces; j += 32) ss += z[j];
          ss = warp_sum(ss);
        }
        sums[n][k] = ss;
      }
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      if (col[k] < 0) continue;
      float g[V];
      ld_v<float, V>(w + col[k], g);
#pragma unroll
      for (int n = 0; n < N; ++n) {
        const float rs = 1.f / sqrtf(sums[n][k] / static_cast<float>(gs) + p.eps);
#pragma unroll
        for (int i = 0; i < V; ++i) a[n][k][i] *= rs * g[i];
      }
    }
  };
  if constexpr (MODE == kStart) {
#pragma unroll
    for (int n = 0; n < N; ++n) {
      if (!used(n)) continue;
      const int at = row - (N - 1) + n;
      int tok = p.tokens[at];
      if (tok < 0 || tok >= p.vocab) {
        if (tid == 0 && p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
        tok = 0;
      }
      const T* emb = static_cast<const T*>(p.table) + tok * p.ld_table;
      const float pos = static_cast<float>(max(p.positions[at], 0));
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        if (col[k] < 0) continue;
        ld_v<T, V>(emb + col[k], a[n][k]);
        if (!p.freq) continue;
        if constexpr (V == 1) {
          const float2 sc = sin_cos(pos, p.freq[col[k] >> 1]);
          a[n][k][0] += col[k] & 1 ? sc.y : sc.x;
        } else {
#pragma unroll
          for (int i = 0; i < V; i += 2) {
            const float2 sc = sin_cos(pos, p.freq[(col[k] + i) >> 1]);
            a[n][k][i] += sc.x;
            a[n][k][i + 1] += sc.y;
          }
        }
      }
    }
    if (p.embed_gain) norm(p.embed_gain);
  } else {
    float b[N][KEEP][V];
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const long long at = row - (N - 1) + n;
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
#pragma unroll
        for (int i = 0; i < V; ++i) b[n][k][i] = 0.f;
        if (col[k] < 0 || !used(n)) continue;
        ld_v<float, V>(p.x + at * p.W + col[k], a[n][k]);
        if (MODE == kAdd && p.y) ld_v<T, V>(static_cast<const T*>(p.y) + at * p.ldy + col[k], b[n][k]);
      }
    }
    if constexpr (MODE == kMixed) {
      for (int j = 0; j < p.top; ++j) {
#pragma unroll
        for (int n = 0; n < N; ++n) {
          if (!used(n)) continue;
          const long long i = static_cast<long long>(row - (N - 1) + n) * p.top + j;
          const T* e = static_cast<const T*>(p.y) + p.pos[i] * p.ldy;
          const float w = p.weight[i];
#pragma unroll
          for (int k = 0; k < KEEP; ++k) {
            if (col[k] < 0) continue;
            float f[V];
            ld_v<T, V>(e + col[k], f);
#pragma unroll
            for (int i = 0; i < V; ++i) b[n][k][i] = fmaf(w, f[i], b[n][k][i]);
          }
        }
      }
    }
    if (MODE == kMixed || p.y) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        if (col[k] < 0) continue;
        float bias[V], scale[V];
#pragma unroll
        for (int i = 0; i < V; ++i) {
          bias[i] = 0.f;
          scale[i] = 1.f;
        }
        if (p.bias) ld_v<float, V>(p.bias + col[k], bias);
        if (p.scale) ld_v<float, V>(p.scale + col[k], scale);
#pragma unroll
        for (int n = 0; n < N; ++n)
#pragma unroll
          for (int i = 0; i < V; ++i) a[n][k][i] = fmaf(b[n][k][i] + bias[i], scale[i], a[n][k][i]);
      }
    }
  }
  if (p.x_out) {
#pragma unroll
    for (int k = 0; k < KEEP; ++k)
      if (col[k] >= 0) st_v<float, V>(p.x_out + static_cast<long long>(row) * p.W + col[k], a[N - 1][k]);
  }
  bool joined = false;                                 // the row above is the token before
  const T* before = nullptr;                           // the token before is in a slot
  T* keep = nullptr;                                   // where the next step of the sequence finds this row
  if constexpr (SHIFT) {
    const int seq = p.seq_of[row], slot = p.slots[seq];
    T* mine = slot >= 0 ? static_cast<T*>(p.last) + static_cast<long long>(slot) * p.h_cols : nullptr;
    bool old;
    if (row < p.n_decode) {
      old = p.positions[row] > 0;
      keep = mine;
    } else {
      const int i = seq - p.n_decode;
      joined = row > p.n_decode + p.cu[i];
      if (row + 1 == p.n_decode + p.cu[i + 1]) keep = static_cast<T*>(p.tail) + static_cast<long long>(i) * p.h_cols;
      old = p.pos0[i] > 0;
    }
    if (!joined && old) before = mine;
  }
  norm(p.gain);
  T* h = static_cast<T*>(p.h) + row * p.ldh;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    if (col[k] < 0) continue;
    const float(&cur)[V] = a[N - 1][k];
    if constexpr (SHIFT) {
      float m[V], prev[V], o[V];
      ld_v<float, V>(p.mu + col[k], m);
#pragma unroll
      for (int i = 0; i < V; ++i) prev[i] = joined ? to_f32<T>(from_f32<T>(a[0][k][i])) : 0.f;
      if (before) ld_v<T, V>(before + col[k], prev);
#pragma unroll
      for (int i = 0; i < V; ++i) o[i] = fmaf(prev[i] - cur[i], m[i], cur[i]);
      st_v<T, V>(h + col[k], o);
      if (keep) st_v<T, V>(keep + col[k], cur);
    } else {
      st_v<T, V>(h + col[k], cur);
    }
  }
  for (int c = p.W + tid; c < p.h_cols; c += blockDim.x) {
    h[c] = from_f32<T>(0.f);
    if (keep) keep[c] = from_f32<T>(0.f);
  }
}

template <typename T, int V, int KEEP, int MODE>
int launch_mode(const PreParams& p, int nw, int units, cudaStream_t s) {
  const dim3 grid(p.rows + p.n_moved), block(nw * 32);
  const size_t smem = 4 * units * sizeof(float);
  if (p.mu) launch_pdl(pre_norm_kernel<T, V, KEEP, MODE, true>, grid, block, smem, s, pdl_all_enabled(), p);
  else launch_pdl(pre_norm_kernel<T, V, KEEP, MODE, false>, grid, block, smem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int V, int KEEP>
int launch_keep(const PreParams& p, int nw, int units, cudaStream_t s) {
  if (p.tokens) return launch_mode<T, V, KEEP, kStart>(p, nw, units, s);
  if (p.pos) return launch_mode<T, V, KEEP, kMixed>(p, nw, units, s);
  return launch_mode<T, V, KEEP, kAdd>(p, nw, units, s);
}

template <typename T, int V>
int launch_pre(const PreParams& p, cudaStream_t s) {
  const int gs = p.W / p.parts, units = p.parts * ((gs + 32 * V - 1) / (32 * V));
  const int nw = std::min(kMaxWarps, (units + 1) / 2), keep = (units + nw - 1) / nw;
  if (keep <= 2) return launch_keep<T, V, 2>(p, nw, units, s);
  if constexpr (V == 4)
    if (keep <= 4) return launch_keep<T, V, 4>(p, nw, units, s);
  return keep <= 8 ? launch_keep<T, V, 8>(p, nw, units, s) : -2;
}

}  // namespace
}  // namespace tsb

// See PreParams. ints: top, vocab, parts, n_decode, n_moved, h_cols, rows, W; lds: y, table, h; ptrs in the order of PreParams: x, x_out, y,
// pos, weight, bias, scale, tokens, table, freq, embed_gain, positions, gain, mu, last, tail, seq_of, slots, cu, pos0, moved, moved_to,
// moved_slots, h. y, the table and h are bf16 (dtype 1) or fp32 (0).
TSB_EXPORT int tsb_pre_norm_step(const int* v, const long long* ld, void* const* q, float eps, int dtype, void* stream) {
  using namespace tsb;
  PreParams p{};
  p.top = v[0]; p.vocab = v[1]; p.parts = v[2]; p.n_decode = v[3]; p.n_moved = v[4]; p.h_cols = v[5]; p.rows = v[6]; p.W = v[7];
  p.ldy = ld[0]; p.ld_table = ld[1]; p.ldh = ld[2]; p.eps = eps;
  auto f = [&](int i) { return static_cast<float*>(q[i]); };
  auto n = [&](int i) { return static_cast<const int*>(q[i]); };
  p.x = f(0); p.x_out = f(1); p.y = q[2]; p.pos = n(3); p.weight = f(4); p.bias = f(5); p.scale = f(6); p.tokens = n(7); p.table = q[8];
  p.freq = static_cast<const float2*>(q[9]); p.embed_gain = f(10); p.positions = n(11); p.gain = f(12); p.mu = f(13); p.last = q[14];
  p.tail = q[15]; p.seq_of = n(16); p.slots = n(17); p.cu = n(18); p.pos0 = n(19); p.moved = q[20]; p.moved_to = q[21];
  p.moved_slots = n(22); p.h = q[23];
  if (p.rows <= 0 || p.W <= 0 || p.parts <= 0 || p.W % p.parts || p.h_cols < p.W || !p.h || !p.gain || (dtype != 0 && dtype != 1) ||
      (p.tokens ? (!p.table || !p.x_out || !p.positions || p.y) : !p.x) || (p.y && !p.x_out) || p.x == p.x_out ||
      (p.pos && (!p.y || !p.weight || p.top <= 0)) || p.n_moved < 0 || (p.n_moved && (!p.moved || !p.moved_to || !p.moved_slots)) ||
      (p.mu && (!p.last || !p.seq_of || !p.slots || !p.positions || p.n_decode < 0 || p.n_decode > p.rows ||
                (p.n_decode < p.rows && (!p.tail || !p.cu || !p.pos0)))))
    return -2;
  p.status = device_status_word();
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto off = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) != 0; };
  const bool vec = (p.W / p.parts) % 4 == 0 && !off(p.x) && !off(p.x_out) && !off(p.y) && !off(p.bias) && !off(p.scale) && !off(p.table) &&
                   !off(p.embed_gain) && !off(p.gain) && !off(p.mu) && !off(p.last) && !off(p.tail) && !off(p.h) && p.ldy % 4 == 0 &&
                   p.ld_table % 4 == 0 && p.ldh % 4 == 0;
  if (dtype == 1) return vec ? launch_pre<__nv_bfloat16, 4>(p, s) : launch_pre<__nv_bfloat16, 1>(p, s);
  return vec ? launch_pre<float, 4>(p, s) : launch_pre<float, 1>(p, s);
}
