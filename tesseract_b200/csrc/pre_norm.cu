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
// A CTA walks kRows rows; a warp owns units of 32 V columns that lie inside one part, and keeps them in registers, also those of the
// row before. The row in front of the CTA's first is worked out once more (x is not updated in place, so it still can be). What the
// next step of a sequence needs of its last row goes to the slot at once for single tokens, and for portions to `tail`: another CTA
// may still have to read the slot. The next launch moves `tail` into the slots.
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
  float* last;              // [slots, W]
  float* tail;              // [prompts, W]
  const int *seq_of, *slots, *cu, *pos0;
  int n_decode;
  const float* moved;       // [n_moved, W]: what the launch before left in its tail
  float* moved_to;          // [slots, W]
  const int* moved_slots;
  int n_moved;
  void* h;                  // [rows, ldh]
  long long ldh;
  int h_cols, rows, W, blocks;
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

template <typename T, int V, int KEEP, bool SHIFT>
__global__ void __launch_bounds__(kMaxWarps * 32)
pre_norm_kernel(PreParams p, int rows_per) {
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ float red[];                       // two turns of a sum per unit
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = blockDim.x >> 5;
  if (static_cast<int>(blockIdx.x) >= p.blocks) {
    const int i = blockIdx.x - p.blocks, slot = p.moved_slots[i];
    if (slot < 0) return;
    for (int c = tid; c < p.W; c += blockDim.x) p.moved_to[static_cast<long long>(slot) * p.W + c] = p.moved[static_cast<long long>(i) * p.W + c];
    return;
  }
  const int gs = p.W / p.parts, pieces = (gs + 32 * V - 1) / (32 * V), units = p.parts * pieces;
  int col[KEEP], part[KEEP];                           // first column of this lane's share of a unit (-1: none)
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int u = warp + k * nw;
    part[k] = u / pieces;
    const int c = (u % pieces) * 32 * V + lane * V;
    col[k] = u < units && c < gs ? part[k] * gs + c : -1;
  }
  int turn = 0;
  // a -> a / rms of its part * w
  auto norm = [&](float (&a)[KEEP][V], const float* w) {
    float* r = red + (turn ^= 1) * units;
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      float ss = 0.f;
      if (col[k] >= 0) {
#pragma unroll
        for (int i = 0; i < V; ++i) ss = fmaf(a[k][i], a[k][i], ss);
      }
      ss = warp_sum(ss);
      if (lane == 0 && warp + k * nw < units) r[warp + k * nw] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      if (col[k] < 0) continue;
      float ss = 0.f, g[V];
      for (int j = 0; j < pieces; ++j) ss += r[part[k] * pieces + j];
      const float rs = 1.f / sqrtf(ss / static_cast<float>(gs) + p.eps);
      ld_v<float, V>(w + col[k], g);
#pragma unroll
      for (int i = 0; i < V; ++i) a[k][i] *= rs * g[i];
    }
  };
  // the normed row; `store`: x goes out
  auto work = [&](int row, bool store, float (&a)[KEEP][V]) {
    if (p.tokens) {
      int tok = p.tokens[row];
      if (tok < 0 || tok >= p.vocab) {
        if (tid == 0 && p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
        tok = 0;
      }
      const T* emb = static_cast<const T*>(p.table) + tok * p.ld_table;
      const float at = static_cast<float>(max(p.positions[row], 0));
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        if (col[k] < 0) continue;
        ld_v<T, V>(emb + col[k], a[k]);
        if (!p.freq) continue;
        if constexpr (V == 1) {
          const float2 sc = sin_cos(at, p.freq[col[k] >> 1]);
          a[k][0] += col[k] & 1 ? sc.y : sc.x;
        } else {
#pragma unroll
          for (int i = 0; i < V; i += 2) {
            const float2 sc = sin_cos(at, p.freq[(col[k] + i) >> 1]);
            a[k][i] += sc.x;
            a[k][i + 1] += sc.y;
          }
        }
      }
      if (p.embed_gain) norm(a, p.embed_gain);
    } else {
      const float* x = p.x + static_cast<long long>(row) * p.W;
      float b[KEEP][V];
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        if (col[k] < 0) continue;
        ld_v<float, V>(x + col[k], a[k]);
        if (p.y && !p.pos) ld_v<T, V>(static_cast<const T*>(p.y) + row * p.ldy + col[k], b[k]);
      }
      if (p.y && p.pos) {
#pragma unroll
        for (int k = 0; k < KEEP; ++k)
#pragma unroll
          for (int i = 0; i < V; ++i) b[k][i] = 0.f;
        for (int j = 0; j < p.top; ++j) {
          const long long at = static_cast<long long>(row) * p.top + j;
          const T* e = static_cast<const T*>(p.y) + p.pos[at] * p.ldy;
          const float w = p.weight[at];
#pragma unroll
          for (int k = 0; k < KEEP; ++k) {
            if (col[k] < 0) continue;
            float f[V];
            ld_v<T, V>(e + col[k], f);
#pragma unroll
            for (int i = 0; i < V; ++i) b[k][i] = fmaf(w, f[i], b[k][i]);
          }
        }
      }
      if (p.y) {
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
          if (col[k] < 0) continue;
          float f[V];
          if (p.bias) {
            ld_v<float, V>(p.bias + col[k], f);
#pragma unroll
            for (int i = 0; i < V; ++i) b[k][i] += f[i];
          }
          if (p.scale) {
            ld_v<float, V>(p.scale + col[k], f);
#pragma unroll
            for (int i = 0; i < V; ++i) a[k][i] = fmaf(b[k][i], f[i], a[k][i]);
          } else {
#pragma unroll
            for (int i = 0; i < V; ++i) a[k][i] += b[k][i];
          }
        }
      }
    }
    if (store && p.x_out) {
#pragma unroll
      for (int k = 0; k < KEEP; ++k)
        if (col[k] >= 0) st_v<float, V>(p.x_out + static_cast<long long>(row) * p.W + col[k], a[k]);
    }
    norm(a, p.gain);
  };
  float cur[KEEP][V], prev[SHIFT ? KEEP : 1][V];
  bool have = false;                                   // prev holds the row before
  for (int r = 0; r < rows_per; ++r) {
    const int row = blockIdx.x * rows_per + r;
    if (row >= p.rows) return;
    if constexpr (SHIFT) {
      const int seq = p.seq_of[row], slot = p.slots[seq];
      bool start = true, old = false, ends = false;
      if (row < p.n_decode) {
        old = p.positions[row] > 0;
      } else {
        const int i = seq - p.n_decode;
        start = row == p.n_decode + p.cu[i];
        ends = row + 1 == p.n_decode + p.cu[i + 1];
        old = p.pos0[i] > 0;
      }
      if (start) {
#pragma unroll
        for (int k = 0; k < KEEP; ++k) {
#pragma unroll
          for (int i = 0; i < V; ++i) prev[k][i] = 0.f;
          if (old && slot >= 0 && col[k] >= 0) ld_v<float, V>(p.last + static_cast<long long>(slot) * p.W + col[k], prev[k]);
        }
      } else if (!have) {
        work(row - 1, false, prev);
      }
      work(row, true, cur);
      have = true;
      float* keep = row < p.n_decode ? (slot >= 0 ? p.last + static_cast<long long>(slot) * p.W : nullptr)
                                     : (ends ? p.tail + static_cast<long long>(seq - p.n_decode) * p.W : nullptr);
      if (keep) {
#pragma unroll
        for (int k = 0; k < KEEP; ++k)
          if (col[k] >= 0) st_v<float, V>(keep + col[k], cur[k]);
      }
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        if (col[k] < 0) continue;
        float m[V], o[V];
        ld_v<float, V>(p.mu + col[k], m);
#pragma unroll
        for (int i = 0; i < V; ++i) {
          o[i] = fmaf(prev[k][i] - cur[k][i], m[i], cur[k][i]);
          prev[k][i] = cur[k][i];
        }
        st_v<T, V>(static_cast<T*>(p.h) + row * p.ldh + col[k], o);
      }
    } else {
      work(row, true, cur);
#pragma unroll
      for (int k = 0; k < KEEP; ++k)
        if (col[k] >= 0) st_v<T, V>(static_cast<T*>(p.h) + row * p.ldh + col[k], cur[k]);
    }
    for (int c = p.W + tid; c < p.h_cols; c += blockDim.x) static_cast<T*>(p.h)[row * p.ldh + c] = from_f32<T>(0.f);
  }
}

template <typename T, int V>
int launch_pre(PreParams& p, cudaStream_t s) {
  const int gs = p.W / p.parts, units = p.parts * ((gs + 32 * V - 1) / (32 * V));
  const int nw = std::min(kMaxWarps, std::max(1, (units + 1) / 2)), keep = (units + nw - 1) / nw;
  const int per = p.rows > 2048 ? 8 : 1;
  p.blocks = (p.rows + per - 1) / per;
  const dim3 grid(p.blocks + p.n_moved), block(nw * 32);
  const size_t smem = 2 * units * sizeof(float);
  if (keep > 8 || smem > 48 * 1024) return -2;
  const bool pdl = pdl_all_enabled();
#define TSB_PRE(K)                                                                              \
  do {                                                                                          \
    if (p.mu) launch_pdl(pre_norm_kernel<T, V, K, true>, grid, block, smem, s, pdl, p, per);    \
    else launch_pdl(pre_norm_kernel<T, V, K, false>, grid, block, smem, s, pdl, p, per);        \
  } while (0)
  if (keep == 1) TSB_PRE(1);
  else if (keep == 2) TSB_PRE(2);
  else if (keep <= 4) TSB_PRE(4);
  else TSB_PRE(8);
#undef TSB_PRE
  return static_cast<int>(cudaGetLastError());
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
  p.freq = static_cast<const float2*>(q[9]); p.embed_gain = f(10); p.positions = n(11); p.gain = f(12); p.mu = f(13); p.last = f(14);
  p.tail = f(15); p.seq_of = n(16); p.slots = n(17); p.cu = n(18); p.pos0 = n(19); p.moved = f(20); p.moved_to = f(21);
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
