// Gated delta rule (linear attention with a decaying, error-correcting state), for ragged batches of sequences.
//
// Per value head, with a state S [dim, vdim] in fp32:
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// q, k, v are short causal convolutions (per channel, then SiLU) of a packed projection; q and k are unit vectors per
// key head (q also times dim^-1/2); g = exp(-exp(A_log) softplus(a + dt_bias)), one per head or, where the caller brings
// `dec`, one per head and row of S (key channel); beta = sigmoid(b); the read-out is divided by its root mean square over
// vdim, scaled by a weight and by SiLU or sigmoid of a gate.
//
// Prompt rows take four launches: `delta_prepare_kernel` (convolution, unit vectors, gates; every token in parallel),
// `conv_state_kernel` (the convolution's tail of each sequence goes to its slot), `delta_scan_kernel` (the
// recurrence) and `delta_gate_norm_kernel`. Decoded rows take one: `delta_step_kernel` does all of it for one token,
// streaming the state through registers once.
//
// The columns of S do not talk to each other, so the recurrence is split over value columns. In the scan eight lanes
// share a column (each holds dim / 8 rows of it in registers), and four tokens are taken at once: the products of the
// state with their k and q are formed from the state before the block, the tokens' influence on one another is a 4 x 4
// triangle of scalars that the prepare kernel has computed, and the state is updated once. That is 3.25 multiply-adds
// per element and token instead of 4, and one reduction latency per four tokens; they are issued on register pairs
// (fma.rn.f32x2). With a decay per channel the products of the decays inside a block are folded into the k and q that meet
// the old state and into the k that the update writes, so that the same scan runs on three vectors per token and value head
// instead of two per token and key head. The one-token kernel uses the same identity: S_new^T q = g (S_old^T q) + (k . q) u, so the state is
// read once. Everything of the recurrence is fp32; nothing here uses the tensor cores.
//
// Packed projection row (element offsets, sections padded to multiples of 8):
//   [ q: Hk * dim | k: Hk * dim | v: H * vdim | .. b: H .. | .. a: H (without dec) .. ]
// A slot's convolution state holds the last taps - 1 rows of the first three sections, in the projection's type.
#include "ragged_conv.cuh"

#include <algorithm>
#include <cstdlib>
#include <type_traits>

namespace tsb {
namespace {

struct DeltaGeom {
  int Hk, H, dim, vdim;      // key heads, value heads, row and column extent of a head's state
  int dkp, vp;               // padded extents of the fp32 operands: dkp in {32, 64, 128, 256}, vp = vdim rounded up to 4
  int off_k, off_v, off_b, off_a;   // section offsets in a projection row (q starts at 0)
  int conv_c;                // columns of the convolved sections (q | k | v with their padding)
  long long ldp;             // projection row stride
};

// What the projection row does not hold: gates [rows, ld_gate] (kind 0: SiLU, 1: sigmoid), inputs of the decays [rows, ld_dec] (fp32,
// H * dim; null: one decay per head, from the row).
struct DeltaSide {
  const void* gate;
  long long ld_gate;
  int gate_kind;
  const float* dec;
  long long ld_dec;
};

constexpr int kBlk = 4;          // tokens the recurrence takes at once
constexpr int kCoef = 36;        // coefficients per (block, value head), see delta_prepare_kernel

template <bool FAST = false>
__device__ __forceinline__ float silu_f(float x) {
  if constexpr (FAST) return __fdividef(x, 1.f + __expf(-x));
  return x / (1.f + expf(-x));
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
// exp(-rate softplus(x)); the short form has 5e-6 of the softplus.
template <bool FAST = false>
__device__ __forceinline__ float decay_f(float x, float rate) {
  if constexpr (!FAST) return expf(-rate * softplus_f(x));
  const float e = __expf(-fabsf(x));
  const float l = e < 0.0625f ? e * (1.f - e * (0.5f - e * (0.33333333f - 0.25f * e))) : __logf(1.f + e);
  return __expf(-rate * (fmaxf(x, 0.f) + l));
}
template <bool FAST = false>
__device__ __forceinline__ float gate_f(float x, int kind) {
  if (kind == 0) return silu_f<FAST>(x);
  return FAST ? __fdividef(1.f, 1.f + __expf(-x)) : sigmoid_f(x);
}

// Sums of 16 values over the warp: lane l returns the sum of v[l % 16].
__device__ __forceinline__ float sums_of_16(float (&v)[16], int lane) {
#pragma unroll
  for (int o = 8; o; o >>= 1) {
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (i >= o) break;
      const float keep = up ? v[i + o] : v[i], give = up ? v[i] : v[i + o];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 16);
}

// N consecutive channels starting at p, of which `valid` exist; vector loads when the caller knows p to be aligned.
template <typename T, int N>
__device__ __forceinline__ void load_ch(const T* p, int valid, bool vec, float (&f)[N]) {
  if (vec && valid >= N) {
    constexpr int kBytes = N * sizeof(T);
    if constexpr (kBytes == 2) {
      f[0] = to_f32<T>(p[0]);
    } else if constexpr (kBytes == 4) {
      const uint32_t r = *reinterpret_cast<const uint32_t*>(p);
#pragma unroll
      for (int i = 0; i < N; ++i) f[i] = to_f32<T>(reinterpret_cast<const T*>(&r)[i]);
    } else if constexpr (kBytes == 8) {
      const uint2 r = *reinterpret_cast<const uint2*>(p);
#pragma unroll
      for (int i = 0; i < N; ++i) f[i] = to_f32<T>(reinterpret_cast<const T*>(&r)[i]);
    } else {
#pragma unroll
      for (int v = 0; v < kBytes / 16; ++v) {
        const uint4 r = reinterpret_cast<const uint4*>(p)[v];
        constexpr int kPer = 16 / sizeof(T);
#pragma unroll
        for (int i = 0; i < kPer; ++i) f[v * kPer + i] = to_f32<T>(reinterpret_cast<const T*>(&r)[i]);
      }
    }
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = i < valid ? to_f32<T>(p[i]) : 0.f;
  }
}
template <int N>
__device__ __forceinline__ void store_f32(float* p, int valid, bool vec, const float (&f)[N]) {
  if (vec && valid >= N && N % 4 == 0) {
#pragma unroll
    for (int v = 0; v < N / 4; ++v) reinterpret_cast<float4*>(p)[v] = make_float4(f[4 * v], f[4 * v + 1], f[4 * v + 2], f[4 * v + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (i < valid) p[i] = f[i];
  }
}

// ------------------------------------------------------------------ prompt rows: convolution, unit vectors, gates
struct DeltaPrepParams {
  DeltaGeom g;
  const void* proj;          // [rows, ldp]
  const float* conv_w;       // [taps, conv_c]
  const float* a_log;        // [H]
  const float* dt_bias;      // [H] or, with dec, [H * dim]
  const float* dec;          // [rows, ld_dec] or null
  long long ld_dec;
  const void* conv_state;    // [slots, taps - 1, conv_c]
  const int* cu;             // [nseq + 1] row offsets of the sequences
  const int* slots;          // [nseq]
  const int* pos0;           // [nseq] position of the first row (0: the sequence starts here)
  const int* blk_seq;        // [blocks] sequence of a block of kBlk tokens
  const int* blk0;           // [nseq + 1] first block of a sequence
  float* kq;                 // [rows, Hk, 2, dkp]: k, then q; with dec [rows, H, 3, dkp], see delta_prepare_kernel
  float* g4;                 // with dec: [blocks, H, dkp] the decays of a whole block
  float* v;                  // [rows, H, vp]
  float* coef;               // [blocks, H, kCoef]
  int blocks;
};

// N consecutive channels as stored, in registers.
template <typename T, int N>
struct alignas(N * sizeof(T) >= 16 ? 16 : N * sizeof(T)) Packed {
  T v[N];
};

// Convolution and SiLU of N channels of a block's tokens. Every input row is requested before the first is used; rows
// past the end of the portion repeat its last one (their results are dropped).
template <typename T, int TAPS, int N>
__device__ __forceinline__ void conv_block(const DeltaPrepParams& p, int row0, int first, int cnt, long long state_row,
                                           bool has_state, int c, int valid, bool vec, float (&y)[kBlk][N]) {
  constexpr int R = TAPS - 1 + kBlk;
  Packed<T, N> x[R];
  const bool whole = vec && valid >= N;
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int t = min(first + r - (TAPS - 1), first + cnt - 1);      // token of this portion, negative: before it
    const T* src = t >= 0 ? static_cast<const T*>(p.proj) + static_cast<long long>(row0 + t) * p.g.ldp + c
                          : static_cast<const T*>(p.conv_state) + (state_row + (TAPS - 1) + t) * p.g.conv_c + c;
    const bool there = t >= 0 || has_state;
#pragma unroll
    for (int i = 0; i < N; ++i) x[r].v[i] = from_f32<T>(0.f);
    if (whole) {
      if (there) x[r] = *reinterpret_cast<const Packed<T, N>*>(src);
    } else {
#pragma unroll
      for (int i = 0; i < N; ++i)
        if (there && i < valid) x[r].v[i] = src[i];
    }
  }
  float w[TAPS][N];
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
    load_ch<float, N>(p.conv_w + static_cast<long long>(j) * p.g.conv_c + c, valid, vec, w[j]);
#pragma unroll
  for (int t = 0; t < kBlk; ++t)
#pragma unroll
    for (int i = 0; i < N; ++i) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j][i], to_f32<T>(x[t + j].v[i]), acc);
      y[t][i] = t < cnt ? silu_f<sizeof(T) == 2>(acc) : 0.f;
    }
}

// One warp per (block of kBlk tokens, unit). Units: the Hk key heads (q and k of the head, and the coefficients of its
// value heads), then blocks of 256 value channels. EPL = dkp / 32 channels of a key head per lane.
//
// Taking tokens 0 .. 3 of a block at once, with d_j = S^T k_j and e_j = S^T q_j formed from the state before the block:
//   u_j = beta_j (v_j - G_j d_j - sum_{i < j} A_ji u_i),  o_j = G_j e_j + sum_{i <= j} W_ji u_i,
//   S <- G_3 S + sum_j c_j k_j u_j^T,
//   G_j = g_0 .. g_j,  c_j = g_{j+1} .. g_3,  A_ji = (g_{i+1} .. g_j)(k_i . k_j),  W_ji = (g_{i+1} .. g_j)(k_i . q_j).
// Coefficients as stored: G (4), beta (4), A (10, 20, 21, 30, 31, 32, 0, 0), c (4), W (4 rows of 4, zero above the
// diagonal). Tokens past the end of the portion get g = 1, beta = 0, k = q = 0: they change nothing.
//
// CH (a decay per channel): G_j, c_j and the factors in A and W are vectors over the channels. A and W sum them in; G_j goes into
// the k and q that meet the old state, c_j into the k of the update (kq: k_j G_j, q_j G_j, k_j c_j per value head; the
// coefficients G and c are 1), and G_3 is kept as it is. All are products of factors up to 1, never quotients.
template <typename T, int TAPS, int EPL, bool CH>
__global__ void __launch_bounds__(128, TAPS <= 4 && EPL <= 4 ? 5 : 1)
delta_prepare_kernel(DeltaPrepParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int blk = blockIdx.y * 4 + warp;
  if (blk >= p.blocks) return;
  const DeltaGeom& g = p.g;
  const int seq = p.blk_seq[blk];
  const int row0 = p.cu[seq], n = p.cu[seq + 1] - row0;
  const int first = (blk - p.blk0[seq]) * kBlk;
  const int cnt = min(kBlk, n - first);
  const bool has_state = p.pos0[seq] > 0;
  const long long state_row = static_cast<long long>(p.slots[seq]) * (TAPS - 1);
  const int unit = blockIdx.x;
  if (unit < g.Hk) {
    const int d0 = lane * EPL;
    const int valid = min(EPL, g.dim - d0);
    const bool vec = g.dim % EPL == 0;
    float qv[kBlk][EPL], kv[kBlk][EPL];
    float gd[CH ? kBlk : 1][EPL];                  // CH: the inputs of a head's decays, requested ahead of the convolution
    auto fetch = [&](int h) {                      // (rows past the end repeat the last one until they are replaced)
#pragma unroll
      for (int t = 0; t < (CH ? kBlk : 0); ++t)
        load_ch<float, EPL>(p.dec + static_cast<long long>(row0 + first + min(t, cnt - 1)) * p.ld_dec + h * g.dim + d0, valid, vec, gd[t]);
    };
    if constexpr (CH) fetch(unit * (g.H / g.Hk));
    conv_block<T, TAPS, EPL>(p, row0, first, cnt, state_row, has_state, unit * g.dim + d0, valid, vec, qv);
    conv_block<T, TAPS, EPL>(p, row0, first, cnt, state_row, has_state, g.off_k + unit * g.dim + d0, valid, vec, kv);
    const float rsqrt_dim = rsqrtf(static_cast<float>(g.dim));
    const int per = g.H / g.Hk;
    const T* proj = static_cast<const T*>(p.proj);
    float* out = p.kq + (static_cast<long long>(row0 + first) * g.Hk + unit) * 2 * g.dkp + d0;
#pragma unroll
    for (int t = 0; t < kBlk; ++t) {
      float sq = 0.f, sk = 0.f;
#pragma unroll
      for (int i = 0; i < EPL; ++i) {
        sq = fmaf(qv[t][i], qv[t][i], sq);
        sk = fmaf(kv[t][i], kv[t][i], sk);
      }
      const float rq = rsqrtf(warp_sum(sq) + 1e-6f) * rsqrt_dim;
      const float rk = rsqrtf(warp_sum(sk) + 1e-6f);
#pragma unroll
      for (int i = 0; i < EPL; ++i) {
        qv[t][i] *= rq;
        kv[t][i] *= rk;
      }
      if (!CH && t < cnt) {
        float* o = out + static_cast<long long>(t) * g.Hk * 2 * g.dkp;
        store_f32<EPL>(o, EPL, true, kv[t]);
        store_f32<EPL>(o + g.dkp, EPL, true, qv[t]);
      }
    }
    if constexpr (CH) {
      for (int hh = 0; hh < per; ++hh) {
        const int h = unit * per + hh;
        if (hh > 0) fetch(h);
        float bias[EPL];
        load_ch<float, EPL>(p.dt_bias + h * g.dim + d0, valid, vec, bias);
        const float rate = expf(p.a_log[h]);
#pragma unroll
        for (int t = 0; t < kBlk; ++t)
#pragma unroll
          for (int e = 0; e < EPL; ++e) gd[t][e] = t < cnt && e < valid ? decay_f<sizeof(T) == 2>(gd[t][e] + bias[e], rate) : 1.f;
        float s[16];                               // A 10, 20, 21, 30, 31, 32, then W 00, 10, 11, 20, .. 33
#pragma unroll
        for (int i = 0; i < 16; ++i) s[i] = 0.f;
#pragma unroll
        for (int i = 0; i < kBlk; ++i) {           // k_i, decayed further and further
          float kd[EPL];
#pragma unroll
          for (int e = 0; e < EPL; ++e) kd[e] = kv[i][e];
#pragma unroll
          for (int j = i; j < kBlk; ++j) {
#pragma unroll
            for (int e = 0; e < EPL; ++e) {
              if (j > i) {
                kd[e] *= gd[j][e];
                s[j * (j - 1) / 2 + i] = fmaf(kd[e], kv[j][e], s[j * (j - 1) / 2 + i]);
              }
              s[6 + j * (j + 1) / 2 + i] = fmaf(kd[e], qv[j][e], s[6 + j * (j + 1) / 2 + i]);
            }
          }
          if (i < cnt) store_f32<EPL>(p.kq + ((static_cast<long long>(row0 + first + i) * g.H + h) * 3 + 2) * g.dkp + d0, EPL, true, kd);
        }
        float G[EPL];
#pragma unroll
        for (int e = 0; e < EPL; ++e) G[e] = 1.f;
#pragma unroll
        for (int t = 0; t < kBlk; ++t) {
          float a[EPL], b[EPL];
#pragma unroll
          for (int e = 0; e < EPL; ++e) {
            G[e] *= gd[t][e];
            a[e] = kv[t][e] * G[e];
            b[e] = qv[t][e] * G[e];
          }
          if (t < cnt) {
            float* o = p.kq + (static_cast<long long>(row0 + first + t) * g.H + h) * 3 * g.dkp + d0;
            store_f32<EPL>(o, EPL, true, a);
            store_f32<EPL>(o + g.dkp, EPL, true, b);
          }
        }
        store_f32<EPL>(p.g4 + (static_cast<long long>(blk) * g.H + h) * g.dkp + d0, EPL, true, G);
        const float sum = sums_of_16(s, lane);
        // coefficients `lane` and, of the last row of W, 32 + lane
        const int wr = (lane - 20) >> 2, wi = (lane - 20) & 3;
        const int src = lane >= 20 ? 6 + wr * (wr + 1) / 2 + wi : lane - 8;
        const float mine = __shfl_sync(0xffffffffu, sum, src & 15), tail = __shfl_sync(0xffffffffu, sum, (12 + lane) & 15);
        float c = 0.f;
        if (lane < 4 || (lane >= 16 && lane < 20)) c = 1.f;
        else if (lane < 8) c = lane - 4 < cnt ? sigmoid_f(to_f32<T>(proj[static_cast<long long>(row0 + first + lane - 4) * g.ldp + g.off_b + h])) : 0.f;
        else if (lane < 14 || (lane >= 20 && wi <= wr)) c = mine;
        float* co = p.coef + (static_cast<long long>(blk) * g.H + h) * kCoef;
        co[lane] = c;
        if (lane < 4) co[32 + lane] = tail;
      }
    } else {
      float kk[kBlk][kBlk], kqd[kBlk][kBlk];          // [j][i]: k_i . k_j (i < j) and k_i . q_j (i <= j)
#pragma unroll
      for (int j = 0; j < kBlk; ++j)
#pragma unroll
        for (int i = 0; i < kBlk; ++i) {
          kk[j][i] = kqd[j][i] = 0.f;
          if (i <= j) {
            float a = 0.f, b = 0.f;
#pragma unroll
            for (int e = 0; e < EPL; ++e) {
              a = fmaf(kv[i][e], kv[j][e], a);
              b = fmaf(kv[i][e], qv[j][e], b);
            }
            if (i < j) kk[j][i] = warp_sum(a);
            kqd[j][i] = warp_sum(b);
          }
        }
      // eight heads at a time: lane = token * 8 + head works out one pair of gates, then lanes 0 .. 7 collect their head's
      for (int h0 = 0; h0 < per; h0 += 8) {
        const int hh = h0 + (lane & 7), tok = lane >> 3;
        const int h = unit * per + min(hh, per - 1);
        float gate = 1.f, beta = 0.f;
        if (tok < cnt) {
          const T* pr = proj + static_cast<long long>(row0 + first + tok) * g.ldp;
          gate = expf(-expf(p.a_log[h]) * softplus_f(to_f32<T>(pr[g.off_a + h]) + p.dt_bias[h]));
          beta = sigmoid_f(to_f32<T>(pr[g.off_b + h]));
        }
        float gd[kBlk], be[kBlk];
#pragma unroll
        for (int t = 0; t < kBlk; ++t) {
          gd[t] = __shfl_sync(0xffffffffu, gate, t * 8 + (lane & 7));
          be[t] = __shfl_sync(0xffffffffu, beta, t * 8 + (lane & 7));
        }
        if (lane >= 8 || hh >= per) continue;
        float4* o = reinterpret_cast<float4*>(p.coef + (static_cast<long long>(blk) * g.H + h) * kCoef);
        const float g10 = gd[1], g21 = gd[2], g32 = gd[3], g20 = g10 * g21, g31 = g21 * g32, g30 = g20 * g32;
        o[0] = make_float4(gd[0], gd[0] * g10, gd[0] * g20, gd[0] * g30);
        o[1] = make_float4(be[0], be[1], be[2], be[3]);
        o[2] = make_float4(g10 * kk[1][0], g20 * kk[2][0], g21 * kk[2][1], g30 * kk[3][0]);
        o[3] = make_float4(g31 * kk[3][1], g32 * kk[3][2], 0.f, 0.f);
        o[4] = make_float4(g30, g31, g32, 1.f);
        o[5] = make_float4(kqd[0][0], 0.f, 0.f, 0.f);
        o[6] = make_float4(g10 * kqd[1][0], kqd[1][1], 0.f, 0.f);
        o[7] = make_float4(g20 * kqd[2][0], g21 * kqd[2][1], kqd[2][2], 0.f);
        o[8] = make_float4(g30 * kqd[3][0], g31 * kqd[3][1], g32 * kqd[3][2], kqd[3][3]);
      }
    }
  } else {
    const int c = (unit - g.Hk) * 256 + lane * 8, total = g.H * g.vdim;
    if (c >= total) return;
    const int valid = min(8, total - c);
    float y[kBlk][8];
    conv_block<T, TAPS, 8>(p, row0, first, cnt, state_row, has_state, g.off_v + c, valid, true, y);
#pragma unroll
    for (int t = 0; t < kBlk; ++t) {
      if (t >= cnt) break;
      float* vr = p.v + static_cast<long long>(row0 + first + t) * g.H * g.vp;
      if (g.vp == g.vdim) {
        store_f32<8>(vr + c, valid, true, y[t]);
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i)
          if (i < valid) vr[static_cast<long long>((c + i) / g.vdim) * g.vp + (c + i) % g.vdim] = y[t][i];
      }
    }
  }
}

// ------------------------------------------------------------------ prompt rows: the recurrence
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(reinterpret_cast<unsigned long long&>(d))
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)),
        "l"(reinterpret_cast<unsigned long long&>(c)));
  return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 d;
  asm("mul.rn.f32x2 %0, %1, %2;"
      : "=l"(reinterpret_cast<unsigned long long&>(d))
      : "l"(reinterpret_cast<unsigned long long&>(a)), "l"(reinterpret_cast<unsigned long long&>(b)));
  return d;
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}

struct DeltaScanParams {
  DeltaGeom g;
  const float* kq;           // [rows, Hk, 2, dkp] or [rows, H, 3, dkp]
  const float* g4;           // [blocks, H, dkp] or null
  const float* v;            // [rows, H, vp]
  const float* coef;         // [blocks, H, kCoef]
  float* state;              // [slots, H, dim, vp]
  float* o;                  // [rows, H, vp]
  const int* cu;
  const int* slots;
  const int* pos0;
  const int* blk0;
};

constexpr int kScanWarps = 4;
constexpr int kScanTile = 16;    // tokens per shared-memory stage

template <int KT, int CT, bool CH>
struct ScanCfg {
  static constexpr int DK = 8 * KT;
  static constexpr int kVecs = CH ? 3 : 2;                            // vectors per token
  static constexpr int kCols = kScanWarps * 4 * CT;                   // value columns per CTA
  static constexpr int kV = kScanTile * kVecs * DK;                   // float offsets within a stage
  static constexpr int kC = kV + kScanTile * kCols;
  static constexpr int kG = kC + kScanTile / kBlk * kCoef;
  static constexpr int kStageFloats = kG + (CH ? kScanTile / kBlk * DK : 0);
  static constexpr int kSmemBytes = 2 * kStageFloats * 4;
};

// Eight lanes share CT columns of S (lane kl of the eight holds rows {32 i + 4 kl .. + 3}); a warp walks 4 * CT columns,
// kBlk tokens at a time. The sums d_j, e_j over the eight lanes are exchanged so that lane j ends up with d_j and lane
// 4 + j with e_j of its columns; every lane then solves for u itself, and lanes 4 .. 7 write the read-outs. A float of k or
// q loaded from shared memory feeds CT columns: with CT = 2 the kernel is bound by those loads, with CT = 4 by the
// multiply-adds; small batches take fewer columns per lane and more warps.
template <int KT, int CT, bool CH>
__global__ void __launch_bounds__(kScanWarps * 32, 2)
delta_scan_kernel(DeltaScanParams p) {
  pdl_grid_wait();
  using Cfg = ScanCfg<KT, CT, CH>;
  constexpr int DK = Cfg::DK, kScanCols = Cfg::kCols, kVecs = Cfg::kVecs;
  extern __shared__ __align__(16) float sm[];
  const DeltaGeom& g = p.g;
  const int seq = blockIdx.z, head = blockIdx.y;
  const int row0 = p.cu[seq], n = p.cu[seq + 1] - row0;
  const int slot = p.slots[seq];
  if (n <= 0 || slot < 0) return;
  const int blk0 = p.blk0[seq], n_blk = (n + kBlk - 1) / kBlk;
  const int hk = CH ? head : head / (g.H / g.Hk), n_hk = CH ? g.H : g.Hk;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kl = lane & 7, cg = lane >> 3;
  const int slice0 = blockIdx.x * kScanCols;
  const int lcol = (warp * 4 + cg) * CT;           // first column of this lane within the slice
  const int col0 = slice0 + lcol;

  float2 S[CT][KT / 2];
  float* st = p.state + (static_cast<long long>(slot) * g.H + head) * g.dim * g.vp;
  const bool has_state = p.pos0[seq] > 0;
#pragma unroll
  for (int c = 0; c < CT; ++c)
#pragma unroll
    for (int e = 0; e < KT; ++e) {
      const int k = ((e >> 2) * 8 + kl) * 4 + (e & 3);
      float val = 0.f;
      if (has_state && k < g.dim && col0 + c < g.vdim) val = st[static_cast<long long>(k) * g.vp + col0 + c];
      if (e & 1) S[c][e >> 1].y = val; else S[c][e >> 1].x = val;
    }

  const int n_tiles = (n + kScanTile - 1) / kScanTile;
  auto issue = [&](int tile) {
    float* base = sm + (tile & 1) * Cfg::kStageFloats;
    const int t0 = tile * kScanTile;
    const int cnt = min(kScanTile, n - t0);
    const int full = (cnt + kBlk - 1) / kBlk * kBlk;     // tokens past the end of the last block are zeros
    constexpr int kRowVec = kVecs * DK / 4;
    for (int i = threadIdx.x; i < full * kRowVec; i += kScanWarps * 32) {
      const int t = i / kRowVec, w = i % kRowVec;
      const int ts = min(t, cnt - 1);
      cp16(smem_u32(base + t * kVecs * DK + w * 4), p.kq + (static_cast<long long>(row0 + t0 + ts) * n_hk + hk) * kVecs * DK + w * 4,
           t < cnt ? 16 : 0);
    }
    if constexpr (CH) {
      for (int i = threadIdx.x; i < full / kBlk * (DK / 4); i += kScanWarps * 32) {
        const int bi = i / (DK / 4), w = i % (DK / 4);
        cp16(smem_u32(base + Cfg::kG + bi * DK + w * 4),
             p.g4 + (static_cast<long long>(blk0 + tile * (kScanTile / kBlk) + bi) * g.H + head) * DK + w * 4, 16);
      }
    }
    constexpr int kColVec = kScanCols / 4;
    for (int i = threadIdx.x; i < full * kColVec; i += kScanWarps * 32) {
      const int t = i / kColVec, w = i % kColVec;
      const int ts = min(t, cnt - 1);
      const int col = slice0 + w * 4;
      const bool ok = col < g.vp;
      cp16(smem_u32(base + Cfg::kV + t * kScanCols + w * 4),
           p.v + (static_cast<long long>(row0 + t0 + ts) * g.H + head) * g.vp + (ok ? col : 0), ok && t < cnt ? 16 : 0);
    }
    constexpr int kCoefVec = kCoef / 4;
    if (threadIdx.x < full / kBlk * kCoefVec) {
      const int bi = threadIdx.x / kCoefVec, w = threadIdx.x % kCoefVec;
      cp16(smem_u32(base + Cfg::kC + bi * kCoef + w * 4),
           p.coef + (static_cast<long long>(blk0 + tile * (kScanTile / kBlk) + bi) * g.H + head) * kCoef + w * 4, 16);
    }
  };
  issue(0);
  asm volatile("cp.async.commit_group;" ::: "memory");

  const int src0 = lane & ~7;
  for (int tile = 0; tile < n_tiles; ++tile) {
    if (tile + 1 < n_tiles) issue(tile + 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const float* base = sm + (tile & 1) * Cfg::kStageFloats;
    const int nb = min(kScanTile / kBlk, n_blk - tile * (kScanTile / kBlk));
    for (int bi = 0; bi < nb; ++bi) {
      const float* kqb = base + bi * kBlk * kVecs * DK;
      const float4* cf = reinterpret_cast<const float4*>(base + Cfg::kC + bi * kCoef);
      float2 k2[CH ? 1 : kBlk][KT / 2];            // (kept for the update, which has vectors of its own with CH)
      float a[2 * kBlk][CT];                       // d_0 .. d_3, e_0 .. e_3 per column
#pragma unroll
      for (int j = 0; j < kBlk; ++j) {
        const float4* kr = reinterpret_cast<const float4*>(kqb + j * kVecs * DK);
        float2(&kj)[KT / 2] = k2[CH ? 0 : j];
        const float4* qr = kr + DK / 4;
        float2 dk[CT], dq[CT];
#pragma unroll
        for (int c = 0; c < CT; ++c) dk[c] = dq[c] = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < KT / 4; ++i) {
          const float4 kk = kr[i * 8 + kl], qq = qr[i * 8 + kl];
          kj[2 * i] = make_float2(kk.x, kk.y);
          kj[2 * i + 1] = make_float2(kk.z, kk.w);
          const float2 q0 = make_float2(qq.x, qq.y), q1 = make_float2(qq.z, qq.w);
#pragma unroll
          for (int c = 0; c < CT; ++c) {
            dk[c] = fma2(S[c][2 * i], kj[2 * i], dk[c]);
            dq[c] = fma2(S[c][2 * i], q0, dq[c]);
            dk[c] = fma2(S[c][2 * i + 1], kj[2 * i + 1], dk[c]);
            dq[c] = fma2(S[c][2 * i + 1], q1, dq[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < CT; ++c) {
          a[j][c] = dk[c].x + dk[c].y;
          a[kBlk + j][c] = dq[c].x + dq[c].y;
        }
      }
      // halve the number of sums held per lane at each exchange
      float r4[4][CT], r2[2][CT], r1[CT];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int c = 0; c < CT; ++c) {
          const float keep = (lane & 4) ? a[4 + i][c] : a[i][c], give = (lane & 4) ? a[i][c] : a[4 + i][c];
          r4[i][c] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
        }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int c = 0; c < CT; ++c) {
          const float keep = (lane & 2) ? r4[2 + i][c] : r4[i][c], give = (lane & 2) ? r4[i][c] : r4[2 + i][c];
          r2[i][c] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
        }
#pragma unroll
      for (int c = 0; c < CT; ++c) {
        const float keep = (lane & 1) ? r2[1][c] : r2[0][c], give = (lane & 1) ? r2[0][c] : r2[1][c];
        r1[c] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
      }
      const float4 G = cf[0], be = cf[1], A0 = cf[2], A1 = cf[3], cc = cf[4];
      float vals[kBlk][CT];
#pragma unroll
      for (int j = 0; j < kBlk; ++j) {
        const float* vr = base + Cfg::kV + (bi * kBlk + j) * kScanCols + lcol;
        if constexpr (CT == 4) {
          const float4 t = *reinterpret_cast<const float4*>(vr);
          vals[j][0] = t.x; vals[j][1] = t.y; vals[j][2] = t.z; vals[j][3] = t.w;
        } else {
#pragma unroll
          for (int c = 0; c < CT; ++c) vals[j][c] = vr[c];
        }
      }
      float u[kBlk][CT];
#pragma unroll
      for (int c = 0; c < CT; ++c) {
        float d[kBlk], vv[kBlk];
#pragma unroll
        for (int j = 0; j < kBlk; ++j) {
          d[j] = __shfl_sync(0xffffffffu, r1[c], src0 + j);
          vv[j] = vals[j][c];
        }
        u[0][c] = be.x * fmaf(-G.x, d[0], vv[0]);
        u[1][c] = be.y * fmaf(-A0.x, u[0][c], fmaf(-G.y, d[1], vv[1]));
        u[2][c] = be.z * fmaf(-A0.z, u[1][c], fmaf(-A0.y, u[0][c], fmaf(-G.z, d[2], vv[2])));
        u[3][c] = be.w * fmaf(-A1.y, u[2][c], fmaf(-A1.x, u[1][c], fmaf(-A0.w, u[0][c], fmaf(-G.w, d[3], vv[3]))));
      }
      if (kl >= 4) {
        const int j = kl - 4, t = tile * kScanTile + bi * kBlk + j;
        const float4 W = cf[5 + j];
        const float Gj = base[Cfg::kC + bi * kCoef + j];
        if (t < n) {
          float* orow = p.o + (static_cast<long long>(row0 + t) * g.H + head) * g.vp + col0;
#pragma unroll
          for (int c = 0; c < CT; ++c)
            if (col0 + c < g.vdim)
              orow[c] = fmaf(Gj, r1[c], fmaf(W.x, u[0][c], fmaf(W.y, u[1][c], fmaf(W.z, u[2][c], W.w * u[3][c]))));
        }
      }
      if constexpr (CH) {
        const float4* gr = reinterpret_cast<const float4*>(base + Cfg::kG + bi * DK);
        const float4* ur = reinterpret_cast<const float4*>(kqb + 2 * DK);
#pragma unroll
        for (int i = 0; i < KT / 4; ++i) {
          const float4 gg = gr[i * 8 + kl];
          const float2 g0 = make_float2(gg.x, gg.y), g1 = make_float2(gg.z, gg.w);
#pragma unroll
          for (int c = 0; c < CT; ++c) {
            S[c][2 * i] = mul2(S[c][2 * i], g0);
            S[c][2 * i + 1] = mul2(S[c][2 * i + 1], g1);
          }
#pragma unroll
          for (int j = 0; j < kBlk; ++j) {
            const float4 kk = ur[j * (kVecs * DK / 4) + i * 8 + kl];
            const float2 k0 = make_float2(kk.x, kk.y), k1 = make_float2(kk.z, kk.w);
#pragma unroll
            for (int c = 0; c < CT; ++c) {
              const float2 uu = make_float2(u[j][c], u[j][c]);
              S[c][2 * i] = fma2(k0, uu, S[c][2 * i]);
              S[c][2 * i + 1] = fma2(k1, uu, S[c][2 * i + 1]);
            }
          }
        }
      } else {
        const float2 g2 = make_float2(G.w, G.w);
        const float cs[kBlk] = {cc.x, cc.y, cc.z, cc.w};
#pragma unroll
        for (int c = 0; c < CT; ++c) {
          float2 uu[kBlk];
#pragma unroll
          for (int j = 0; j < kBlk; ++j) uu[j] = make_float2(cs[j] * u[j][c], cs[j] * u[j][c]);
#pragma unroll
          for (int i = 0; i < KT / 2; ++i) {
            float2 acc = mul2(S[c][i], g2);
#pragma unroll
            for (int j = 0; j < kBlk; ++j) acc = fma2(k2[j][i], uu[j], acc);
            S[c][i] = acc;
          }
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int c = 0; c < CT; ++c)
#pragma unroll
    for (int e = 0; e < KT; ++e) {
      const int k = ((e >> 2) * 8 + kl) * 4 + (e & 3);
      if (k < g.dim && col0 + c < g.vdim)
        st[static_cast<long long>(k) * g.vp + col0 + c] = (e & 1) ? S[c][e >> 1].y : S[c][e >> 1].x;
    }
}

// ------------------------------------------------------------------ read-out norm and gate
// y = o / rms(o) * weight * gate per (row, head), in the projection's type; columns past H * vdim of the output row
// are zeroed by the last head's warp. A warp takes one head of kNormRows rows; heads of up to 128 columns are read once,
// all rows at a time, wider ones are read twice.
constexpr int kNormRows = 4;

template <typename T, bool NARROW>
__global__ void __launch_bounds__(256)
delta_gate_norm_kernel(DeltaGeom g, const float* o, const T* gate, long long ldg, int kind, const float* weight, T* y, long long ldy,
                       int y_cols, int rows, float eps) {
  pdl_trigger();
  pdl_grid_wait();
  const int h = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= g.H) return;
  constexpr bool kFast = sizeof(T) == 2;
  const bool vec = g.vdim % 4 == 0 && ldy % 4 == 0 && ldg % 4 == 0;
  const int row_a = blockIdx.y * kNormRows, cnt = min(kNormRows, rows - row_a);
  const float inv_n = 1.f / static_cast<float>(g.vdim);
  const float* o0 = o + (static_cast<long long>(row_a) * g.H + h) * g.vp;
  const T* g0 = gate + static_cast<long long>(row_a) * ldg + h * g.vdim;
  T* y0 = y + row_a * ldy + h * g.vdim;
  const long long so = static_cast<long long>(g.H) * g.vp;
  auto store = [&](T* dst, int c, const float (&f)[4]) {
    if (vec) {
      if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(dst + c) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
      else *reinterpret_cast<float4*>(dst + c) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < g.vdim) dst[c + e] = from_f32<T>(f[e]);
    }
  };
  if constexpr (NARROW) {
    const int c = lane * 4, valid = g.vdim - c;
    float f[kNormRows][4], gt[kNormRows][4], wt[4];
#pragma unroll
    for (int r = 0; r < kNormRows; ++r) {
      const int rr = min(r, cnt - 1);
      load_ch<float, 4>(o0 + rr * so + c, valid, true, f[r]);
      load_ch<T, 4>(g0 + rr * ldg + c, valid, vec, gt[r]);
    }
    load_ch<float, 4>(weight + c, valid, true, wt);
#pragma unroll
    for (int r = 0; r < kNormRows; ++r) {
      const float ss = warp_sum(f[r][0] * f[r][0] + f[r][1] * f[r][1] + f[r][2] * f[r][2] + f[r][3] * f[r][3]);
      const float rs = rsqrtf(fmaf(ss, inv_n, eps));
#pragma unroll
      for (int e = 0; e < 4; ++e) f[r][e] *= rs * wt[e] * gate_f<kFast>(gt[r][e], kind);
      if (r < cnt && valid > 0) store(y0 + r * ldy, c, f[r]);
    }
  } else {
    for (int r = 0; r < cnt; ++r) {
      float ss = 0.f;
      for (int c = lane * 4; c < g.vdim; c += 128) {
        float f[4];
        load_ch<float, 4>(o0 + r * so + c, g.vdim - c, true, f);
        ss += f[0] * f[0] + f[1] * f[1] + f[2] * f[2] + f[3] * f[3];
      }
      const float rs = rsqrtf(fmaf(warp_sum(ss), inv_n, eps));
      for (int c = lane * 4; c < g.vdim; c += 128) {
        float f[4], gt[4], wt[4];
        load_ch<float, 4>(o0 + r * so + c, g.vdim - c, true, f);
        load_ch<T, 4>(g0 + r * ldg + c, g.vdim - c, vec, gt);
        load_ch<float, 4>(weight + c, g.vdim - c, true, wt);
#pragma unroll
        for (int e = 0; e < 4; ++e) f[e] *= rs * wt[e] * gate_f<kFast>(gt[e], kind);
        store(y0 + r * ldy, c, f);
      }
    }
  }
  if (h == g.H - 1)
    for (int r = 0; r < cnt; ++r)
      for (int c = g.H * g.vdim + lane; c < y_cols; c += 32) y[(row_a + r) * ldy + c] = from_f32<T>(0.f);
}

// ------------------------------------------------------------------ decoded rows: one token per sequence, one launch
struct DeltaStepParams {
  DeltaGeom g;
  DeltaSide side;
  const void* proj;
  const float* conv_w;
  const float* a_log;
  const float* dt_bias;
  const float* norm_w;
  void* conv_state;
  float* state;
  const int* slots;          // [rows], -1: padding
  const int* pos;            // [rows]
  void* y;
  long long ldy;
  int y_cols, taps;
  float eps;
  int kh;                    // key heads per CTA
};

constexpr int kStepThreads = 256;
constexpr int kStepWarps = kStepThreads / 32;

// CTA = (sequence, KH key heads): it owns the heads' q / k channels and all value heads that read them. A warp holds RPW
// rows of a 128-column block of S: dim / 8 rounded up.
template <typename T, int RPW, bool CH>
__global__ void __launch_bounds__(kStepThreads, RPW <= 16 ? 2 : 1)
delta_step_kernel(DeltaStepParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const DeltaGeom& g = p.g;
  extern __shared__ __align__(16) float sm[];
  const int per1 = g.H / g.Hk, KH = p.kh, per = KH * per1, hk = blockIdx.y * KH;    // value heads per key head and of this CTA
  float* sq = sm;                          // [KH * dkp]
  float* sk = sq + KH * g.dkp;             // [KH * dkp]
  float* sv = sk + KH * g.dkp;             // [per * vp]
  float* so = sv + per * g.vp;             // [per * vp]
  float* part = so + per * g.vp;           // [8 warps][2][128]
  float* red = part + kStepWarps * 256;    // [KH][4]: factors of q and k, k . q of the unit vectors
  float* sd = red + KH * 4;                // CH: [per * dkp] decays
  const int row = blockIdx.x;
  const int slot = p.slots[row];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  T* y = static_cast<T*>(p.y) + row * p.ldy;
  if (hk + KH == g.Hk)
    for (int c = g.H * g.vdim + tid; c < p.y_cols; c += kStepThreads) y[c] = from_f32<T>(0.f);
  if (slot < 0) {
    for (int c = tid; c < per * g.vdim; c += kStepThreads) y[hk * per1 * g.vdim + c] = from_f32<T>(0.f);
    return;
  }
  const bool has_state = p.pos[row] > 0;
  const T* proj = static_cast<const T*>(p.proj) + row * g.ldp;
  const int tail = p.taps - 1;
  T* cs = static_cast<T*>(p.conv_state) + static_cast<long long>(slot) * tail * g.conv_c;
  // The state streams through registers one (head, 128-column block) at a time; the first block is requested before the
  // convolution, every later one as soon as its predecessor has been stored.
  const int col_blocks = (g.vp + 127) / 128, steps = per * col_blocks;
  float4 S[RPW];
  auto state_at = [&](int it) {
    return p.state + (static_cast<long long>(slot) * g.H + hk * per1 + it / col_blocks) * g.dim * g.vp + (it % col_blocks) * 128 +
           lane * 4;
  };
  auto fetch = [&](int it) {
    const float* st = state_at(it);
    const bool ok = has_state && (it % col_blocks) * 128 + lane * 4 < g.vp;
#pragma unroll
    for (int i = 0; i < RPW; ++i) {
      const int k = warp + kStepWarps * i;
      S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (ok && k < g.dim) S[i] = __ldcs(reinterpret_cast<const float4*>(st + static_cast<long long>(k) * g.vp));
    }
  };
  fetch(0);
  // channel i of this CTA (its q, its k, then the v of its heads): column in the projection, place in shared memory
  const int n_q = KH * g.dim, n_ch = 2 * n_q + per * g.vdim;
  auto channel = [&](int i, int* c) -> float* {
    if (i < 2 * n_q) {
      const bool is_k = i >= n_q;
      const int j = is_k ? i - n_q : i;
      *c = (is_k ? g.off_k : 0) + hk * g.dim + j;
      return (is_k ? sk : sq) + (j / g.dim) * g.dkp + j % g.dim;
    }
    const int v = i - 2 * n_q;
    *c = g.off_v + hk * per1 * g.vdim + v;
    return sv + (v / g.vdim) * g.vp + v % g.vdim;
  };
  for (int i0 = tid; i0 < n_ch; i0 += 2 * kStepThreads) {
    float x[2][8], w[2][8];               // both channels' inputs are requested before anything is written
    int c[2];
    float* dst[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int i = i0 + h * kStepThreads;
      dst[h] = i < n_ch ? channel(i, &c[h]) : nullptr;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        x[h][j] = w[h][j] = 0.f;
        if (dst[h] && j <= tail) {
          w[h][j] = p.conv_w[static_cast<long long>(j) * g.conv_c + c[h]];
          if (j == tail) x[h][j] = to_f32<T>(proj[c[h]]);
          else if (has_state) x[h][j] = to_f32<T>(cs[static_cast<long long>(j) * g.conv_c + c[h]]);
        }
      }
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      if (!dst[h]) continue;
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        acc = fmaf(w[h][j], x[h][j], acc);
        if (j > 0 && j <= tail) cs[static_cast<long long>(j - 1) * g.conv_c + c[h]] = from_f32<T>(x[h][j]);
      }
      *dst[h] = silu_f<sizeof(T) == 2>(acc);
    }
  }
  if constexpr (CH) {
    for (int i = tid; i < per * g.dim; i += kStepThreads) {
      const int h = hk * per1 + i / g.dim, d = i % g.dim;
      sd[(i / g.dim) * g.dkp + d] =
          decay_f<sizeof(T) == 2>(p.side.dec[row * p.side.ld_dec + h * g.dim + d] + p.dt_bias[h * g.dim + d], expf(p.a_log[h]));
    }
  }
  __syncthreads();
  for (int kh = warp; kh < KH; kh += kStepWarps) {
    float sqq = 0.f, skk = 0.f, sqk = 0.f;
    for (int d = lane; d < g.dim; d += 32) {
      const float a = sq[kh * g.dkp + d], b = sk[kh * g.dkp + d];
      sqq = fmaf(a, a, sqq);
      skk = fmaf(b, b, skk);
      sqk = fmaf(a, b, sqk);
    }
    sqq = warp_sum(sqq);
    skk = warp_sum(skk);
    sqk = warp_sum(sqk);
    if (lane == 0) {
      const float rq = 1.f / (sqrtf(sqq + 1e-6f) * sqrtf(static_cast<float>(g.dim))), rk = 1.f / sqrtf(skk + 1e-6f);
      red[kh * 4] = rq;
      red[kh * 4 + 1] = rk;
      red[kh * 4 + 2] = sqk * rq * rk;
    }
  }
  __syncthreads();

  float decay = 0.f, beta = 0.f;
  for (int it = 0; it < steps; ++it) {
    const int hh = it / col_blocks, h = hk * per1 + hh, kh = hh / per1;
    const float rq = red[kh * 4], rk = red[kh * 4 + 1], kq = red[kh * 4 + 2];
    const float *hq = sq + kh * g.dkp, *hkk = sk + kh * g.dkp;
    if (it % col_blocks == 0) {
      decay = 1.f;                        // (CH: the products with the state take their channel's decay along)
      if constexpr (!CH) decay = expf(-expf(p.a_log[h]) * softplus_f(to_f32<T>(proj[g.off_a + h]) + p.dt_bias[h]));
      beta = sigmoid_f(to_f32<T>(proj[g.off_b + h]));
    }
    float* st = state_at(it);
    {
      const int col = (it % col_blocks) * 128 + lane * 4;
      const bool col_ok = col < g.vp;
      float4 dk = make_float4(0.f, 0.f, 0.f, 0.f), dq = dk;
#pragma unroll
      for (int i = 0; i < RPW; ++i) {
        const int k = warp + kStepWarps * i;
        float kk = k < g.dim ? hkk[k] * rk : 0.f, qq = k < g.dim ? hq[k] * rq : 0.f;
        if constexpr (CH) {
          const float dd = k < g.dim ? sd[hh * g.dkp + k] : 0.f;
          kk *= dd;
          qq *= dd;
        }
        dk.x = fmaf(S[i].x, kk, dk.x); dk.y = fmaf(S[i].y, kk, dk.y);
        dk.z = fmaf(S[i].z, kk, dk.z); dk.w = fmaf(S[i].w, kk, dk.w);
        dq.x = fmaf(S[i].x, qq, dq.x); dq.y = fmaf(S[i].y, qq, dq.y);
        dq.z = fmaf(S[i].z, qq, dq.z); dq.w = fmaf(S[i].w, qq, dq.w);
      }
      *reinterpret_cast<float4*>(part + warp * 256 + lane * 4) = dk;
      *reinterpret_cast<float4*>(part + warp * 256 + 128 + lane * 4) = dq;
      __syncthreads();
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
      if (col_ok) {
        float4 sdk = make_float4(0.f, 0.f, 0.f, 0.f), sdq = sdk;
#pragma unroll
        for (int w = 0; w < kStepWarps; ++w) {
          const float4 a = *reinterpret_cast<const float4*>(part + w * 256 + lane * 4);
          sdk.x += a.x; sdk.y += a.y; sdk.z += a.z; sdk.w += a.w;
        }
        const float* vr = sv + hh * g.vp + col;
        // (columns past vdim read padding that may hold anything; they are never stored as part of a result)
        u.x = beta * (vr[0] - decay * sdk.x);
        u.y = col + 1 < g.vdim ? beta * (vr[1] - decay * sdk.y) : 0.f;
        u.z = col + 2 < g.vdim ? beta * (vr[2] - decay * sdk.z) : 0.f;
        u.w = col + 3 < g.vdim ? beta * (vr[3] - decay * sdk.w) : 0.f;
        if (warp == 0) {
#pragma unroll
          for (int w = 0; w < kStepWarps; ++w) {
            const float4 a = *reinterpret_cast<const float4*>(part + w * 256 + 128 + lane * 4);
            sdq.x += a.x; sdq.y += a.y; sdq.z += a.z; sdq.w += a.w;
          }
          float* orow = so + hh * g.vp + col;
          orow[0] = fmaf(decay, sdq.x, kq * u.x);
          orow[1] = fmaf(decay, sdq.y, kq * u.y);
          orow[2] = fmaf(decay, sdq.z, kq * u.z);
          orow[3] = fmaf(decay, sdq.w, kq * u.w);
        }
#pragma unroll
        for (int i = 0; i < RPW; ++i) {
          const int k = warp + kStepWarps * i;
          if (k < g.dim) {
            const float kk = hkk[k] * rk, dd = CH ? sd[hh * g.dkp + k] : decay;
            float4 s = S[i];
            s.x = fmaf(s.x, dd, kk * u.x);
            s.y = fmaf(s.y, dd, kk * u.y);
            s.z = fmaf(s.z, dd, kk * u.z);
            s.w = fmaf(s.w, dd, kk * u.w);
            __stcs(reinterpret_cast<float4*>(st + static_cast<long long>(k) * g.vp), s);
          }
        }
      }
      if (it + 1 < steps) fetch(it + 1);
      __syncthreads();
    }
  }
  // read-out norm and gate: one warp per value head
  const T* gate = static_cast<const T*>(p.side.gate) + row * p.side.ld_gate;
  for (int hh = warp; hh < per; hh += kStepWarps) {
    const float* orow = so + hh * g.vp;
    const int c0 = (hk * per1 + hh) * g.vdim;
    float ss = 0.f;
    for (int c = lane; c < g.vdim; c += 32) ss = fmaf(orow[c], orow[c], ss);
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / static_cast<float>(g.vdim) + p.eps);
    for (int c = lane; c < g.vdim; c += 32)
      y[c0 + c] = from_f32<T>(orow[c] * r * p.norm_w[c] * gate_f(to_f32<T>(gate[c0 + c]), p.side.gate_kind));
  }
}

// geom: 11 ints in the order of DeltaGeom (without ldp), then the gate's kind; off_a is not used with dec
bool read_geom(const int* v, long long ldp, const void* gate, long long ld_gate, const float* dec, long long ld_dec, DeltaGeom* g, DeltaSide* side) {
  g->Hk = v[0]; g->H = v[1]; g->dim = v[2]; g->vdim = v[3]; g->dkp = v[4]; g->vp = v[5];
  g->off_k = v[6]; g->off_v = v[7]; g->off_b = v[8]; g->off_a = v[9]; g->conv_c = v[10];
  g->ldp = ldp;
  *side = {gate, ld_gate, v[11], dec, ld_dec};
  if (!gate || ld_gate < g->H * g->vdim || v[11] < 0 || v[11] > 1 || ldp < g->off_b + g->H || (!dec && ldp < g->off_a + g->H) ||
      (dec && (ld_dec < g->H * g->dim || ld_dec % 4 || (reinterpret_cast<uintptr_t>(dec) & 15))))
    return false;
  const bool dk_ok = g->dkp == 32 || g->dkp == 64 || g->dkp == 128 || g->dkp == 256;
  return g->Hk > 0 && g->H > 0 && g->H % g->Hk == 0 && g->dim > 0 && g->vdim > 0 && dk_ok && g->dim <= g->dkp &&
         g->vp >= g->vdim && g->vp % 4 == 0 && g->conv_c > 0 && ldp % 8 == 0 && g->off_k % 8 == 0 && g->off_v % 8 == 0 && g->conv_c % 8 == 0;
}

template <typename T, int TAPS, bool CH>
int launch_prepare_taps(const DeltaPrepParams& p, cudaStream_t s) {
  const DeltaGeom& g = p.g;
  const dim3 grid(g.Hk + (g.H * g.vdim + 255) / 256, (p.blocks + 3) / 4);
  const bool pdl = pdl_all_enabled();
  switch (g.dkp) {
    case 32: launch_pdl(delta_prepare_kernel<T, TAPS, 1, CH>, grid, dim3(128), 0, s, pdl, p); break;
    case 64: launch_pdl(delta_prepare_kernel<T, TAPS, 2, CH>, grid, dim3(128), 0, s, pdl, p); break;
    case 128: launch_pdl(delta_prepare_kernel<T, TAPS, 4, CH>, grid, dim3(128), 0, s, pdl, p); break;
    default: launch_pdl(delta_prepare_kernel<T, TAPS, 8, CH>, grid, dim3(128), 0, s, pdl, p); break;
  }
  return static_cast<int>(cudaGetLastError());
}

template <typename T, bool CH>
int launch_prepare(const DeltaPrepParams& p, int taps, cudaStream_t s) {
  switch (taps) {
    case 1: return launch_prepare_taps<T, 1, CH>(p, s);
    case 2: return launch_prepare_taps<T, 2, CH>(p, s);
    case 3: return launch_prepare_taps<T, 3, CH>(p, s);
    case 4: return launch_prepare_taps<T, 4, CH>(p, s);
    case 5: return launch_prepare_taps<T, 5, CH>(p, s);
    case 6: return launch_prepare_taps<T, 6, CH>(p, s);
    case 7: return launch_prepare_taps<T, 7, CH>(p, s);
    case 8: return launch_prepare_taps<T, 8, CH>(p, s);
    default: return -2;
  }
}

template <int KT, int CT, bool CH>
int launch_scan_cols(const DeltaScanParams& p, int nseq, cudaStream_t s) {
  using Cfg = ScanCfg<KT, CT, CH>;
  auto kern = delta_scan_kernel<KT, CT, CH>;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmemBytes);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  const dim3 grid((p.g.vdim + Cfg::kCols - 1) / Cfg::kCols, p.g.H, nseq);
  // launched after its predecessor has left: CTAs that start early land on whatever SMs drain first and stay there for
  // the whole scan, several on one SM while others idle
  launch_pdl(kern, grid, dim3(kScanWarps * 32), Cfg::kSmemBytes, s, false, p);
  return static_cast<int>(cudaGetLastError());
}

template <int KT, bool CH>
int launch_scan(const DeltaScanParams& p, int nseq, cudaStream_t s) {
  static const int forced = [] { const char* e = getenv("TESSERACT_DELTA_COLS"); return e ? atoi(e) : 0; }();
  // columns of the whole launch against what one warp per scheduler covers
  const long long cols = static_cast<long long>(nseq) * p.g.H * p.g.vdim, one = 4ll * sm_count() * 4;
  int ct = forced ? forced : (cols >= 5 * one ? 4 : (cols >= one ? 2 : 1));
  if (KT > 16 && ct > 2) ct = 2;
  if constexpr (KT <= 16)
    if (ct == 4) return launch_scan_cols<KT, 4, CH>(p, nseq, s);
  return ct >= 2 ? launch_scan_cols<KT, 2, CH>(p, nseq, s) : launch_scan_cols<KT, 1, CH>(p, nseq, s);
}

template <bool CH>
int launch_scan_dim(const DeltaScanParams& p, int nseq, cudaStream_t s) {
  switch (p.g.dkp) {
    case 32: return launch_scan<4, CH>(p, nseq, s);
    case 64: return launch_scan<8, CH>(p, nseq, s);
    case 128: return launch_scan<16, CH>(p, nseq, s);
    default: return launch_scan<32, CH>(p, nseq, s);
  }
}

template <typename T, int RPW, bool CH>
int launch_step(DeltaStepParams p, int rows, cudaStream_t s) {
  // several key heads per CTA where that leaves every SM its CTAs: the state of the next one is under way early
  const int per1 = p.g.H / p.g.Hk;
  p.kh = 1;
  while (p.kh * per1 < 4 && p.g.Hk % (2 * p.kh) == 0 && static_cast<long long>(rows) * (p.g.Hk / (2 * p.kh)) >= 3 * sm_count()) p.kh *= 2;
  const int per = p.kh * per1;
  const int smem = (2 * p.kh * p.g.dkp + 2 * per * p.g.vp + kStepWarps * 256 + p.kh * 4 + (CH ? per * p.g.dkp : 0)) * 4;
  if (smem > 200 * 1024) return -2;
  auto kern = delta_step_kernel<T, RPW, CH>;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  launch_pdl(kern, dim3(rows, p.g.Hk / p.kh), dim3(kStepThreads), smem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace
}  // namespace tsb

// Prompt rows [rows, ldp] of nseq sequences, cut into blocks of 4 tokens from each sequence's first row (blk_seq [blocks],
// blk0 [nseq + 1]). dtype: 0 = fp32, 1 = bf16 (projection, gate, convolution state, y). `kq`, `v`, `coef`, `o` are fp32 scratch
// of rows * Hk * 2 * dkp, rows * H * vp, blocks * H * 36 and rows * H * vp elements (16-byte aligned). With `dec` [rows, ld_dec]
// (dt_bias then is [H * dim]) kq has rows * H * 3 * dkp elements and `g4` is scratch of blocks * H * dkp. See the structures above
// for the rest.
TSB_EXPORT int tsb_delta_prefill(const void* proj, long long ldp, const int* geom, const void* gate, long long ld_gate, const float* dec,
                                 long long ld_dec, const float* conv_w, const float* a_log, const float* dt_bias, const float* norm_w,
                                 void* conv_state, float* state, const int* cu, const int* slots, const int* pos0, const int* blk_seq,
                                 const int* blk0, float* kq, float* g4, float* v, float* coef, float* o, void* y, long long ldy, int y_cols,
                                 int rows, int blocks, int nseq, int taps, float eps, int dtype, void* stream) {
  using namespace tsb;
  DeltaGeom g;
  DeltaSide side;
  if (!read_geom(geom, ldp, gate, ld_gate, dec, ld_dec, &g, &side) || rows <= 0 || blocks <= 0 || nseq <= 0 || nseq > 65535 || taps < 1 ||
      taps > 8 || (blocks + 3) / 4 > 65535 || (rows + kNormRows - 1) / kNormRows > 65535 || (dtype != 0 && dtype != 1) ||
      y_cols < g.H * g.vdim || (dec && !g4))
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  DeltaPrepParams pp{g, proj, conv_w, a_log, dt_bias, dec, ld_dec, conv_state, cu, slots, pos0, blk_seq, blk0, kq, g4, v, coef, blocks};
  int rc = dec ? (dtype == 1 ? launch_prepare<__nv_bfloat16, true>(pp, taps, s) : launch_prepare<float, true>(pp, taps, s))
               : (dtype == 1 ? launch_prepare<__nv_bfloat16, false>(pp, taps, s) : launch_prepare<float, false>(pp, taps, s));
  if (rc) return rc;
  const bool pdl = pdl_all_enabled();
  if (taps > 1) {
    const dim3 grid((g.conv_c + 255) / 256, nseq);
    if (dtype == 1)
      launch_pdl(conv_state_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl, static_cast<const __nv_bfloat16*>(proj), g.ldp, g.conv_c,
                 static_cast<__nv_bfloat16*>(conv_state), cu, slots, pos0, taps - 1);
    else
      launch_pdl(conv_state_kernel<float>, grid, dim3(256), 0, s, pdl, static_cast<const float*>(proj), g.ldp, g.conv_c,
                 static_cast<float*>(conv_state), cu, slots, pos0, taps - 1);
    rc = static_cast<int>(cudaGetLastError());
    if (rc) return rc;
  }
  DeltaScanParams sp{g, kq, g4, v, coef, state, o, cu, slots, pos0, blk0};
  rc = dec ? launch_scan_dim<true>(sp, nseq, s) : launch_scan_dim<false>(sp, nseq, s);
  if (rc) return rc;
  const dim3 ngrid((g.H + 7) / 8, (rows + kNormRows - 1) / kNormRows);
  auto norm = [&](auto tag, auto narrow) {
    using T = decltype(tag);
    launch_pdl(delta_gate_norm_kernel<T, decltype(narrow)::value>, ngrid, dim3(256), 0, s, pdl, g, o, static_cast<const T*>(gate), ld_gate,
               side.gate_kind, norm_w, static_cast<T*>(y), ldy, y_cols, rows, eps);
  };
  const bool narrow = g.vdim <= 128;
  if (dtype == 1) narrow ? norm(__nv_bfloat16{}, std::true_type{}) : norm(__nv_bfloat16{}, std::false_type{});
  else narrow ? norm(float{}, std::true_type{}) : norm(float{}, std::false_type{});
  return static_cast<int>(cudaGetLastError());
}

// Decoded rows: row i is the next token of the sequence in slot slots[i] (-1: padding, y = 0) at position pos[i].
TSB_EXPORT int tsb_delta_step(const void* proj, long long ldp, const int* geom, const void* gate, long long ld_gate, const float* dec,
                              long long ld_dec, const float* conv_w, const float* a_log, const float* dt_bias, const float* norm_w,
                              void* conv_state, float* state, const int* slots, const int* pos, void* y, long long ldy, int y_cols, int rows,
                              int taps, float eps, int dtype, void* stream) {
  using namespace tsb;
  DeltaGeom g;
  DeltaSide side;
  if (!read_geom(geom, ldp, gate, ld_gate, dec, ld_dec, &g, &side) || rows <= 0 || g.Hk > 65535 || taps < 1 || taps > 8 ||
      (dtype != 0 && dtype != 1) || y_cols < g.H * g.vdim)
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  DeltaStepParams p{g, side, proj, conv_w, a_log, dt_bias, norm_w, conv_state, state, slots, pos, y, ldy, y_cols, taps, eps, 1};
#define TSB_STEP(R)                                                                                                       \
  if (dec) return dtype == 1 ? launch_step<__nv_bfloat16, R, true>(p, rows, s) : launch_step<float, R, true>(p, rows, s); \
  return dtype == 1 ? launch_step<__nv_bfloat16, R, false>(p, rows, s) : launch_step<float, R, false>(p, rows, s)
  switch (g.dkp) {
    case 32: TSB_STEP(4);
    case 64: TSB_STEP(8);
    case 128: TSB_STEP(16);
    default: TSB_STEP(32);
  }
#undef TSB_STEP
}
