// Recurrences over a matrix state per head, S [values e][keys d] in fp32:
//
//   S_t = diag(w_t) S_(t-1) + v_t k_t^T,   o_t = S q_t   with S = S_t (AFTER) or S_(t-1)
//
// w is a factor per key column. `StateStep` takes one token, `state_scan` walks a portion token by token; both keep everything in
// fp32. The caller brings q, k, w and v.
#pragma once

#include "warp_mma.cuh"

namespace tsb {

// One token, 256 threads. LPR lanes share a row of the state (PPL times four columns each), RPT rows are in flight per lane; the
// first ones are requested by the constructor. D is a multiple of 4 up to 4 LPR PPL, E any. sq, sk, sw [D], sv [E] in shared memory
// must be complete when `run` is called; so [E] is after the next barrier.
template <int LPR, int PPL, int RPT, bool AFTER>
struct StateStep {
  static constexpr int kGroups = 256 / LPR;
  float* st;
  int E, D, grp, gl;
  bool fresh;
  float4 S[RPT][PPL];

  __device__ __forceinline__ void fetch(int e0) {
#pragma unroll
    for (int r = 0; r < RPT; ++r)
#pragma unroll
      for (int i = 0; i < PPL; ++i) {
        const int e = e0 + r * kGroups, d = (gl + i * LPR) * 4;
        S[r][i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && e < E && d < D) S[r][i] = __ldcs(reinterpret_cast<const float4*>(st + static_cast<long long>(e) * D + d));
      }
  }
  __device__ __forceinline__ StateStep(float* st_, int E_, int D_, bool fresh_)
      : st(st_), E(E_), D(D_), grp(threadIdx.x / LPR), gl(threadIdx.x % LPR), fresh(fresh_) {
    fetch(grp);
  }
  __device__ __forceinline__ void run(const float* sq, const float* sk, const float* sw, const float* sv, float* so) {
    float4 q[PPL], k[PPL], w[PPL];
#pragma unroll
    for (int i = 0; i < PPL; ++i) {
      const int d = (gl + i * LPR) * 4;
      const bool ok = d < D;
      q[i] = ok ? *reinterpret_cast<const float4*>(sq + d) : make_float4(0.f, 0.f, 0.f, 0.f);
      k[i] = ok ? *reinterpret_cast<const float4*>(sk + d) : make_float4(0.f, 0.f, 0.f, 0.f);
      w[i] = ok ? *reinterpret_cast<const float4*>(sw + d) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int e0 = grp; e0 - grp < E; e0 += kGroups * RPT) {          // (uniform bounds: the sums are shuffles)
      if (e0 != grp) fetch(e0);
      float o[RPT];
#pragma unroll
      for (int r = 0; r < RPT; ++r) {
        const int e = e0 + r * kGroups;
        const float v = e < E ? sv[e] : 0.f;
        o[r] = 0.f;
#pragma unroll
        for (int i = 0; i < PPL; ++i) {
          float4 s = S[r][i];
          if (!AFTER) o[r] = fmaf(s.x, q[i].x, fmaf(s.y, q[i].y, fmaf(s.z, q[i].z, fmaf(s.w, q[i].w, o[r]))));
          s.x = fmaf(w[i].x, s.x, k[i].x * v); s.y = fmaf(w[i].y, s.y, k[i].y * v);
          s.z = fmaf(w[i].z, s.z, k[i].z * v); s.w = fmaf(w[i].w, s.w, k[i].w * v);
          if (AFTER) o[r] = fmaf(s.x, q[i].x, fmaf(s.y, q[i].y, fmaf(s.z, q[i].z, fmaf(s.w, q[i].w, o[r]))));
          const int d = (gl + i * LPR) * 4;
          if (e < E && d < D) __stcs(reinterpret_cast<float4*>(st + static_cast<long long>(e) * D + d), s);
        }
      }
#pragma unroll
      for (int r = 0; r < RPT; ++r) {
#pragma unroll
        for (int m = LPR / 2; m; m >>= 1) o[r] += __shfl_xor_sync(0xffffffffu, o[r], m);
        const int e = e0 + r * kGroups;
        if (gl == 0 && e < E) so[e] = o[r];
      }
    }
  }
};

// A portion of n tokens, 128 threads: warp w walks the state's rows e0 + 4 w .. + 3, lane l holds their columns l + 32 i. `fetch(t, d, q,
// k, w)` gives a token's operands at column d < D, `value(t, e)` its value; `emit(t, e, o[4])` receives the read-out of four rows.
constexpr int kScanRows = 16;
template <int RL>
struct ScanShape {
  static constexpr int kTok = RL > 4 ? 8 : 16, kCols = RL * 32;
  static constexpr int kFloats = kTok * (3 * kCols + kScanRows);
};

template <int RL, bool AFTER, typename Fetch, typename Value, typename Emit>
__device__ __forceinline__ void state_scan(float* sm, float* st, int E, int D, bool fresh, int n, int e_first, Fetch fetch, Value value,
                                           Emit emit) {
  using C = ScanShape<RL>;
  float *sq = sm, *sk = sq + C::kTok * C::kCols, *sw = sk + C::kTok * C::kCols, *sv = sw + C::kTok * C::kCols;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, e0 = e_first + warp * 4;
  float S[RL][4];
#pragma unroll
  for (int i = 0; i < RL; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = lane + 32 * i;
      S[i][j] = !fresh && d < D && e0 + j < E ? st[static_cast<long long>(e0 + j) * D + d] : 0.f;
    }
  for (int t0 = 0; t0 < n; t0 += C::kTok) {
    const int cnt = min(C::kTok, n - t0);
    __syncthreads();
    for (int i = tid; i < cnt * C::kCols; i += 128) {
      const int r = i / C::kCols, d = i % C::kCols;
      float q = 0.f, k = 0.f, w = 0.f;
      if (d < D) fetch(t0 + r, d, q, k, w);
      sq[i] = q;
      sk[i] = k;
      sw[i] = w;
    }
    for (int i = tid; i < cnt * kScanRows; i += 128) sv[i] = e_first + i % kScanRows < E ? value(t0 + i / kScanRows, e_first + i % kScanRows) : 0.f;
    __syncthreads();
    for (int r = 0; r < cnt; ++r) {
      float v[4], o[4] = {};
#pragma unroll
      for (int j = 0; j < 4; ++j) v[j] = sv[r * kScanRows + warp * 4 + j];
#pragma unroll
      for (int i = 0; i < RL; ++i) {
        const float q = sq[r * C::kCols + lane + 32 * i], k = sk[r * C::kCols + lane + 32 * i], w = sw[r * C::kCols + lane + 32 * i];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (!AFTER) o[j] = fmaf(S[i][j], q, o[j]);
          S[i][j] = fmaf(w, S[i][j], k * v[j]);
          if (AFTER) o[j] = fmaf(S[i][j], q, o[j]);
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] = warp_sum(o[j]);
      if (lane == 0 && e0 < E) emit(t0 + r, e0, o);
    }
  }
#pragma unroll
  for (int i = 0; i < RL; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = lane + 32 * i;
      if (d < D && e0 + j < E) st[static_cast<long long>(e0 + j) * D + d] = S[i][j];
    }
}

// A few long portions are cut into spans of kStateSpan tokens that are worked on at once: what every span but the last adds to
// nothing and what it leaves of what was there, then this pass, then the read-outs from the state at the start of every span.
constexpr int kStateSpan = 512;

struct SpanParams {
  const int* seq;            // [spans], or null: every portion is one
  const int* first;          // [sequences + 1] first span of a sequence
  float* carry;              // [spans, H, E, D]: what a span adds, then the state at its start
  float* left;               // [spans, H, D or 1]: the factor that a span leaves of every column
  int n;
};

static __global__ void __launch_bounds__(256)
state_carry_kernel(SpanParams p, const float* state, const int* slots, const int* pos0, int E, int D, int per_column) {
  pdl_trigger();
  pdl_grid_wait();
  const int i = (blockIdx.x * 256 + threadIdx.x) * 4, h = blockIdx.y, H = gridDim.y, seq = blockIdx.z;
  const int first = p.first[seq], n = p.first[seq + 1] - first, slot = slots[seq];
  if (i >= E * D || n < 2 || slot < 0) return;
  const long long one = static_cast<long long>(E) * D;
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (pos0[seq] > 0) s = *reinterpret_cast<const float4*>(state + (static_cast<long long>(slot) * H + h) * one + i);
  for (int k = 0; k < n; ++k) {
    const long long at = static_cast<long long>(first + k) * H + h;
    float4* c = reinterpret_cast<float4*>(p.carry + at * one + i);
    const float4 add = k + 1 < n ? *c : make_float4(0.f, 0.f, 0.f, 0.f);
    float4 w = make_float4(0.f, 0.f, 0.f, 0.f);
    if (k + 1 < n) {
      if (per_column) w = *reinterpret_cast<const float4*>(p.left + at * D + i % D);
      else w.x = w.y = w.z = w.w = p.left[at];
    }
    *c = s;
    s = make_float4(fmaf(w.x, s.x, add.x), fmaf(w.y, s.y, add.y), fmaf(w.z, s.z, add.z), fmaf(w.w, s.w, add.w));
  }
}

}  // namespace tsb
