// Linear attention with a decay per key channel and token, for ragged batches of sequences, in two forms. Time mixing (a bonus for
// the current token, which the read-out sees otherwise):
//
//   o_t = (S_(t-1) + v_t (u k_t)^T) r_t,  S_t = diag(w_t) S_(t-1) + v_t k_t^T,  w = exp(-exp(d + w0))      per head
//
// and gated linear attention (the read-out sees the state with the current token in it):
//
//   S_t = diag(w_t) S_(t-1) + v_t k_t^T,  o_t = S_t r_t,  w = sigmoid(d + w0)^(1 / tau)
//
//   out = o / rms(o) * norm * silu(gate)
//
// S is [values][keys] in fp32 and stays so. token_shift_kernel makes the inputs of the five projections, mixes of a row and the
// one before it.
//
// Prompts in bf16 with heads of up to 128 columns run on the tensor cores (time_mix_chunk_kernel): blocks of 16 tokens, four of
// them prepared at once. With W_i the product of the decays of the block's tokens up to i, R_i = r_i W_(i-1) / W_15 and
// K_j = k_j W_15 / W_j (the product of the decays behind j),
//   S  <- S diag(W_15)
//   o_i = S R_i + sum_{j < i} (R_i . K_j) v_j + (u k_i . r_i) v_i
//   S  <- S + sum_j v_j K_j^T
// (gated: R_i = r_i W_i / W_15, and the sum takes j = i along instead of the bonus). Where a channel decays by more than 2^60 in a block, 1 / W_15 is not formed: R_i = r_i W_(i-1) (gated: W_i) meets S before it decays, and the
// pairs are summed with the decays in between, one by one. S stays in the accumulators of the products (values on rows), which is
// also the layout in which it enters the read-out. Factors that must not lose their 32 bits meet the tensor cores as two bf16 halves
// (16 bits).
// fp32 models and wider heads take time_mix_scan_kernel (token by token) and time_mix_norm_kernel; decoded tokens
// time_mix_step_kernel.
#include "linear_state.cuh"
#include "ragged_conv.cuh"

#include <algorithm>

namespace tsb {
namespace {

// ------------------------------------------------------------------ mixes of a row and the one before it
struct ShiftParams {
  const void* h;
  long long ldh;
  const float* mu;          // [n, C]
  void* last;               // [slots, C]
  void* xs;                 // [n (+ 1), rows, ldx]
  long long stream, ldx;
  const int* positions;     // [rows]
  const int* seq_of;        // [rows]
  const int* slots;         // [sequences]
  const int* cu;            // [prompts + 1] rows relative to n_decode
  const int* pos0;          // [prompts]
  int n_decode, rows, C, n, keep;
};

// A thread takes one 16-byte column of kRows rows in a row (the mix factors stay in registers).
template <typename T, int N, int kRows>
__global__ void __launch_bounds__(128)
token_shift_kernel(ShiftParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>;
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= p.C) return;
  float mu[N][V];
#pragma unroll
  for (int s = 0; s < N; ++s)
#pragma unroll
    for (int i = 0; i < V; ++i) mu[s][i] = p.mu[s * p.C + c + i];
  const T* h = static_cast<const T*>(p.h) + c;
  T* last = static_cast<T*>(p.last) + c;
  T* xs = static_cast<T*>(p.xs) + c;
  float prev[V];
  bool have = false;
  for (int r = 0; r < kRows; ++r) {
    const int row = blockIdx.y * kRows + r;
    if (row >= p.rows) return;
    float x[V];
    ld16<T>(h + row * p.ldh, x);
    const int seq = p.seq_of[row], slot = p.slots[seq];
    bool start = true, old = false;              // the sequence's first row of this step; there is an earlier token
    if (row < p.n_decode) {
      old = p.positions[row] > 0;
    } else {
      start = row == p.n_decode + p.cu[seq - p.n_decode];
      old = p.pos0[seq - p.n_decode] > 0;
    }
    if (start) {
#pragma unroll
      for (int i = 0; i < V; ++i) prev[i] = 0.f;
      if (old && slot >= 0) ld16<T>(last + static_cast<long long>(slot) * p.C, prev);
    } else if (!have) {
      ld16<T>(h + (row - 1) * p.ldh, prev);
    }
    T* out = xs + row * p.ldx;
    if (p.keep) {
      st16<T>(out, x);
      out += p.stream;
    }
#pragma unroll
    for (int s = 0; s < N; ++s) {
      float y[V];
#pragma unroll
      for (int i = 0; i < V; ++i) y[i] = fmaf(prev[i] - x[i], mu[s][i], x[i]);
      st16<T>(out + s * p.stream, y);
    }
    if (row < p.n_decode && slot >= 0) st16<T>(last + static_cast<long long>(slot) * p.C, x);
#pragma unroll
    for (int i = 0; i < V; ++i) prev[i] = x[i];
    have = true;
  }
}

// tanh of columns of a projection, 16 bytes a thread.
template <typename T>
__global__ void __launch_bounds__(256)
tanh_rows_kernel(const T* x, long long ld, T* out, int cols, long long vecs) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>;
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= vecs) return;
  const long long row = i / (cols / V);
  const int c = static_cast<int>(i % (cols / V)) * V;
  float f[V];
  ld16<T>(x + row * ld + c, f);
#pragma unroll
  for (int k = 0; k < V; ++k) f[k] = tanhf(f[k]);
  st16<T>(out + row * cols + c, f);
}

// ------------------------------------------------------------------ the recurrence
enum MixKind { kTime, kGated };

struct MixParams {
  int H, dim, dp, ep, rp, off_k, off_v, off_g, off_low, rows, n_seq, ld, ldo;    // dim: columns of a value head, ep: as stored; dp: of a key
  const void* proj;          // [rows, ld]: r, k (heads of dp columns), v, gate (of ep), time mixing: the decay's inputs
  const float* dec;          // [rows, ld_dec] (time mixing: prompts)
  long long ld_dec;
  const void* w2;            // [H * dp, rp] (time mixing, decoded rows)
  const float* w0;           // [H * dp]
  const float* u;            // [H * dp] (time mixing)
  const float* norm;         // [H * ep]
  float* state;              // [slots, H, ep, dp]
  const int* slots;
  const int* positions;      // decoded rows
  const int* cu;             // prompts
  const int* pos0;
  void* out;                 // [rows, ldo]
  float* o;                  // [rows, H, ep] read-outs of the scan
  SpanParams span;
  float eps, out_scale, r_scale, inv_tau;
};

template <int KIND, bool FAST = false>
__device__ __forceinline__ float decay_of(float x, float inv_tau) {
  if constexpr (KIND == kTime) return expf(-(FAST ? __expf(x) : expf(x)));
  return expf(-inv_tau * (fmaxf(-x, 0.f) + log1pf(FAST ? __expf(-fabsf(x)) : expf(-fabsf(x)))));
}

template <typename T, int RL, int KIND>
__global__ void __launch_bounds__(128)
time_mix_scan_kernel(MixParams p) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ float sm[ScanShape<RL>::kFloats];
  const int h = blockIdx.y, seq = blockIdx.z, slot = p.slots[seq];
  const int row0 = p.cu[seq], n = p.cu[seq + 1] - row0;
  if (slot < 0 || n <= 0) return;
  const T* x = static_cast<const T*>(p.proj) + static_cast<long long>(row0) * p.ld;
  const float* dec = p.dec + static_cast<long long>(row0) * p.ld_dec + h * p.dp;
  const float* w0 = p.w0 + h * p.dp;
  float* st = p.state + (static_cast<long long>(slot) * p.H + h) * p.ep * p.dp;
  float* o = p.o + static_cast<long long>(row0) * p.H * p.ep + h * p.ep;
  state_scan<RL, KIND == kGated>(
      sm, st, p.ep, p.dp, p.pos0[seq] == 0, n, blockIdx.x * kScanRows,
      [&](int t, int d, float& q, float& k, float& w) {
        const T* r = x + static_cast<long long>(t) * p.ld + h * p.dp + d;
        q = p.r_scale * to_f32<T>(r[0]);
        k = to_f32<T>(r[p.off_k]);
        w = decay_of<KIND>(dec[t * p.ld_dec + d] + w0[d], p.inv_tau);
      },
      [&](int t, int e) { return to_f32<T>(x[static_cast<long long>(t) * p.ld + p.off_v + h * p.ep + e]); },
      [&](int t, int e, const float (&f)[4]) {
        *reinterpret_cast<float4*>(o + static_cast<long long>(t) * p.H * p.ep + e) = make_float4(f[0], f[1], f[2], f[3]);
      });
}

// out = (o + v (u k . r)) / rms * norm * silu(gate): one warp per (row, head). Gated: without the bonus.
template <typename T, int KIND>
__global__ void __launch_bounds__(256)
time_mix_norm_kernel(MixParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const long long w = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= static_cast<long long>(p.rows) * p.H) return;
  const long long row = w / p.H;
  const int h = static_cast<int>(w % p.H);
  const T *x = static_cast<const T*>(p.proj) + row * p.ld, *v = x + p.off_v + h * p.ep, *gate = x + p.off_g + h * p.ep;
  const float *o = p.o + w * p.ep, *norm = p.norm + h * p.ep;
  T* out = static_cast<T*>(p.out) + row * p.ldo + h * p.ep;
  float bonus = 0.f, ss = 0.f;
  if constexpr (KIND == kTime) {
    const T* r = x + h * p.dp;
    const float* u = p.u + h * p.dp;
    for (int d = lane; d < p.dp; d += 32) bonus = fmaf(u[d] * to_f32<T>(r[p.off_k + d]), to_f32<T>(r[d]), bonus);
    bonus = warp_sum(bonus);
  }
  for (int d = lane; d < p.ep; d += 32) {
    const float f = fmaf(to_f32<T>(v[d]), bonus, o[d]);
    ss = fmaf(f, f, ss);
  }
  const float r = p.out_scale / sqrtf(warp_sum(ss) / static_cast<float>(p.dim) + p.eps);
  for (int d = lane; d < p.ep; d += 32) {
    const float f = fmaf(to_f32<T>(v[d]), bonus, o[d]);
    out[d] = from_f32<T>(f * r * norm[d] * silu_f32(to_f32<T>(gate[d])));
  }
}

// ------------------------------------------------------------------ prompts, bf16
template <int DT>
struct MixChunk {
  static constexpr int kTok = 64, kWarps = DT / 16, kThreads = kWarps * 32, kParts = DT / 64;
  static constexpr int kLd = DT + 8, kLdO = DT + 4;
  // bytes of a stage: r (its place is taken by the high half of the decayed r), k likewise, v, decay inputs (by the read-outs)
  static constexpr int kTile = kTok * kLd * 2, kR = 0, kK = kTile, kV = 2 * kTile, kO = 3 * kTile, kStage = kO + kTok * kLdO * 4;
  // what exists once: the low halves, the pair products, the blocks' decays, the bonus of every token
  static constexpr int kRl = 2 * kStage, kKl = kRl + kTile, kA = kKl + kTile, kTot = kA + kParts * 4096, kBonus = kTot + 4 * DT * 4;
  static constexpr int kSmem = kBonus + kParts * kTok * 4;
};
constexpr float kSteep = 8.6736174e-19f;       // 2^-60: a block that decays a channel further takes the slow pair products

// Sums of N values over the warp, N a power of two: lane l returns the sum of v[l % N].
template <int N>
__device__ __forceinline__ float transpose_sum(float (&v)[N], int lane) {
#pragma unroll
  for (int o = N / 2; o; o >>= 1) {
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
      if (i >= o) break;
      const float keep = up ? v[i + o] : v[i], give = up ? v[i] : v[i + o];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
#pragma unroll
  for (int o = N; o < 32; o <<= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
  return v[0];
}

// CTA = (head, sequence or span); warp w owns the state's rows (values) 16 w .. + 15. The next 64 tokens arrive while some are
// worked on. OUT = false: only what a span adds and leaves.
template <int DT, bool OUT, int KIND>
__global__ void __launch_bounds__(MixChunk<DT>::kThreads, DT == 64 ? 2 : 1)
time_mix_chunk_kernel(MixParams p) {
  using T = __nv_bfloat16;
  using C = MixChunk<DT>;
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  T *srl = reinterpret_cast<T*>(smem + C::kRl), *skl = reinterpret_cast<T*>(smem + C::kKl);
  float *sa = reinterpret_cast<float*>(smem + C::kA), *stot = reinterpret_cast<float*>(smem + C::kTot);
  float* sbonus = reinterpret_cast<float*>(smem + C::kBonus);
  const int h = blockIdx.x, seq = p.span.seq ? p.span.seq[blockIdx.y] : blockIdx.y, slot = p.slots[seq];
  int row0 = p.cu[seq], n = p.cu[seq + 1] - row0, idx = 0, spans = 1;
  if (p.span.seq) {
    idx = blockIdx.y - p.span.first[seq];
    spans = p.span.first[seq + 1] - p.span.first[seq];
    row0 += idx * kStateSpan;
    n = min(kStateSpan, n - idx * kStateSpan);
  }
  const bool last = idx == spans - 1;
  if (slot < 0 || n <= 0 || (!OUT && last)) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const T* proj = static_cast<const T*>(p.proj) + static_cast<long long>(row0) * p.ld;
  float* carry = spans > 1 ? p.span.carry + (static_cast<long long>(blockIdx.y) * p.H + h) * p.ep * p.dp : nullptr;
  const float* dec = p.dec + static_cast<long long>(row0) * p.ld_dec + h * p.dp;
  float* st = p.state + (static_cast<long long>(slot) * p.H + h) * p.ep * p.dp;
  const int e0 = warp * 16;
  auto issue = [&](int t0) {
    uint8_t* stage = smem + (t0 / C::kTok & 1) * C::kStage;
    const uint32_t base = smem_u32(stage);
    const int cnt = min(C::kTok, n - t0);
    for (int i = tid; i < C::kTok * (DT / 8); i += C::kThreads) {
      const int r = i / (DT / 8), d = (i % (DT / 8)) * 8;
      const bool key = r < cnt && d < p.dp, val = r < cnt && d < p.ep;
      const T* src = proj + static_cast<long long>(r < cnt ? t0 + r : 0) * p.ld + d;
      const uint32_t at = base + (r * C::kLd + d) * 2;
      if constexpr (OUT) cp_async_16(at + C::kR, key ? src + h * p.dp : proj, key ? 16 : 0);
      cp_async_16(at + C::kK, key ? src + p.off_k + h * p.dp : proj, key ? 16 : 0);
      cp_async_16(at + C::kV, val ? src + p.off_v + h * p.ep : proj, val ? 16 : 0);
    }
    for (int i = tid; i < C::kTok * (DT / 4); i += C::kThreads) {
      const int r = i / (DT / 4), d = (i % (DT / 4)) * 4;
      const bool ok = r < cnt && d < p.dp;
      cp_async_16(base + C::kO + (r * C::kLdO + d) * 4, ok ? dec + (t0 + r) * p.ld_dec + d : dec, ok ? 16 : 0);
    }
    cp_commit();
  };
  issue(0);
  float S[DT / 8][4];
  {
    const float* from = !OUT ? nullptr : carry ? carry : p.pos0[seq] > 0 ? st : nullptr;
#pragma unroll
    for (int j = 0; j < DT / 8; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = e0 + g + 8 * e, c = j * 8 + 2 * t4;
        float2 v = make_float2(0.f, 0.f);
        if (from && r < p.ep && c < p.dp) v = *reinterpret_cast<const float2*>(from + static_cast<long long>(r) * p.dp + c);
        S[j][2 * e] = v.x;
        S[j][2 * e + 1] = v.y;
      }
  }
  // this thread's share of the preparation: two channels of one block of 16 tokens
  const int blk = warp / C::kParts, part = warp % C::kParts, d0 = part * 64 + lane * 2;
  constexpr bool kOwn = KIND == kGated;                      // token i sees its own key and value like the others
  float w0[2] = {}, uu[2] = {};
  if (d0 < p.dp) {
    w0[0] = p.w0[h * p.dp + d0];
    w0[1] = p.w0[h * p.dp + d0 + 1];
    if constexpr (KIND == kTime) {
      uu[0] = p.u[h * p.dp + d0];
      uu[1] = p.u[h * p.dp + d0 + 1];
    }
  }
  const uint32_t aRl = smem_u32(srl), aKl = smem_u32(skl);
  // rows of the epilogue: kLanes lanes of four columns share one
  constexpr int kLanes = DT / 4, kPer = 32 / kLanes, kIter = C::kTok / (C::kWarps * kPer);
  const int er = warp * kPer + lane / kLanes, ec = lane % kLanes * 4;

  float left = 1.f;                                          // (OUT = false) what the span leaves of column tid
  for (int t0 = 0; t0 < n; t0 += C::kTok) {
    const int cnt = min(C::kTok, n - t0);
    uint8_t* stage = smem + (t0 / C::kTok & 1) * C::kStage;
    T *sr = reinterpret_cast<T*>(stage + C::kR), *sk = reinterpret_cast<T*>(stage + C::kK), *sv = reinterpret_cast<T*>(stage + C::kV);
    float* so = reinterpret_cast<float*>(stage + C::kO);
    const uint32_t aR = smem_u32(sr), aK = smem_u32(sk), aV = smem_u32(sv);
    cp_wait<0>();
    __syncthreads();
    if (t0 + C::kTok < n) issue(t0 + C::kTok);
    bool steep;
    {
      __nv_bfloat162 r[16], k[16];
      float w[16][2];
      const int row = blk * 16;
      float tot[2] = {1.f, 1.f}, bonus[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        if constexpr (OUT) r[i] = *reinterpret_cast<const __nv_bfloat162*>(sr + (row + i) * C::kLd + d0);
        k[i] = *reinterpret_cast<const __nv_bfloat162*>(sk + (row + i) * C::kLd + d0);
        const float2 dv = *reinterpret_cast<const float2*>(so + (row + i) * C::kLdO + d0);
        const bool real = row + i < cnt;                     // (a token that is not there decays nothing)
        w[i][0] = real ? decay_of<KIND, true>(dv.x + w0[0], p.inv_tau) : 1.f;
        w[i][1] = real ? decay_of<KIND, true>(dv.y + w0[1], p.inv_tau) : 1.f;
        tot[0] *= w[i][0];
        tot[1] *= w[i][1];
        if constexpr (OUT && !kOwn)
          bonus[i] = fmaf(__low2float(r[i]) * uu[0], __low2float(k[i]), __high2float(r[i]) * uu[1] * __high2float(k[i]));
      }
      float f[2] = {p.r_scale, p.r_scale};
      steep = false;
      if constexpr (OUT) {
        if constexpr (!kOwn) {
          const float b = transpose_sum<16>(bonus, lane);
          if (lane < 16) sbonus[part * C::kTok + row + lane] = b;
        }
        steep = __syncthreads_or(tot[0] < kSteep || tot[1] < kSteep) != 0;
        if (!steep) {
          f[0] /= tot[0];
          f[1] /= tot[1];
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int at = (row + i) * C::kLd + d0;
          if constexpr (kOwn) {
            f[0] *= w[i][0];
            f[1] *= w[i][1];
          }
          split_bf16x2(__low2float(r[i]) * f[0], __high2float(r[i]) * f[1], reinterpret_cast<uint32_t*>(sr + at), reinterpret_cast<uint32_t*>(srl + at));
          if constexpr (!kOwn) {
            f[0] *= w[i][0];
            f[1] *= w[i][1];
          }
        }
      }
      *reinterpret_cast<float2*>(stot + blk * DT + d0) = make_float2(tot[0], tot[1]);
      f[0] = f[1] = 1.f;
#pragma unroll
      for (int i = 15; i >= 0; --i) {
        const int at = (row + i) * C::kLd + d0;
        split_bf16x2(__low2float(k[i]) * f[0], __high2float(k[i]) * f[1], reinterpret_cast<uint32_t*>(sk + at), reinterpret_cast<uint32_t*>(skl + at));
        f[0] *= w[i][0];
        f[1] *= w[i][1];
      }
      if (OUT && steep) {
        // what token i takes of token j's value, two j at a time: the decays in between, one by one
        float* a = sa + (part * 4 + blk) * 256;
#pragma unroll
        for (int jj = 0; jj < 16; jj += 2) {
          float v[32];
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const int j = jj + q;
            float x0 = __low2float(k[j]) * p.r_scale, x1 = __high2float(k[j]) * p.r_scale;
#pragma unroll
            for (int i = 0; i < 16; ++i) {
              v[q * 16 + i] = 0.f;
              if (i < j + !kOwn) continue;
              if (kOwn && i > j) {
                x0 *= w[i][0];
                x1 *= w[i][1];
              }
              v[q * 16 + i] = fmaf(__low2float(r[i]), x0, __high2float(r[i]) * x1);
              if (!kOwn) {
                x0 *= w[i][0];
                x1 *= w[i][1];
              }
            }
          }
          a[(jj + (lane >> 4)) * 16 + (lane & 15)] = transpose_sum<32>(v, lane);
        }
      }
    }
    if (OUT && C::kParts > 1) __syncthreads();
    else __syncwarp();
    if (OUT && !steep && warp < 4) {
      // the same from the prepared factors: rows i, columns j; this layout is also that of the operand it becomes
      float c[3][2][4] = {};
      const int row = warp * 16;
#pragma unroll
      for (int ks = 0; ks < DT / 16; ++ks) {
        uint32_t qh[4], ql[4], kh[4], kl[4];
        ldmat_x4(qh, aR + frag_a(lane, row, ks * 16, C::kLd));
        ldmat_x4(ql, aRl + frag_a(lane, row, ks * 16, C::kLd));
        ldmat_x4(kh, aK + frag_b(lane, row, ks * 16, C::kLd));
        ldmat_x4(kl, aKl + frag_b(lane, row, ks * 16, C::kLd));
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          mma_bf16(c[0][j], qh, kh[2 * j], kh[2 * j + 1]);
          mma_bf16(c[1][j], ql, kh[2 * j], kh[2 * j + 1]);
          mma_bf16(c[2][j], qh, kl[2 * j], kl[2 * j + 1]);
        }
      }
      uint32_t* frag = reinterpret_cast<uint32_t*>(sa) + warp * 256;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {                        // rows i = g + 8 e, columns j 8 + 2 t, + 1
          float x[2];
#pragma unroll
          for (int q = 0; q < 2; ++q)
            x[q] = j * 8 + 2 * t4 + q < g + 8 * e + kOwn ? c[0][j][2 * e + q] + (c[1][j][2 * e + q] + c[2][j][2 * e + q]) : 0.f;
          uint32_t hi, lo;
          split_bf16x2(x[0], x[1], &hi, &lo);
          frag[(e * 4 + j) * 32 + lane] = hi;
          frag[(e * 4 + 2 + j) * 32 + lane] = lo;
        }
    }
    __syncthreads();
    if (!OUT && tid < DT) left *= (stot[tid] * stot[DT + tid]) * (stot[2 * DT + tid] * stot[3 * DT + tid]);
    uint2 gate[kIter];                                       // requested before the products
#pragma unroll
    for (int i = 0; i < kIter; ++i) {
      if (!OUT) break;
      const int r = min(i * C::kWarps * kPer + er, cnt - 1);
      gate[i] = *reinterpret_cast<const uint2*>(proj + static_cast<long long>(t0 + r) * p.ld + p.off_g + h * p.ep + min(ec, p.ep - 4));
    }
#pragma unroll 1
    for (int b = 0; b < 4; ++b) {
      if (b * 16 >= cnt) break;
      const int row = b * 16;
      if (!steep) {
#pragma unroll
        for (int j = 0; j < DT / 8; ++j) {
          const float2 f = *reinterpret_cast<const float2*>(stot + b * DT + j * 8 + 2 * t4);
          S[j][0] *= f.x; S[j][1] *= f.y; S[j][2] *= f.x; S[j][3] *= f.y;
        }
      }
      float acc[3][2][4] = {};
#pragma unroll
      for (int ks = 0; ks < DT / 16; ++ks) {
        if (!OUT) break;
        uint32_t hi[4], lo[4], qh[4], ql[4];
        split_bf16x2(S[2 * ks][0], S[2 * ks][1], &hi[0], &lo[0]);
        split_bf16x2(S[2 * ks][2], S[2 * ks][3], &hi[1], &lo[1]);
        split_bf16x2(S[2 * ks + 1][0], S[2 * ks + 1][1], &hi[2], &lo[2]);
        split_bf16x2(S[2 * ks + 1][2], S[2 * ks + 1][3], &hi[3], &lo[3]);
        ldmat_x4(qh, aR + frag_b(lane, row, ks * 16, C::kLd));
        ldmat_x4(ql, aRl + frag_b(lane, row, ks * 16, C::kLd));
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          mma_bf16(acc[0][c], hi, qh[2 * c], qh[2 * c + 1]);
          mma_bf16(acc[1][c], lo, qh[2 * c], qh[2 * c + 1]);
          mma_bf16(acc[2][c], hi, ql[2 * c], ql[2 * c + 1]);
        }
      }
      uint32_t vt[4];
      ldmat_x4_trans(vt, aV + frag_a_trans(lane, row, e0, C::kLd));
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        if (!OUT) break;
        uint32_t hi[2], lo[2];
        if (!steep) {
          const uint32_t* frag = reinterpret_cast<const uint32_t*>(sa) + b * 256 + c * 128 + lane;
          hi[0] = frag[0]; hi[1] = frag[32]; lo[0] = frag[64]; lo[1] = frag[96];
        } else {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float x[2] = {};
#pragma unroll
            for (int q = 0; q < C::kParts; ++q) {
              const float* a = sa + (q * 4 + b) * 256 + (e * 8 + 2 * t4) * 16 + c * 8 + g;
              x[0] += a[0];
              x[1] += a[16];
            }
            split_bf16x2(x[0], x[1], &hi[e], &lo[e]);
          }
        }
        mma_bf16(acc[0][c], vt, hi[0], hi[1]);
        mma_bf16(acc[1][c], vt, lo[0], lo[1]);
#pragma unroll
        for (int e = 0; e < 4; ++e)
          so[(row + c * 8 + 2 * t4 + (e & 1)) * C::kLdO + e0 + g + 8 * (e >> 1)] = acc[0][c][e] + (acc[1][c][e] + acc[2][c][e]);
      }
#pragma unroll
      for (int j = 0; j < DT / 8; j += 2) {
        uint32_t kh[4], kl[4];
        ldmat_x4_trans(kh, aK + frag_b_trans(lane, row, j * 8, C::kLd));
        ldmat_x4_trans(kl, aKl + frag_b_trans(lane, row, j * 8, C::kLd));
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          if (steep) {
            const float2 f = *reinterpret_cast<const float2*>(stot + b * DT + (j + c) * 8 + 2 * t4);
            S[j + c][0] *= f.x; S[j + c][1] *= f.y; S[j + c][2] *= f.x; S[j + c][3] *= f.y;
          }
          mma_bf16(S[j + c], vt, kh[2 * c], kh[2 * c + 1]);
          mma_bf16(S[j + c], vt, kl[2 * c], kl[2 * c + 1]);
        }
      }
    }
    __syncthreads();
    if (!OUT) continue;
    // bonus, norm and gate
    float4 nm = make_float4(0.f, 0.f, 0.f, 0.f);
    if (ec < p.ep) nm = *reinterpret_cast<const float4*>(p.norm + h * p.ep + ec);
#pragma unroll
    for (int i = 0; i < kIter; ++i) {
      const int r = i * C::kWarps * kPer + er;
      float4 o = *reinterpret_cast<const float4*>(so + r * C::kLdO + ec);
      if constexpr (!kOwn) {
        float bonus = sbonus[r];
        if (C::kParts > 1) bonus += sbonus[C::kTok + r];
        const uint2 vv = *reinterpret_cast<const uint2*>(sv + r * C::kLd + ec);
        const __nv_bfloat162 va = *reinterpret_cast<const __nv_bfloat162*>(&vv.x), vb = *reinterpret_cast<const __nv_bfloat162*>(&vv.y);
        o.x = fmaf(bonus, __low2float(va), o.x); o.y = fmaf(bonus, __high2float(va), o.y);
        o.z = fmaf(bonus, __low2float(vb), o.z); o.w = fmaf(bonus, __high2float(vb), o.w);
      }
      float ss = fmaf(o.x, o.x, fmaf(o.y, o.y, fmaf(o.z, o.z, o.w * o.w)));
#pragma unroll
      for (int m = kLanes / 2; m; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
      if (r >= cnt || ec >= p.ep) continue;
      const float rs = p.out_scale * rsqrtf(ss / static_cast<float>(p.dim) + p.eps);
      const __nv_bfloat162 ga = *reinterpret_cast<const __nv_bfloat162*>(&gate[i].x), gb = *reinterpret_cast<const __nv_bfloat162*>(&gate[i].y);
      auto silu = [](float x) { return __fdividef(x, 1.f + __expf(-x)); };
      *reinterpret_cast<uint2*>(static_cast<T*>(p.out) + static_cast<long long>(row0 + t0 + r) * p.ldo + h * p.ep + ec) =
          make_uint2(pack_bf16x2(o.x * rs * nm.x * silu(__low2float(ga)), o.y * rs * nm.y * silu(__high2float(ga))),
                     pack_bf16x2(o.z * rs * nm.z * silu(__low2float(gb)), o.w * rs * nm.w * silu(__high2float(gb))));
    }
    __syncthreads();
  }
  float* to = !OUT ? carry : last ? st : nullptr;
  if (!to) return;
  if (!OUT && tid < p.dp) p.span.left[(static_cast<long long>(blockIdx.y) * p.H + h) * p.dp + tid] = left;
#pragma unroll
  for (int j = 0; j < DT / 8; ++j)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = e0 + g + 8 * e, c = j * 8 + 2 * t4;
      if (r < p.ep && c < p.dp) *reinterpret_cast<float2*>(to + static_cast<long long>(r) * p.dp + c) = make_float2(S[j][2 * e], S[j][2 * e + 1]);
    }
}

// Decoded rows: CTA = (row, head). The state is requested first, the decays are worked out while it arrives.
template <typename T, int LPR, int PPL, int RPT, int KIND>
__global__ void __launch_bounds__(256)
time_mix_step_kernel(MixParams p) {
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ __align__(16) float sm[];
  float *sq = sm, *sk = sq + p.dp, *sw = sk + p.dp, *sv = sw + p.dp, *so = sv + p.ep, *th = so + p.ep, *red = th + p.rp;
  const int row = blockIdx.x, h = blockIdx.y, slot = p.slots[row];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const T* x = static_cast<const T*>(p.proj) + static_cast<long long>(row) * p.ld;
  T* out = static_cast<T*>(p.out) + static_cast<long long>(row) * p.ldo + h * p.ep;
  if (slot < 0) {
    for (int d = tid; d < p.ep; d += 256) out[d] = from_f32<T>(0.f);
    return;
  }
  StateStep<LPR, PPL, RPT, KIND == kGated> step(p.state + (static_cast<long long>(slot) * p.H + h) * p.ep * p.dp, p.ep, p.dp, p.positions[row] <= 0);
  float bonus = 0.f;
  for (int d = tid; d < p.dp; d += 256) {
    sq[d] = p.r_scale * to_f32<T>(x[h * p.dp + d]);
    sk[d] = to_f32<T>(x[p.off_k + h * p.dp + d]);
    if constexpr (KIND == kTime) bonus = fmaf(p.u[h * p.dp + d] * sk[d], sq[d], bonus);
    else sw[d] = decay_of<KIND>(p.dec[row * p.ld_dec + h * p.dp + d] + p.w0[h * p.dp + d], p.inv_tau);
  }
  for (int e = tid; e < p.ep; e += 256) sv[e] = to_f32<T>(x[p.off_v + h * p.ep + e]);
  if constexpr (KIND == kTime) {
    const T* wl = x + p.off_low;
    for (int j = tid; j < p.rp; j += 256) th[j] = to_f32<T>(from_f32<T>(tanhf(to_f32<T>(wl[j]))));
    bonus = warp_sum(bonus);
    if (lane == 0) red[warp] = bonus;
    __syncthreads();
    // four lanes per channel, 16 bytes of its row of the matrix at a time
    constexpr int V = kVec16<T>;
    const T* w2 = static_cast<const T*>(p.w2) + static_cast<long long>(h) * p.dp * p.rp;
    for (int d = tid >> 2; d < p.dp; d += 64) {            // (dp is a multiple of 16: a warp's eight channels exist or do not)
      float a = 0.f;
      for (int j = (tid & 3) * V; j < p.rp; j += 4 * V) {
        float f[V];
        ld16<T>(w2 + static_cast<long long>(d) * p.rp + j, f);
#pragma unroll
        for (int i = 0; i < V; ++i) a = fmaf(f[i], th[j + i], a);
      }
      a += __shfl_xor_sync(0xffffffffu, a, 1);
      a += __shfl_xor_sync(0xffffffffu, a, 2);
      if ((tid & 3) == 0) sw[d] = decay_of<KIND>(a + p.w0[h * p.dp + d], 1.f);
    }
    bonus = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) bonus += red[w];
  }
  __syncthreads();
  step.run(sq, sk, sw, sv, so);
  __syncthreads();
  float ss = 0.f;
  for (int d = tid; d < p.ep; d += 256) {
    const float f = fmaf(sv[d], bonus, so[d]);
    ss = fmaf(f, f, ss);
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) ss += red[w];
  const float r = p.out_scale / sqrtf(ss / static_cast<float>(p.dim) + p.eps);
  for (int d = tid; d < p.ep; d += 256)
    out[d] = from_f32<T>(fmaf(sv[d], bonus, so[d]) * r * p.norm[h * p.ep + d] * silu_f32(to_f32<T>(x[p.off_g + h * p.ep + d])));
}

template <typename T, int KIND>
int run_scan(const MixParams& p, cudaStream_t s) {
  const dim3 grid((p.ep + kScanRows - 1) / kScanRows, p.H, p.n_seq);
  const bool pdl = pdl_all_enabled();
  if (p.dp <= 64) launch_pdl(time_mix_scan_kernel<T, 2, KIND>, grid, dim3(128), 0, s, pdl, p);
  else if (p.dp <= 128) launch_pdl(time_mix_scan_kernel<T, 4, KIND>, grid, dim3(128), 0, s, pdl, p);
  else launch_pdl(time_mix_scan_kernel<T, 8, KIND>, grid, dim3(128), 0, s, pdl, p);
  const long long warps = static_cast<long long>(p.rows) * p.H;
  launch_pdl(time_mix_norm_kernel<T, KIND>, dim3(static_cast<unsigned>((warps + 7) / 8)), dim3(256), 0, s, pdl, p);
  return static_cast<int>(cudaGetLastError());
}

template <int DT, bool OUT, int KIND>
int launch_chunk(const MixParams& p, cudaStream_t s) {
  auto kern = time_mix_chunk_kernel<DT, OUT, KIND>;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MixChunk<DT>::kSmem);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  launch_pdl(kern, dim3(p.H, p.span.seq ? p.span.n : p.n_seq), dim3(MixChunk<DT>::kThreads), MixChunk<DT>::kSmem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <int DT, int KIND>
int run_chunk(const MixParams& p, cudaStream_t s) {
  if (p.span.seq) {
    if (const int rc = launch_chunk<DT, false, KIND>(p, s)) return rc;
    launch_pdl(state_carry_kernel, dim3((p.ep * p.dp / 4 + 255) / 256, p.H, p.n_seq), dim3(256), 0, s, pdl_all_enabled(), p.span,
               static_cast<const float*>(p.state), p.slots, p.pos0, p.ep, p.dp, 1);
  }
  return launch_chunk<DT, true, KIND>(p, s);
}

template <typename T, int KIND>
int run_step(const MixParams& p, cudaStream_t s) {
  const int smem = (3 * p.dp + 2 * p.ep + p.rp + 8) * 4;
  if (smem > 48 * 1024) return -2;
  const dim3 grid(p.rows, p.H);
  const bool pdl = pdl_all_enabled();
  if (p.dp <= 32) launch_pdl(time_mix_step_kernel<T, 8, 1, 1, KIND>, grid, dim3(256), smem, s, pdl, p);
  else if (p.dp <= 64) launch_pdl(time_mix_step_kernel<T, 16, 1, 4, KIND>, grid, dim3(256), smem, s, pdl, p);
  else if (p.dp <= 128) launch_pdl(time_mix_step_kernel<T, 32, 1, 16, KIND>, grid, dim3(256), smem, s, pdl, p);
  else launch_pdl(time_mix_step_kernel<T, 32, 2, 8, KIND>, grid, dim3(256), smem, s, pdl, p);
  return static_cast<int>(cudaGetLastError());
}

// ints: H, dim, dp, ep, rp, off_k, off_v, off_g, off_low, rows, sequences, row strides of the projection, the result and the decays, kind
// (0 time mixing, 1 gated linear attention); floats: eps, out_scale, r_scale, 1 / tau
bool read_mix(const int* v, const float* f, MixParams* p, int* kind) {
  p->H = v[0]; p->dim = v[1]; p->dp = v[2]; p->ep = v[3]; p->rp = v[4]; p->off_k = v[5]; p->off_v = v[6]; p->off_g = v[7]; p->off_low = v[8];
  p->rows = v[9]; p->n_seq = v[10]; p->ld = v[11]; p->ldo = v[12]; p->ld_dec = v[13];
  *kind = v[14];
  p->eps = f[0]; p->out_scale = f[1]; p->r_scale = f[2]; p->inv_tau = f[3];
  return p->H > 0 && p->H <= 65535 && p->dim > 0 && p->ep >= p->dim && p->ep % 16 == 0 && p->dp > 0 && p->dp % 16 == 0 && p->dp <= 256 && p->rp >= 0 &&
         p->rp % 16 == 0 && p->off_k % 8 == 0 && p->off_v % 8 == 0 && p->off_g % 8 == 0 && p->off_low % 8 == 0 && p->rows > 0 && p->ld % 8 == 0 &&
         p->ld_dec % 4 == 0 && p->n_seq > 0 && p->n_seq <= 65535 && (*kind == kTime || *kind == kGated);
}

template <typename T, int N>
void launch_shift(const ShiftParams& p, cudaStream_t s) {
  const int cols = (p.C / kVec16<T> + 127) / 128;
  if (p.rows <= 512) launch_pdl(token_shift_kernel<T, N, 1>, dim3(cols, p.rows), dim3(128), 0, s, pdl_all_enabled(), p);
  else launch_pdl(token_shift_kernel<T, N, 8>, dim3(cols, (p.rows + 7) / 8), dim3(128), 0, s, pdl_all_enabled(), p);
}

template <typename T>
int run_shift(const ShiftParams& p, int n_prompts, cudaStream_t s) {
  switch (p.n) {
    case 1: launch_shift<T, 1>(p, s); break;
    case 5: launch_shift<T, 5>(p, s); break;
    default: return -2;
  }
  if (n_prompts > 0)       // a portion's last row: behind the reads of the one before it
    launch_pdl(conv_state_kernel<T>, dim3((p.C + 255) / 256, n_prompts), dim3(256), 0, s, pdl_all_enabled(),
               static_cast<const T*>(p.h) + p.n_decode * p.ldh, p.ldh, p.C, static_cast<T*>(p.last), p.cu, p.slots + p.n_decode, p.pos0, 1);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace
}  // namespace tsb

// See ShiftParams. Rows below n_decode are single tokens, the others portions. C is a multiple of 8; n is 1 or 5.
TSB_EXPORT int tsb_token_shift(const void* h, long long ldh, const float* mu, void* last, void* xs, long long stream_elems, long long ldx,
                               const int* positions, const int* seq_of, const int* slots, const int* cu, const int* pos0, int n_decode, int rows,
                               int C, int n, int keep, int n_prompts, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || C <= 0 || C % 8 || ldh % 8 || ldx % 8 || stream_elems % 8 || n_prompts < 0 || n_prompts > 65535 || n_decode < 0 ||
      n_decode > rows || (rows > n_decode && (!cu || !pos0 || n_prompts == 0)))
    return -2;
  ShiftParams p{h, ldh, mu, last, xs, stream_elems, ldx, positions, seq_of, slots, cu, pos0, n_decode, rows, C, n, keep};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) return run_shift<__nv_bfloat16>(p, n_prompts, s);
  if (dtype == 0) return run_shift<float>(p, n_prompts, s);
  return -2;
}

// out [rows, cols] = tanh of x's first `cols` columns (row stride ld); cols and ld are multiples of 8.
TSB_EXPORT int tsb_tanh_rows(const void* x, long long ld, void* out, int rows, int cols, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || cols <= 0 || cols % 8 || ld % 8 || (dtype != 0 && dtype != 1) || (reinterpret_cast<uintptr_t>(x) & 15)) return -2;
  const long long vecs = static_cast<long long>(rows) * cols / (dtype == 1 ? 8 : 4);
  const dim3 grid(static_cast<unsigned>((vecs + 255) / 256));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1)
    launch_pdl(tanh_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const __nv_bfloat16*>(x), ld,
               static_cast<__nv_bfloat16*>(out), cols, vecs);
  else
    launch_pdl(tanh_rows_kernel<float>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const float*>(x), ld, static_cast<float*>(out), cols, vecs);
  return static_cast<int>(cudaGetLastError());
}

// ints and floats: see read_mix. ptrs: proj, w2, w0, u, norm, state, slots, positions, out, dec (time mixing: w2 and u, gated: dec). Row i is
// the next token of the sequence in slot slots[i] (-1: padding, out = 0).
TSB_EXPORT int tsb_time_mix_step(const int* ints, const float* floats, void* const* q, int dtype, void* stream) {
  using namespace tsb;
  MixParams p{};
  int kind;
  if (!read_mix(ints, floats, &p, &kind)) return -2;
  p.proj = q[0]; p.w2 = q[1]; p.w0 = static_cast<const float*>(q[2]); p.u = static_cast<const float*>(q[3]);
  p.norm = static_cast<const float*>(q[4]); p.state = static_cast<float*>(q[5]); p.slots = static_cast<const int*>(q[6]);
  p.positions = static_cast<const int*>(q[7]); p.out = q[8]; p.dec = static_cast<const float*>(q[9]);
  if (kind == kTime ? (!p.w2 || !p.u || p.rp <= 0) : !p.dec) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) return kind == kTime ? run_step<__nv_bfloat16, kTime>(p, s) : run_step<__nv_bfloat16, kGated>(p, s);
  if (dtype == 0) return kind == kTime ? run_step<float, kTime>(p, s) : run_step<float, kGated>(p, s);
  return -2;
}

// ptrs: proj, dec, w0, u, norm, state, slots, cu, pos0, out, o ([rows, H, ep] fp32; null: bf16 on the tensor cores, dp and ep <= 128), and for
// `spans` spans of 512 tokens (0: every portion is walked in one): their sequences, the first span of every sequence, carry [spans, H,
// ep, dp], left [spans, H, dp].
TSB_EXPORT int tsb_time_mix_prefill(const int* ints, const float* floats, void* const* q, int spans, int dtype, void* stream) {
  using namespace tsb;
  MixParams p{};
  int kind;
  if (!read_mix(ints, floats, &p, &kind)) return -2;
  p.proj = q[0]; p.dec = static_cast<const float*>(q[1]); p.w0 = static_cast<const float*>(q[2]); p.u = static_cast<const float*>(q[3]);
  p.norm = static_cast<const float*>(q[4]); p.state = static_cast<float*>(q[5]); p.slots = static_cast<const int*>(q[6]);
  p.cu = static_cast<const int*>(q[7]); p.pos0 = static_cast<const int*>(q[8]); p.out = q[9]; p.o = static_cast<float*>(q[10]);
  if (!p.dec || (kind == kTime && !p.u)) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (!p.o) {
    if (spans > 0) {
      p.span = {static_cast<const int*>(q[11]), static_cast<const int*>(q[12]), static_cast<float*>(q[13]), static_cast<float*>(q[14]), spans};
      if (spans > 65535 || !p.span.seq || !p.span.first || !p.span.carry || !p.span.left) return -2;
    }
    const int wide = std::max(p.dp, p.ep);
    if (dtype != 1 || wide > 128 || p.ldo % 4 || (reinterpret_cast<uintptr_t>(p.out) & 7)) return -2;
    if (kind == kTime) return wide <= 64 ? run_chunk<64, kTime>(p, s) : run_chunk<128, kTime>(p, s);
    return wide <= 64 ? run_chunk<64, kGated>(p, s) : run_chunk<128, kGated>(p, s);
  }
  if (dtype == 1) return kind == kTime ? run_scan<__nv_bfloat16, kTime>(p, s) : run_scan<__nv_bfloat16, kGated>(p, s);
  if (dtype == 0) return kind == kTime ? run_scan<float, kTime>(p, s) : run_scan<float, kGated>(p, s);
  return -2;
}
