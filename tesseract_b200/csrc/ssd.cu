// State-space duality (a matrix state per head with a scalar decay per token), for ragged batches:
//
//   S_t = exp(-exp(A_log) dt) S_(t-1) + (dt x_t) B_t^T,  y_t = S_t C_t + D x_t                      per head, S [vdim][state]
//   out = y * silu(z), normed in equal parts (part_norm_kernel)
//
// x, B and C pass a short causal convolution with bias and SiLU (ssd_conv_kernel, which also turns the dt projection into dt and
// the logarithm of the decay); heads share the B and C of their group. The state and what decays it are fp32.
//
// Prompts in bf16 run on the tensor cores in the chunked form (ssd_chunk_kernel), 64 tokens at a time, L_i the sum of the
// logarithms up to token i of the chunk:
//   y_i = exp(L_i) S C_i + sum_{j <= i} exp(L_i - L_j) dt_j (B_j . C_i) x_j + D x_i
//   S  <- exp(L_63) S + sum_j (exp(L_63 - L_j) dt_j x_j) B_j^T
// S stays in the accumulators of the products (values on rows), which is also the layout in which it enters the read-out. S, the
// decayed scores and the decayed x go in as two bf16 halves (16 bits); B, C and x are bf16 as the convolution leaves them.
// fp32 models take ssd_scan_kernel (token by token), decoded tokens ssd_step_kernel.
#include "linear_state.cuh"
#include "ragged_conv.cuh"

#include <algorithm>

namespace tsb {
namespace {

constexpr int kBlk = 16;           // tokens of a portion that a thread of the convolution walks

struct SsdParams {
  int H, vdim, vp, N, np, G, taps, rows, n_decode, n_seq, blocks, ld, ldo;
  int off_x, off_b, off_c, off_dt, conv_c;      // sections of a projection row (z starts at 0), convolved columns
  const void* proj;          // [rows, ld]
  const float* conv_w;       // [taps, conv_c]
  const float* conv_b;       // [conv_c]
  const float* a_log;        // [H]
  const float* dt_bias;      // [H]
  void* conv_state;          // [slots, taps - 1, conv_c]
  void* xbc;                 // [rows, conv_c]
  float2* gates;             // [rows, H]: dt, log2 of the decay
  const float* d;            // [H]
  float* state;              // [slots, H, vp, np]
  const int* slots;          // decoded rows, then prompts
  const int* positions;
  const int* cu;             // prompts, relative to n_decode
  const int* pos0;
  const int* blk_seq;
  const int* blk0;
  void* out;                 // [rows, ldo]: y
  SpanParams span;
};

__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// A thread takes 16 bytes of columns of one decoded row or of a tile of up to kBlk tokens of a portion; the last column blocks take
// the heads' step sizes.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
ssd_conv_kernel(SsdParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>, TAIL = TAPS - 1;
  const int conv_blocks = (p.conv_c / V + 127) / 128;
  const bool decode = static_cast<int>(blockIdx.y) < p.n_decode;
  int row, cnt = 1, before = 0, slot;            // first row, its tokens, tokens of this portion in front of it
  bool old;                                      // the slot's tail belongs to this sequence
  if (decode) {
    row = blockIdx.y;
    slot = p.slots[row];
    old = p.positions[row] > 0;
  } else {
    const int blk = blockIdx.y - p.n_decode, seq = p.blk_seq[blk];
    before = (blk - p.blk0[seq]) * kBlk;
    row = p.n_decode + p.cu[seq] + before;
    cnt = min(kBlk, p.cu[seq + 1] - p.cu[seq] - before);
    slot = p.slots[p.n_decode + seq];
    old = p.pos0[seq] > 0;
  }
  const T* proj = static_cast<const T*>(p.proj) + static_cast<long long>(row) * p.ld;
  if (static_cast<int>(blockIdx.x) >= conv_blocks) {
    for (int i = (blockIdx.x - conv_blocks) * 128 + threadIdx.x; i < cnt * p.H; i += (gridDim.x - conv_blocks) * 128) {
      const int t = i / p.H, h = i % p.H;
      const float dt = softplus_f32(to_f32<T>(proj[static_cast<long long>(t) * p.ld + p.off_dt + h]) + p.dt_bias[h]);
      p.gates[(static_cast<long long>(row) + t) * p.H + h] = make_float2(dt, -expf(p.a_log[h]) * dt * 1.4426950408889634f);
    }
    return;
  }
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= p.conv_c) return;
  T* st = static_cast<T*>(p.conv_state) + static_cast<long long>(max(slot, 0)) * TAIL * p.conv_c + c;
  float w[TAPS][V], b[V];
#pragma unroll
  for (int i = 0; i < V; i += 4) {
    *reinterpret_cast<float4*>(&b[i]) = *reinterpret_cast<const float4*>(p.conv_b + c + i);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) *reinterpret_cast<float4*>(&w[j][i]) = *reinterpret_cast<const float4*>(p.conv_w + j * p.conv_c + c + i);
  }
  const T* x = proj + p.off_x + c;
  T* out = static_cast<T*>(p.xbc) + static_cast<long long>(row) * p.conv_c + c;
  constexpr int kStep = 4;                       // tokens whose inputs are requested together
  uint4 in[TAIL + kStep];                        // the window: the tokens in front, then these
#pragma unroll
  for (int r = 0; r < TAIL; ++r) {
    const int t = r - TAIL;
    in[r] = make_uint4(0u, 0u, 0u, 0u);
    if (before + t >= 0) in[r] = *reinterpret_cast<const uint4*>(x + static_cast<long long>(t) * p.ld);
    else if (old && slot >= 0) in[r] = *reinterpret_cast<const uint4*>(st + static_cast<long long>(TAIL + before + t) * p.conv_c);
  }
#pragma unroll 1
  for (int t0 = 0; t0 < cnt; t0 += kStep) {
#pragma unroll
    for (int t = 0; t < kStep; ++t)
      in[TAIL + t] = t0 + t < cnt ? *reinterpret_cast<const uint4*>(x + static_cast<long long>(t0 + t) * p.ld) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
    for (int t = 0; t < kStep; ++t) {
      if (t0 + t >= cnt) break;
      float y[V];
#pragma unroll
      for (int i = 0; i < V; ++i) {
        float a = b[i];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) a = fmaf(w[j][i], to_f32<T>(reinterpret_cast<const T*>(&in[t + j])[i]), a);
        y[i] = sizeof(T) == 2 ? __fdividef(a, 1.f + __expf(-a)) : silu_f32(a);
      }
      st16<T>(out + static_cast<long long>(t0 + t) * p.conv_c, y);
    }
    if (decode) break;
#pragma unroll
    for (int r = 0; r < TAIL; ++r) in[r] = in[r + kStep];
  }
  if (decode && slot >= 0) {
#pragma unroll
    for (int j = 0; j < TAIL; ++j) *reinterpret_cast<uint4*>(st + static_cast<long long>(j) * p.conv_c) = in[j + 1];
  }
}

// ------------------------------------------------------------------ prompts token by token (fp32 models)
template <typename T, int RL>
__global__ void __launch_bounds__(128)
ssd_scan_kernel(SsdParams p) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ float sm[ScanShape<RL>::kFloats];
  const int h = blockIdx.y, seq = blockIdx.z, slot = p.slots[seq];
  const int row0 = p.cu[seq], n = p.cu[seq + 1] - row0, grp = h / (p.H / p.G);
  if (slot < 0 || n <= 0) return;
  const T* xbc = static_cast<const T*>(p.xbc) + static_cast<long long>(row0) * p.conv_c;
  const float2* gates = p.gates + static_cast<long long>(row0) * p.H + h;
  const T *x = xbc + h * p.vp, *B = xbc + p.H * p.vp + grp * p.np, *C = B + p.G * p.np;
  T* out = static_cast<T*>(p.out) + static_cast<long long>(row0) * p.ldo + h * p.vp;
  const float skip = p.d[h];
  state_scan<RL, true>(
      sm, p.state + (static_cast<long long>(slot) * p.H + h) * p.vp * p.np, p.vp, p.np, p.pos0[seq] == 0, n, blockIdx.x * kScanRows,
      [&](int t, int d, float& q, float& k, float& w) {
        const float2 g = gates[static_cast<long long>(t) * p.H];
        q = to_f32<T>(C[static_cast<long long>(t) * p.conv_c + d]);
        k = g.x * to_f32<T>(B[static_cast<long long>(t) * p.conv_c + d]);
        w = exp2f(g.y);
      },
      [&](int t, int e) { return to_f32<T>(x[static_cast<long long>(t) * p.conv_c + e]); },
      [&](int t, int e, const float (&o)[4]) {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          out[static_cast<long long>(t) * p.ldo + e + j] = from_f32<T>(fmaf(skip, to_f32<T>(x[static_cast<long long>(t) * p.conv_c + e + j]), o[j]));
      });
}

// ------------------------------------------------------------------ decoded rows: CTA = (row, head)
template <typename T, int LPR, int PPL, int RPT>
__global__ void __launch_bounds__(256)
ssd_step_kernel(SsdParams p) {
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ __align__(16) float sm[];
  float *sq = sm, *sk = sq + p.np, *sw = sk + p.np, *sv = sw + p.np, *so = sv + p.vp;
  const int row = blockIdx.x, h = blockIdx.y, slot = p.slots[row], tid = threadIdx.x, grp = h / (p.H / p.G);
  T* out = static_cast<T*>(p.out) + static_cast<long long>(row) * p.ldo + h * p.vp;
  if (slot < 0) {
    for (int e = tid; e < p.vp; e += 256) out[e] = from_f32<T>(0.f);
    return;
  }
  StateStep<LPR, PPL, RPT, true> step(p.state + (static_cast<long long>(slot) * p.H + h) * p.vp * p.np, p.vp, p.np, p.positions[row] <= 0);
  const T* xbc = static_cast<const T*>(p.xbc) + static_cast<long long>(row) * p.conv_c;
  const float2 g = p.gates[static_cast<long long>(row) * p.H + h];
  const float w = exp2f(g.y);
  const T* B = xbc + p.H * p.vp + grp * p.np;
  for (int d = tid; d < p.np; d += 256) {
    sq[d] = to_f32<T>(B[p.G * p.np + d]);
    sk[d] = g.x * to_f32<T>(B[d]);
    sw[d] = w;
  }
  for (int e = tid; e < p.vp; e += 256) sv[e] = to_f32<T>(xbc[h * p.vp + e]);
  __syncthreads();
  step.run(sq, sk, sw, sv, so);
  __syncthreads();
  for (int e = tid; e < p.vp; e += 256) out[e] = from_f32<T>(fmaf(p.d[h], sv[e], so[e]));
}

// ------------------------------------------------------------------ prompts, bf16
template <int NT>
struct SsdChunk {
  static constexpr int kTok = 64, kCols = 64, kThreads = 128;
  static constexpr int kLdN = NT + 8, kLdX = kCols + 8;
  // bytes: C, B, x / y, the decayed scores in two halves, step sizes and logarithms
  static constexpr int kC = 0, kB = kTok * kLdN * 2, kX = 2 * kB, kPh = kX + kTok * kLdX * 2, kPl = kPh + kTok * kLdX * 2;
  static constexpr int kG = kPl + kTok * kLdX * 2, kL = kG + kTok * 8, kSmem = kL + 4 * kTok * 4;
};

// CTA = (head and 64 of its value columns, sequence or span); warp w owns the state's rows (values) 16 w .. + 15 of them. OUT = false:
// only what a span adds and leaves.
template <int NT, bool OUT>
__global__ void __launch_bounds__(128, NT <= 128 ? 3 : 1)
ssd_chunk_kernel(SsdParams p) {
  using T = __nv_bfloat16;
  using K = SsdChunk<NT>;
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  T *sc = reinterpret_cast<T*>(smem + K::kC), *sb = reinterpret_cast<T*>(smem + K::kB), *sx = reinterpret_cast<T*>(smem + K::kX);
  T *sph = reinterpret_cast<T*>(smem + K::kPh), *spl = reinterpret_cast<T*>(smem + K::kPl);
  const float2* sg = reinterpret_cast<const float2*>(smem + K::kG);
  const int tiles = (p.vp + K::kCols - 1) / K::kCols, h = blockIdx.x / tiles, c0 = blockIdx.x % tiles * K::kCols;
  const int seq = p.span.seq ? p.span.seq[blockIdx.y] : blockIdx.y, slot = p.slots[seq], grp = h / (p.H / p.G);
  int row0 = p.cu[seq], n = p.cu[seq + 1] - row0, idx = 0, spans = 1;
  if (p.span.seq) {
    idx = blockIdx.y - p.span.first[seq];
    spans = p.span.first[seq + 1] - p.span.first[seq];
    row0 += idx * kStateSpan;
    n = min(kStateSpan, n - idx * kStateSpan);
  }
  const bool final = idx == spans - 1;
  if (slot < 0 || n <= 0 || (!OUT && final)) return;
  float* carry = spans > 1 ? p.span.carry + (static_cast<long long>(blockIdx.y) * p.H + h) * p.vp * p.np : nullptr;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const T* xbc = static_cast<const T*>(p.xbc) + static_cast<long long>(row0) * p.conv_c;
  const T *x = xbc + h * p.vp + c0, *B = xbc + p.H * p.vp + grp * p.np, *C = B + p.G * p.np;
  const float2* gates = p.gates + static_cast<long long>(row0) * p.H + h;
  float* st = p.state + (static_cast<long long>(slot) * p.H + h) * p.vp * p.np;
  float* sl = reinterpret_cast<float*>(smem + K::kL) + warp * K::kTok;      // (every warp has its own copy)
  const int e0 = warp * 16, cols = min(K::kCols, p.vp - c0);
  const float skip = p.d[h];
  float S[NT / 8][4];
  {
    const float* from = !OUT ? nullptr : carry ? carry : p.pos0[seq] > 0 ? st : nullptr;
#pragma unroll
    for (int j = 0; j < NT / 8; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = e0 + g + 8 * e, c = j * 8 + 2 * t4;
        float2 v = make_float2(0.f, 0.f);
        if (from && r < cols && c < p.np) v = *reinterpret_cast<const float2*>(from + static_cast<long long>(c0 + r) * p.np + c);
        S[j][2 * e] = v.x;
        S[j][2 * e + 1] = v.y;
      }
  }
  const uint32_t aC = smem_u32(sc), aB = smem_u32(sb), aX = smem_u32(sx), aPh = smem_u32(sph), aPl = smem_u32(spl);

  float left = 0.f;                            // (OUT = false) logarithm of what the span leaves
  for (int t0 = 0; t0 < n; t0 += K::kTok) {
    const int cnt = min(K::kTok, n - t0);
    for (int i = tid; i < K::kTok * (NT / 8); i += K::kThreads) {
      const int r = i / (NT / 8), d = (i % (NT / 8)) * 8;
      const bool ok = r < cnt && d < p.np;
      const long long at = static_cast<long long>(t0 + r) * p.conv_c + d;
      if constexpr (OUT) cp_async_16(aC + (r * K::kLdN + d) * 2, ok ? C + at : C, ok ? 16 : 0);
      cp_async_16(aB + (r * K::kLdN + d) * 2, ok ? B + at : B, ok ? 16 : 0);
    }
    for (int i = tid; i < K::kTok * (K::kCols / 8); i += K::kThreads) {
      const int r = i / (K::kCols / 8), d = (i % (K::kCols / 8)) * 8;
      const bool ok = r < cnt && d < cols;
      cp_async_16(aX + (r * K::kLdX + d) * 2, ok ? x + static_cast<long long>(t0 + r) * p.conv_c + d : x, ok ? 16 : 0);
    }
    if (tid < K::kTok) {
      const bool ok = tid < cnt;
      cp_async_8(smem_u32(sg + tid), ok ? gates + static_cast<long long>(t0 + tid) * p.H : gates, ok ? 8 : 0);
    }
    cp_commit();
    cp_wait<0>();
    __syncthreads();
    float last;                                // L of the chunk's end
    {
      const float a = sg[2 * lane].y, b = sg[2 * lane + 1].y;
      float sum = a + b;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
      }
      sl[2 * lane] = sum - b;
      sl[2 * lane + 1] = sum;
      last = __shfl_sync(0xffffffffu, sum, 31);
      __syncwarp();
      left += last;
    }
    if constexpr (OUT) {
      // decayed scores: this warp's 16 keys j against the tokens i from their block on
      float a[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j][0] = a[j][1] = a[j][2] = a[j][3] = 0.f;
#pragma unroll 2
      for (int ks = 0; ks < NT / 16; ++ks) {
        uint32_t kb[4], q[4];
        ldmat_x4(kb, aB + frag_a(lane, warp * 16, ks * 16, K::kLdN));
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (i < warp) continue;
          ldmat_x4(q, aC + frag_b(lane, i * 16, ks * 16, K::kLdN));
          mma_bf16(a[2 * i], kb, q[0], q[1]);
          mma_bf16(a[2 * i + 1], kb, q[2], q[3]);
        }
      }
      const int j0 = warp * 16 + g, j1 = j0 + 8;
      const float l0 = sl[j0], l1 = sl[j1], d0 = sg[j0].x, d1 = sg[j1].x;
#pragma unroll
      for (int b = 0; b < 8; ++b) {
        if (b < 2 * warp) continue;
        const int i = b * 8 + 2 * t4;
        const float la = sl[i], lb = sl[i + 1];
        const float f0 = i >= j0 ? a[b][0] * d0 * exp2f(la - l0) : 0.f, f1 = i + 1 >= j0 ? a[b][1] * d0 * exp2f(lb - l0) : 0.f;
        const float f2 = i >= j1 ? a[b][2] * d1 * exp2f(la - l1) : 0.f, f3 = i + 1 >= j1 ? a[b][3] * d1 * exp2f(lb - l1) : 0.f;
        split_bf16x2(f0, f1, reinterpret_cast<uint32_t*>(sph + j0 * K::kLdX + i), reinterpret_cast<uint32_t*>(spl + j0 * K::kLdX + i));
        split_bf16x2(f2, f3, reinterpret_cast<uint32_t*>(sph + j1 * K::kLdX + i), reinterpret_cast<uint32_t*>(spl + j1 * K::kLdX + i));
      }
    }
    if constexpr (OUT) __syncthreads();
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < NT / 16; ++ks) {
      if (!OUT) break;
      uint32_t hi[4], lo[4];
      split_bf16x2(S[2 * ks][0], S[2 * ks][1], &hi[0], &lo[0]);
      split_bf16x2(S[2 * ks][2], S[2 * ks][3], &hi[1], &lo[1]);
      split_bf16x2(S[2 * ks + 1][0], S[2 * ks + 1][1], &hi[2], &lo[2]);
      split_bf16x2(S[2 * ks + 1][2], S[2 * ks + 1][3], &hi[3], &lo[3]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        uint32_t q[4];
        ldmat_x4(q, aC + frag_b(lane, i * 16, ks * 16, K::kLdN));
        mma_bf16(acc[2 * i], hi, q[0], q[1]);
        mma_bf16(acc[2 * i + 1], hi, q[2], q[3]);
        mma_bf16(acc[2 * i], lo, q[0], q[1]);
        mma_bf16(acc[2 * i + 1], lo, q[2], q[3]);
      }
    }
#pragma unroll
    for (int b = 0; b < 8; ++b) {
      if (!OUT) break;
      const float la = exp2f(sl[b * 8 + 2 * t4]), lb = exp2f(sl[b * 8 + 2 * t4 + 1]);
      acc[b][0] *= la; acc[b][1] *= lb; acc[b][2] *= la; acc[b][3] *= lb;
    }
    const float whole = exp2f(last);
#pragma unroll
    for (int j = 0; j < NT / 8; ++j) {
      S[j][0] *= whole; S[j][1] *= whole; S[j][2] *= whole; S[j][3] *= whole;
    }
#pragma unroll
    for (int jb = 0; jb < 4; ++jb) {
      if (jb * 16 >= cnt) break;
      uint32_t xt[4], hi[4], lo[4];
      ldmat_x4_trans(xt, aX + frag_a_trans(lane, jb * 16, e0, K::kLdX));
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (!OUT || i < jb) continue;
        uint32_t ph[4], pl[4];
        ldmat_x4_trans(ph, aPh + frag_b_trans(lane, jb * 16, i * 16, K::kLdX));
        ldmat_x4_trans(pl, aPl + frag_b_trans(lane, jb * 16, i * 16, K::kLdX));
        mma_bf16(acc[2 * i], xt, ph[0], ph[1]);
        mma_bf16(acc[2 * i + 1], xt, ph[2], ph[3]);
        mma_bf16(acc[2 * i], xt, pl[0], pl[1]);
        mma_bf16(acc[2 * i + 1], xt, pl[2], pl[3]);
      }
      float w[4];                              // what the chunk's end sees of tokens 16 jb + 2 t, + 1, + 8, + 9
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int j = jb * 16 + 2 * t4 + (e & 1) + (e >> 1) * 8;
        w[e] = sg[j].x * exp2f(last - sl[j]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(&xt[e]);
        split_bf16x2(__low2float(v) * w[e & 2], __high2float(v) * w[(e & 2) + 1], &hi[e], &lo[e]);
      }
#pragma unroll
      for (int j = 0; j < NT / 8; j += 2) {
        uint32_t b[4];
        ldmat_x4_trans(b, aB + frag_b_trans(lane, jb * 16, j * 8, K::kLdN));
        mma_bf16(S[j], hi, b[0], b[1]);
        mma_bf16(S[j + 1], hi, b[2], b[3]);
        mma_bf16(S[j], lo, b[0], b[1]);
        mma_bf16(S[j + 1], lo, b[2], b[3]);
      }
    }
    if constexpr (!OUT) {
      __syncthreads();
      continue;
    }
    // y takes the place of x (a warp's own columns)
    __syncwarp();
#pragma unroll
    for (int b = 0; b < 8; ++b)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        T* at = sx + (b * 8 + 2 * t4 + (e & 1)) * K::kLdX + e0 + g + 8 * (e >> 1);
        *at = from_f32<T>(fmaf(skip, to_f32<T>(*at), acc[b][e]));
      }
    __syncwarp();
    T* out = static_cast<T*>(p.out) + static_cast<long long>(row0 + t0) * p.ldo + h * p.vp + c0 + e0;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = i * 16 + (lane >> 1), d = (lane & 1) * 8;
      if (r < cnt && e0 + d < cols)
        *reinterpret_cast<uint4*>(out + static_cast<long long>(r) * p.ldo + d) = *reinterpret_cast<const uint4*>(sx + r * K::kLdX + e0 + d);
    }
    __syncthreads();
  }
  float* to = !OUT ? carry : final ? st : nullptr;
  if (!to) return;
  if (!OUT && tid == 0 && c0 == 0) p.span.left[static_cast<long long>(blockIdx.y) * p.H + h] = exp2f(left);
#pragma unroll
  for (int j = 0; j < NT / 8; ++j)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = e0 + g + 8 * e, c = j * 8 + 2 * t4;
      if (r < cols && c < p.np)
        *reinterpret_cast<float2*>(to + static_cast<long long>(c0 + r) * p.np + c) = make_float2(S[j][2 * e], S[j][2 * e + 1]);
    }
}

// In place: y * silu(z), then every part of a row's logical columns over its root mean square, times weight and scale. CTA = (row,
// part); a part of up to 256 * KEEP vectors stays in registers (VEC), other layouts go column by column.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
part_norm_kernel(T* t, long long ld, const T* z, long long ldz, const float* weight, int vdim, int vp, int per, float eps, float scale) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>, kKeep = VEC ? 4 : 1;
  __shared__ float red[8];
  const int row = blockIdx.y, j0 = blockIdx.x * per, tid = threadIdx.x, nt = blockDim.x;
  T* x = t + row * ld;
  const T* gate = z ? z + row * ldz : nullptr;
  auto column = [&](int j) { return vp == vdim ? j : j / vdim * vp + j % vdim; };
  auto gated = [&](int c) { return to_f32<T>(x[c]) * (gate ? silu_f32(to_f32<T>(gate[c])) : 1.f); };
  float keep[kKeep][V], ss = 0.f;
  if constexpr (VEC) {
#pragma unroll
    for (int k = 0; k < kKeep; ++k) {
      const int j = (k * nt + tid) * V;
      if (j >= per) break;
      ld16<T>(x + j0 + j, keep[k]);
      if (gate) {
        float f[V];
        ld16<T>(gate + j0 + j, f);
#pragma unroll
        for (int i = 0; i < V; ++i) keep[k][i] *= sizeof(T) == 2 ? __fdividef(f[i], 1.f + __expf(-f[i])) : silu_f32(f[i]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(keep[k][i], keep[k][i], ss);
    }
  } else {
    for (int j = tid; j < per; j += nt) {
      const float f = gated(column(j0 + j));
      ss = fmaf(f, f, ss);
    }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < nt / 32; ++w) ss += red[w];
  const float r = scale / sqrtf(ss / static_cast<float>(per) + eps);
  if constexpr (VEC) {
#pragma unroll
    for (int k = 0; k < kKeep; ++k) {
      const int j = (k * nt + tid) * V;
      if (j >= per) break;
#pragma unroll
      for (int i = 0; i < V; i += 4) {
        const float4 w = *reinterpret_cast<const float4*>(weight + j0 + j + i);
        keep[k][i] *= r * w.x; keep[k][i + 1] *= r * w.y; keep[k][i + 2] *= r * w.z; keep[k][i + 3] *= r * w.w;
      }
      st16<T>(x + j0 + j, keep[k]);
    }
  } else {
    for (int j = tid; j < per; j += nt) {
      const int c = column(j0 + j);
      x[c] = from_f32<T>(gated(c) * r * weight[c]);
    }
  }
}

template <typename T, int TAPS>
int launch_conv(const SsdParams& p, cudaStream_t s) {
  const int cb = (p.conv_c / kVec16<T> + 127) / 128, hb = (p.H + 127) / 128;
  const unsigned y = p.n_decode + p.blocks;
  if (y > 65535) return -2;
  launch_pdl(ssd_conv_kernel<T, TAPS>, dim3(cb + hb, y), dim3(128), 0, s, pdl_all_enabled(), p);
  if (TAPS > 1 && p.rows > p.n_decode)
    launch_pdl(conv_state_kernel<T>, dim3((p.conv_c + 255) / 256, p.n_seq), dim3(256), 0, s, pdl_all_enabled(),
               static_cast<const T*>(p.proj) + static_cast<long long>(p.n_decode) * p.ld + p.off_x, static_cast<long long>(p.ld), p.conv_c,
               static_cast<T*>(p.conv_state), p.cu, p.slots + p.n_decode, p.pos0, TAPS - 1);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int run_conv(const SsdParams& p, cudaStream_t s) {
  switch (p.taps) {
    case 1: return launch_conv<T, 1>(p, s);
    case 2: return launch_conv<T, 2>(p, s);
    case 3: return launch_conv<T, 3>(p, s);
    case 4: return launch_conv<T, 4>(p, s);
    case 5: return launch_conv<T, 5>(p, s);
    case 6: return launch_conv<T, 6>(p, s);
    case 7: return launch_conv<T, 7>(p, s);
    case 8: return launch_conv<T, 8>(p, s);
    default: return -2;
  }
}

template <typename T>
int run_scan(const SsdParams& p, cudaStream_t s) {
  const dim3 grid((p.vp + kScanRows - 1) / kScanRows, p.H, p.n_seq);
  const bool pdl = pdl_all_enabled();
  if (p.np <= 64) launch_pdl(ssd_scan_kernel<T, 2>, grid, dim3(128), 0, s, pdl, p);
  else if (p.np <= 128) launch_pdl(ssd_scan_kernel<T, 4>, grid, dim3(128), 0, s, pdl, p);
  else launch_pdl(ssd_scan_kernel<T, 8>, grid, dim3(128), 0, s, pdl, p);
  return static_cast<int>(cudaGetLastError());
}

template <int NT, bool OUT>
int launch_chunk(const SsdParams& p, cudaStream_t s) {
  auto kern = ssd_chunk_kernel<NT, OUT>;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SsdChunk<NT>::kSmem);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  const int tiles = (p.vp + SsdChunk<NT>::kCols - 1) / SsdChunk<NT>::kCols;
  launch_pdl(kern, dim3(p.H * tiles, p.span.seq ? p.span.n : p.n_seq), dim3(SsdChunk<NT>::kThreads), SsdChunk<NT>::kSmem, s,
             pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <int NT>
int run_chunk(const SsdParams& p, cudaStream_t s) {
  if (p.span.seq) {
    if (const int rc = launch_chunk<NT, false>(p, s)) return rc;
    launch_pdl(state_carry_kernel, dim3((p.vp * p.np / 4 + 255) / 256, p.H, p.n_seq), dim3(256), 0, s, pdl_all_enabled(), p.span,
               static_cast<const float*>(p.state), p.slots, p.pos0, p.vp, p.np, 0);
  }
  return launch_chunk<NT, true>(p, s);
}

template <typename T>
int run_step(const SsdParams& p, cudaStream_t s) {
  const int smem = (3 * p.np + 2 * p.vp) * 4;
  if (smem > 48 * 1024) return -2;
  const dim3 grid(p.n_decode, p.H);
  const bool pdl = pdl_all_enabled();
  if (p.np <= 32) launch_pdl(ssd_step_kernel<T, 8, 1, 2>, grid, dim3(256), smem, s, pdl, p);
  else if (p.np <= 64) launch_pdl(ssd_step_kernel<T, 16, 1, 4>, grid, dim3(256), smem, s, pdl, p);
  else if (p.np <= 128) launch_pdl(ssd_step_kernel<T, 32, 1, 8>, grid, dim3(256), smem, s, pdl, p);
  else launch_pdl(ssd_step_kernel<T, 32, 2, 8>, grid, dim3(256), smem, s, pdl, p);
  return static_cast<int>(cudaGetLastError());
}

bool read_ssd(const int* v, SsdParams* p) {
  p->H = v[0]; p->vdim = v[1]; p->vp = v[2]; p->N = v[3]; p->np = v[4]; p->G = v[5]; p->taps = v[6]; p->rows = v[7]; p->n_decode = v[8];
  p->n_seq = v[9]; p->blocks = v[10]; p->ld = v[11]; p->ldo = v[12];
  if (p->H <= 0 || p->H > 65535 || p->G <= 0 || p->H % p->G || p->vdim <= 0 || p->vp < p->vdim || p->vp % 8 || p->N <= 0 || p->np < p->N ||
      p->np % 16 || p->np > 256 || p->rows <= 0 || p->n_decode < 0 || p->n_decode > p->rows || p->ld % 8 || p->n_seq < 0 || p->n_seq > 65535)
    return false;
  p->off_x = p->H * p->vp;
  p->off_b = 2 * p->off_x;
  p->off_c = p->off_b + p->G * p->np;
  p->off_dt = p->off_c + p->G * p->np;
  p->conv_c = p->off_dt - p->off_x;
  return true;
}

}  // namespace
}  // namespace tsb

// ints: H, vdim, vp, state, np, groups, taps, rows, n_decode, prompt sequences, tiles of 16 tokens of their portions, projection row
// stride, result row stride. ptrs: proj, conv_w, conv_b, a_log, dt_bias, conv_state, xbc, gates, slots, positions, cu, pos0, blk_seq, blk0.
TSB_EXPORT int tsb_ssd_conv(const int* ints, void* const* q, int dtype, void* stream) {
  using namespace tsb;
  SsdParams p{};
  if (!read_ssd(ints, &p)) return -2;
  p.proj = q[0]; p.conv_w = static_cast<const float*>(q[1]); p.conv_b = static_cast<const float*>(q[2]); p.a_log = static_cast<const float*>(q[3]);
  p.dt_bias = static_cast<const float*>(q[4]); p.conv_state = q[5]; p.xbc = q[6]; p.gates = static_cast<float2*>(q[7]);
  p.slots = static_cast<const int*>(q[8]); p.positions = static_cast<const int*>(q[9]); p.cu = static_cast<const int*>(q[10]);
  p.pos0 = static_cast<const int*>(q[11]); p.blk_seq = static_cast<const int*>(q[12]); p.blk0 = static_cast<const int*>(q[13]);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) return run_conv<__nv_bfloat16>(p, s);
  if (dtype == 0) return run_conv<float>(p, s);
  return -2;
}

// ptrs: proj, xbc, gates, d, state, slots, positions, out: the first n_decode rows.
TSB_EXPORT int tsb_ssd_step(const int* ints, void* const* q, int dtype, void* stream) {
  using namespace tsb;
  SsdParams p{};
  if (!read_ssd(ints, &p) || p.n_decode <= 0) return -2;
  p.proj = q[0]; p.xbc = q[1]; p.gates = static_cast<float2*>(q[2]); p.d = static_cast<const float*>(q[3]); p.state = static_cast<float*>(q[4]);
  p.slots = static_cast<const int*>(q[5]); p.positions = static_cast<const int*>(q[6]); p.out = q[7];
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) return run_step<__nv_bfloat16>(p, s);
  if (dtype == 0) return run_step<float>(p, s);
  return -2;
}

// ptrs: proj, xbc, gates, d, state, slots, cu, pos0, out, all from the first prompt row (sequence) on; for `spans` spans of 512 tokens
// (0, or fp32: every portion is walked in one) their sequences, the first span of every sequence, carry [spans, H, vp, np], left
// [spans, H].
TSB_EXPORT int tsb_ssd_prefill(const int* ints, void* const* q, int spans, int dtype, void* stream) {
  using namespace tsb;
  SsdParams p{};
  if (!read_ssd(ints, &p) || p.n_seq <= 0) return -2;
  p.proj = q[0]; p.xbc = q[1]; p.gates = static_cast<float2*>(q[2]); p.d = static_cast<const float*>(q[3]); p.state = static_cast<float*>(q[4]);
  p.slots = static_cast<const int*>(q[5]); p.cu = static_cast<const int*>(q[6]); p.pos0 = static_cast<const int*>(q[7]); p.out = q[8];
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) {
    if (p.ldo % 8 || (reinterpret_cast<uintptr_t>(p.out) & 15)) return -2;
    if (spans > 0) {
      p.span = {static_cast<const int*>(q[9]), static_cast<const int*>(q[10]), static_cast<float*>(q[11]), static_cast<float*>(q[12]), spans};
      if (spans > 65535 || !p.span.seq || !p.span.first || !p.span.carry || !p.span.left) return -2;
    }
    return p.np <= 64 ? run_chunk<64>(p, s) : p.np <= 128 ? run_chunk<128>(p, s) : run_chunk<256>(p, s);
  }
  if (dtype == 0) return run_scan<float>(p, s);
  return -2;
}

// t [rows, ld] in place, z [rows, ldz] or null; see part_norm_kernel. dtype: 0 = fp32, 1 = bf16.
TSB_EXPORT int tsb_part_norm(void* t, long long ld, const void* z, long long ldz, const float* weight, int rows, int heads, int vdim, int vp,
                             int parts, float eps, float scale, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || heads <= 0 || vdim <= 0 || vp < vdim || parts <= 0 || (heads * vdim) % parts || (dtype != 0 && dtype != 1)) return -2;
  const int per = heads * vdim / parts, V = dtype == 1 ? 8 : 4;
  auto off = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) != 0; };
  const bool vec = vp == vdim && per % V == 0 && per <= 1024 * V && ld % V == 0 && ldz % V == 0 && !off(t) && !off(z) && !off(weight);
  const int lanes = vec ? (per / V + 3) / 4 : per;
  const int nt = std::min(256, (std::max(lanes, std::min(per / V, 128)) + 31) / 32 * 32);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto run = [&](auto zero) {
    using T = decltype(zero);
    for (int r0 = 0; r0 < rows; r0 += 65535) {
      const dim3 grid(parts, std::min(rows - r0, 65535));
      T* x = static_cast<T*>(t) + r0 * ld;
      const T* gate = z ? static_cast<const T*>(z) + r0 * ldz : nullptr;
      if (vec) launch_pdl(part_norm_kernel<T, true>, grid, dim3(nt), 0, s, pdl_all_enabled(), x, ld, gate, ldz, weight, vdim, vp, per, eps, scale);
      else launch_pdl(part_norm_kernel<T, false>, grid, dim3(nt), 0, s, pdl_all_enabled(), x, ld, gate, ldz, weight, vdim, vp, per, eps, scale);
    }
  };
  if (dtype == 1) run(__nv_bfloat16{});
  else run(0.f);
  return static_cast<int>(cudaGetLastError());
}
