// Retention (linear attention with one fixed decay per head, no softmax and no denominator), for ragged batches:
//
//   S_t = decay S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t,  out = o / rms(o) * silu(gate)      per head
//
// with q and k rotated by position (pairs (u_i, v_i) stored hp columns apart, see rotated_piece) and k scaled. The state is
// fp32 and stays so.
//
// Prompts in bf16 run on the tensor cores in the chunked form. A sequence's portion is cut into spans of 256 tokens that are
// worked on at once, and a span into chunks of 64:
//   retention_span_kernel<.., false>  the state that a span adds to nothing (all spans but a sequence's last)
//   retention_carry_kernel            the state at the start of every span
//   retention_span_kernel<.., true>   the read-outs:  o_i = decay^(i+1) q_i S + sum_{j <= i} decay^(i-j) (q_i . k_j) v_j
//                                     and the update   S <- decay^n S + sum_j decay^(n-1-j) k_j v_j^T  chunk by chunk
// S lives in fp32 accumulators. Where a factor that must not lose its 32 bits meets the tensor cores (S in the read-out, the
// decayed keys in the update, the decayed scores), it goes in as two bf16 halves whose sum carries 16 bits.
// fp32 models take retention_scan_kernel (token by token, state in registers) and retention_norm_kernel.
// Decoded tokens take retention_step_kernel: the state streams through registers once.
#include "warp_mma.cuh"

#include <algorithm>

namespace tsb {
namespace {

constexpr int kSpan = 256;
constexpr int kTok = 64;          // tokens of a chunk

struct RetParams {
  int H, dp, hp, vp, vdim;        // per head: query / key columns (padded), rotated half, value columns (padded, real)
  int off_k, off_v, off_g;        // sections of a projection row (q starts at 0)
  const void* proj;
  long long ldp;
  float in_scale, k_scale;        // k_scale contains in_scale twice: once for k, once for v
  const float* log2_decay;        // [H]
  const float2* table;            // [positions, hp] cos, sin
  float* state;                   // [slots, H, dp, vp]
  const int* slots;               // [sequences of this launch]
  const int* positions;           // [rows] (decoded rows)
  const int* cu;                  // [n_seq + 1]
  const int* pos0;                // [n_seq]
  const int* tile_seq;            // [spans]
  const int* tile0;               // [n_seq + 1]
  float* carry;                   // [spans, H, dp, vp]
  float* o;                       // [rows, H, vp] fp32 read-outs, where the norm needs a launch of its own
  void* out;                      // [rows, ldo], head h at h * vp
  long long ldo;
  float eps;
  int rows, n_seq, spans;
};

// decay^n. (n = 0 gives 1 also for a decay of zero, whose logarithm the caller has made a large negative number.)
__device__ __forceinline__ float decay_pow(float log2_decay, int n) { return exp2f(log2_decay * static_cast<float>(n)); }

// ------------------------------------------------------------------ prompts, bf16
template <int DT, int ET, bool OUT>
struct SpanCfg {
  static constexpr int kBuf = DT <= 128 ? 2 : 1;       // chunks in shared memory: the next one arrives while one is worked on
  static constexpr int kLdQ = DT + 8, kLdV = ET + 8;
  // elements of a chunk's buffers (q is only there for read-outs), then what exists once
  static constexpr int kK = 0, kQ = kK + kTok * kLdQ, kV = kQ + (OUT ? kTok * kLdQ : 0), kChunkElems = kV + kTok * kLdV;
  static constexpr int kSh = kBuf * kChunkElems, kSl = kSh + (OUT ? DT * kLdV : 0), kElems = kSl + (OUT ? DT * kLdV : 0);
  static constexpr int kTable = kElems * 2, kRow = kTable + kTok * DT / 2 * 8;
  static constexpr int kSmem = kRow + 4 * kTok * 4;
  static constexpr int kWarps = DT > 128 ? 16 : 8, kThreads = kWarps * 32;
  // fragments of S: a warp holds kMT blocks of 16 rows x kNT blocks of 8 columns; kSplit warps share a block of rows
  static constexpr int kBlocks = DT / 16, kMT = kBlocks >= kWarps ? kBlocks / kWarps : 1, kSplit = kBlocks >= kWarps ? 1 : kWarps / kBlocks;
  static constexpr int kNT = ET / kSplit / 8;
  // read-out: 4 groups of 16 tokens x kCols groups of columns, kOT blocks of 8 each
  static constexpr int kCols = kWarps / 4, kOT = ET / kCols / 8;
};

template <int DT, int ET, bool OUT>
__global__ void __launch_bounds__(SpanCfg<DT, ET, OUT>::kThreads)
retention_span_kernel(RetParams p) {
  using T = __nv_bfloat16;
  using C = SpanCfg<DT, ET, OUT>;
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  T* sm = reinterpret_cast<T*>(smem);
  float2* stab = reinterpret_cast<float2*>(smem + C::kTable);      // [kTok][hp] cos, sin
  float* srow = reinterpret_cast<float*>(smem + C::kRow);          // [kCols][kTok]
  const int span = blockIdx.x, h = blockIdx.y, e0 = blockIdx.z * ET;
  const int seq = p.tile_seq[span], idx = span - p.tile0[seq], n_spans = p.tile0[seq + 1] - p.tile0[seq];
  const int slot = p.slots[seq];
  if (slot < 0 || (!OUT && idx == n_spans - 1)) return;
  const int row0 = p.cu[seq] + idx * kSpan, n = min(kSpan, p.cu[seq + 1] - row0);
  const int pos = p.pos0[seq] + idx * kSpan;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const float lg = p.log2_decay[h];
  const long long head_state = static_cast<long long>(p.dp) * p.vp;
  float* st = p.state + (static_cast<long long>(slot) * p.H + h) * head_state;
  float* cr = p.carry ? p.carry + (static_cast<long long>(span) * p.H + h) * head_state : nullptr;
  const T* proj = static_cast<const T*>(p.proj) + static_cast<long long>(row0) * p.ldp;

  // one chunk as it is in memory; rows and columns that do not exist arrive as zeros
  auto issue = [&](int t0) {
    T* buf = sm + (C::kBuf == 2 ? (t0 / kTok & 1) : 0) * C::kChunkElems;
    const int cnt = min(kTok, n - t0);
    const T* src = proj + static_cast<long long>(t0) * p.ldp;
    constexpr int kPQ = DT / 8, kPV = ET / 8;
    for (int i = tid; i < kTok * kPQ; i += C::kThreads) {
      const int r = i / kPQ, d = (i % kPQ) * 8;
      const bool ok = r < cnt && d < p.dp;
      const T* q = ok ? src + r * p.ldp + h * p.dp + d : proj;
      cp_async_16(smem_u32(buf + C::kK + r * C::kLdQ + d), ok ? q + p.off_k : q, ok ? 16 : 0);
      if constexpr (OUT) cp_async_16(smem_u32(buf + C::kQ + r * C::kLdQ + d), q, ok ? 16 : 0);
    }
    for (int i = tid; i < kTok * kPV; i += C::kThreads) {
      const int r = i / kPV, c = (i % kPV) * 8;
      const bool ok = r < cnt && e0 + c < p.vp;
      cp_async_16(smem_u32(buf + C::kV + r * C::kLdV + c), ok ? src + r * p.ldp + p.off_v + h * p.vp + e0 + c : proj, ok ? 16 : 0);
    }
    const float2* tab = p.table + static_cast<long long>(pos + t0) * p.hp;     // rows of consecutive positions: one run
    for (int i = tid * 2; i < cnt * p.hp; i += 2 * C::kThreads) cp_async_16(smem_u32(stab + i), tab + i, 16);
    cp_commit();
  };
  issue(0);

  const int m0 = warp / C::kSplit * C::kMT * 16, n0 = warp % C::kSplit * (ET / C::kSplit);
  float S[C::kMT][C::kNT][4];
  {
    const float* src = !OUT ? nullptr : n_spans > 1 ? cr : p.pos0[seq] > 0 ? st : nullptr;
#pragma unroll
    for (int i = 0; i < C::kMT; ++i)
#pragma unroll
      for (int j = 0; j < C::kNT; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int d = m0 + i * 16 + g + 8 * e, c = e0 + n0 + j * 8 + 2 * t4;
          float2 v = make_float2(0.f, 0.f);
          if (src && d < p.dp && c < p.vp) v = *reinterpret_cast<const float2*>(src + static_cast<long long>(d) * p.vp + c);
          S[i][j][2 * e] = v.x;
          S[i][j][2 * e + 1] = v.y;
        }
  }
  const uint32_t aSh = smem_u32(sm + C::kSh), aSl = smem_u32(sm + C::kSl);
  for (int t0 = 0; t0 < n; t0 += kTok) {
    const int cnt = min(kTok, n - t0);
    T* buf = sm + (C::kBuf == 2 ? (t0 / kTok & 1) : 0) * C::kChunkElems;
    cp_wait<0>();
    __syncthreads();                       // the chunk has arrived, and everyone is done with the one before
    {
      // scale, and rotate in place: a thread takes both halves of eight pairs
      const int np = p.hp / 8, per = np + (p.dp - 2 * p.hp) / 8;
      for (int i = tid; i < cnt * per; i += C::kThreads) {
        const int r = i / per, w = i % per;
#pragma unroll
        for (int which = 0; which < (OUT ? 2 : 1); ++which) {
          T* x = buf + (which ? C::kQ : C::kK) + r * C::kLdQ;
          const float s = which ? p.in_scale : p.k_scale;
          float u[8];
          if (w < np) {
            float v[8], a[8], b[8];
            ld16<T>(x + w * 8, u);
            ld16<T>(x + p.hp + w * 8, v);
#pragma unroll
            for (int e = 0; e < 8; e += 2) {
              const float4 cs = *reinterpret_cast<const float4*>(stab + r * p.hp + w * 8 + e);
              a[e] = (u[e] * cs.x - v[e] * cs.y) * s;
              b[e] = (v[e] * cs.x + u[e] * cs.y) * s;
              a[e + 1] = (u[e + 1] * cs.z - v[e + 1] * cs.w) * s;
              b[e + 1] = (v[e + 1] * cs.z + u[e + 1] * cs.w) * s;
            }
            st16<T>(x + w * 8, a);
            st16<T>(x + p.hp + w * 8, b);
          } else {
            const int d = 2 * p.hp + (w - np) * 8;
            ld16<T>(x + d, u);
#pragma unroll
            for (int e = 0; e < 8; ++e) u[e] *= s;
            st16<T>(x + d, u);
          }
        }
      }
    }
    if constexpr (OUT) {
#pragma unroll
      for (int i = 0; i < C::kMT; ++i)
#pragma unroll
        for (int j = 0; j < C::kNT; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int at = (m0 + i * 16 + g + 8 * e) * C::kLdV + n0 + j * 8 + 2 * t4;
            split_bf16x2(S[i][j][2 * e], S[i][j][2 * e + 1], reinterpret_cast<uint32_t*>(sm + C::kSh + at),
                         reinterpret_cast<uint32_t*>(sm + C::kSl + at));
          }
    }
    __syncthreads();
    if (C::kBuf == 2 && t0 + kTok < n) issue(t0 + kTok);
    const uint32_t aQ = smem_u32(buf + C::kQ), aK = smem_u32(buf + C::kK), aV = smem_u32(buf + C::kV);
    if constexpr (OUT) {
      const int rg = warp & 3, r0 = rg * 16, c0 = (warp >> 2) * (ET / C::kCols);
      float acc[C::kOT][4];
#pragma unroll
      for (int j = 0; j < C::kOT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
      float sc[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll 2
      for (int ks = 0; ks < DT / 16; ++ks) {
        uint32_t a[4], b[4];
        ldmat_x4(a, aQ + frag_a(lane, r0, ks * 16, C::kLdQ));
#pragma unroll
        for (int j = 0; j < C::kOT; j += 2) {
          ldmat_x4_trans(b, aSh + frag_b_trans(lane, ks * 16, c0 + j * 8, C::kLdV));
          mma_bf16(acc[j], a, b[0], b[1]);
          mma_bf16(acc[j + 1], a, b[2], b[3]);
          ldmat_x4_trans(b, aSl + frag_b_trans(lane, ks * 16, c0 + j * 8, C::kLdV));
          mma_bf16(acc[j], a, b[0], b[1]);
          mma_bf16(acc[j + 1], a, b[2], b[3]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (j > rg) break;                       // keys after the last of these tokens
          ldmat_x4(b, aK + frag_b(lane, j * 16, ks * 16, C::kLdQ));
          mma_bf16(sc[2 * j], a, b[0], b[1]);
          mma_bf16(sc[2 * j + 1], a, b[2], b[3]);
        }
      }
      const float w0 = decay_pow(lg, r0 + g + 1), w1 = decay_pow(lg, r0 + g + 9);
#pragma unroll
      for (int j = 0; j < C::kOT; ++j) {
        acc[j][0] *= w0; acc[j][1] *= w0; acc[j][2] *= w1; acc[j][3] *= w1;
      }
      // decay^(i - key) as decay^(i - first key of the block) times decay^-(place in the block); a decay so steep that the second
      // factor could overflow takes the power itself
      const bool steep = lg < -8.f;
      float back_in[2][2];
#pragma unroll
      for (int b = 0; b < 2; ++b)
#pragma unroll
        for (int e = 0; e < 2; ++e) back_in[b][e] = decay_pow(lg, -(b * 8 + 2 * t4 + e));
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (j > rg) break;
        uint32_t hi[4], lo[4];
        const float from[2] = {decay_pow(lg, r0 + g - 16 * j), decay_pow(lg, r0 + g + 8 - 16 * j)};
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          float f[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int back = r0 + g + (e >> 1) * 8 - (j * 16 + b * 8 + 2 * t4 + (e & 1));
            const float w = steep ? decay_pow(lg, back) : from[e >> 1] * back_in[b][e & 1];
            f[e] = back < 0 ? 0.f : sc[2 * j + b][e] * w;
          }
          split_bf16x2(f[0], f[1], &hi[2 * b], &lo[2 * b]);
          split_bf16x2(f[2], f[3], &hi[2 * b + 1], &lo[2 * b + 1]);
        }
#pragma unroll
        for (int c = 0; c < C::kOT; c += 2) {
          uint32_t b[4];
          ldmat_x4_trans(b, aV + frag_b_trans(lane, j * 16, c0 + c * 8, C::kLdV));
          mma_bf16(acc[c], hi, b[0], b[1]);
          mma_bf16(acc[c + 1], hi, b[2], b[3]);
          mma_bf16(acc[c], lo, b[0], b[1]);
          mma_bf16(acc[c + 1], lo, b[2], b[3]);
        }
      }
      if (p.o) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = r0 + g + 8 * e;
          if (r >= cnt) continue;
          float* o = p.o + (static_cast<long long>(row0 + t0 + r) * p.H + h) * p.vp + e0 + c0;
#pragma unroll
          for (int j = 0; j < C::kOT; ++j)
            if (e0 + c0 + j * 8 + 2 * t4 < p.vp) *reinterpret_cast<float2*>(o + j * 8 + 2 * t4) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
        }
      } else {
        __nv_bfloat162 gate[2][C::kOT];            // requested before the norm's barrier
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = min(r0 + g + 8 * e, cnt - 1);
          const T* gr = proj + (t0 + r) * p.ldp + p.off_g + h * p.vp;
#pragma unroll
          for (int j = 0; j < C::kOT; ++j) gate[e][j] = *reinterpret_cast<const __nv_bfloat162*>(gr + min(c0 + j * 8 + 2 * t4, p.vp - 2));
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float ss = 0.f;
#pragma unroll
          for (int j = 0; j < C::kOT; ++j) ss = fmaf(acc[j][2 * e], acc[j][2 * e], fmaf(acc[j][2 * e + 1], acc[j][2 * e + 1], ss));
          ss += __shfl_xor_sync(0xffffffffu, ss, 1);
          ss += __shfl_xor_sync(0xffffffffu, ss, 2);
          if (t4 == 0) srow[(warp >> 2) * kTok + r0 + g + 8 * e] = ss;
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = r0 + g + 8 * e;
          if (r >= cnt) continue;
          float ss = 0.f;
#pragma unroll
          for (int q = 0; q < C::kCols; ++q) ss += srow[q * kTok + r];
          const float rs = rsqrtf(ss / static_cast<float>(p.vdim) + p.eps);
          T* out = static_cast<T*>(p.out) + static_cast<long long>(row0 + t0 + r) * p.ldo + h * p.vp;
#pragma unroll
          for (int j = 0; j < C::kOT; ++j) {
            const int c = c0 + j * 8 + 2 * t4;
            if (c >= p.vp) continue;
            const float g0 = p.in_scale * __low2float(gate[e][j]), g1 = p.in_scale * __high2float(gate[e][j]);
            *reinterpret_cast<uint32_t*>(out + c) =
                pack_bf16x2(acc[j][2 * e] * rs * __fdividef(g0, 1.f + __expf(-g0)), acc[j][2 * e + 1] * rs * __fdividef(g1, 1.f + __expf(-g1)));
          }
        }
      }
    }
    const float wn = decay_pow(lg, cnt);
#pragma unroll
    for (int i = 0; i < C::kMT; ++i)
#pragma unroll
      for (int j = 0; j < C::kNT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][j][e] *= wn;
#pragma unroll
    for (int ks = 0; ks < kTok / 16; ++ks) {
      if (ks * 16 >= cnt) break;
      float w[4];                          // what is left of tokens 16 ks + 2 t, + 1, + 8, + 9 at the end of the chunk
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int back = cnt - 1 - (ks * 16 + 2 * t4 + (e & 1) + (e >> 1) * 8);
        w[e] = back < 0 ? 0.f : decay_pow(lg, back);
      }
      uint32_t hi[C::kMT][4], lo[C::kMT][4];
#pragma unroll
      for (int i = 0; i < C::kMT; ++i) {
        uint32_t a[4];
        ldmat_x4_trans(a, aK + frag_a_trans(lane, ks * 16, m0 + i * 16, C::kLdQ));
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const __nv_bfloat162 k = *reinterpret_cast<const __nv_bfloat162*>(&a[e]);
          split_bf16x2(__low2float(k) * w[e & 2], __high2float(k) * w[(e & 2) + 1], &hi[i][e], &lo[i][e]);
        }
      }
#pragma unroll
      for (int j = 0; j < C::kNT; j += 2) {
        uint32_t b[4];
        ldmat_x4_trans(b, aV + frag_b_trans(lane, ks * 16, n0 + j * 8, C::kLdV));
#pragma unroll
        for (int i = 0; i < C::kMT; ++i) {
          mma_bf16(S[i][j], hi[i], b[0], b[1]);
          mma_bf16(S[i][j + 1], hi[i], b[2], b[3]);
          mma_bf16(S[i][j], lo[i], b[0], b[1]);
          mma_bf16(S[i][j + 1], lo[i], b[2], b[3]);
        }
      }
    }
    if (C::kBuf == 1 && t0 + kTok < n) {
      __syncthreads();
      issue(t0 + kTok);
    }
  }
  float* dst = !OUT ? cr : idx == n_spans - 1 ? st : nullptr;
  if (!dst) return;
#pragma unroll
  for (int i = 0; i < C::kMT; ++i)
#pragma unroll
    for (int j = 0; j < C::kNT; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = m0 + i * 16 + g + 8 * e, c = e0 + n0 + j * 8 + 2 * t4;
        if (d < p.dp && c < p.vp)
          *reinterpret_cast<float2*>(dst + static_cast<long long>(d) * p.vp + c) = make_float2(S[i][j][2 * e], S[i][j][2 * e + 1]);
      }
}

// What every span adds -> the state at its start. Sequences of one span need none of it.
__global__ void __launch_bounds__(256)
retention_carry_kernel(RetParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const long long head_state = static_cast<long long>(p.dp) * p.vp;
  const long long i = (blockIdx.x * 256ll + threadIdx.x) * 4;
  const int h = blockIdx.y, seq = blockIdx.z;
  const int first = p.tile0[seq], n = p.tile0[seq + 1] - first, slot = p.slots[seq];
  if (i >= head_state || n < 2 || slot < 0) return;
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.pos0[seq] > 0) s = *reinterpret_cast<const float4*>(p.state + (static_cast<long long>(slot) * p.H + h) * head_state + i);
  const float w = decay_pow(p.log2_decay[h], kSpan);
  float4* c = reinterpret_cast<float4*>(p.carry + (static_cast<long long>(first) * p.H + h) * head_state + i);
  const long long step = p.H * head_state / 4;
  float4 next = c[0];
  for (int k = 0; k < n; ++k) {
    const float4 add = next;
    if (k + 2 < n) next = c[(k + 1) * step];
    c[k * step] = s;
    s = make_float4(fmaf(w, s.x, add.x), fmaf(w, s.y, add.y), fmaf(w, s.z, add.z), fmaf(w, s.w, add.w));
  }
}

// ------------------------------------------------------------------ prompts token by token (fp32 models)
constexpr int kScanTok = 16, kScanCols = 16;

// Four warps of four value columns; lane l holds rows l + 32 i of them.
template <typename T, int RL>
__global__ void __launch_bounds__(128)
retention_scan_kernel(RetParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>, DP = RL * 32;
  __shared__ __align__(16) float sq[kScanTok][DP], sk[kScanTok][DP], sv[kScanTok][kScanCols];
  const int h = blockIdx.y, seq = blockIdx.z, slot = p.slots[seq];
  const int row0 = p.cu[seq], n = p.cu[seq + 1] - row0, pos = p.pos0[seq];
  if (slot < 0 || n <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c0 = blockIdx.x * kScanCols + warp * 4;
  float* st = p.state + (static_cast<long long>(slot) * p.H + h) * p.dp * p.vp;
  const float w = decay_pow(p.log2_decay[h], 1);
  const bool mine = c0 < p.vp;
  float4 S[RL];
#pragma unroll
  for (int i = 0; i < RL; ++i) {
    const int d = lane + 32 * i;
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (pos > 0 && mine && d < p.dp) S[i] = *reinterpret_cast<const float4*>(st + static_cast<long long>(d) * p.vp + c0);
  }
  const T* proj = static_cast<const T*>(p.proj);
  for (int t0 = 0; t0 < n; t0 += kScanTok) {
    const int cnt = min(kScanTok, n - t0);
    __syncthreads();
    for (int i = tid; i < cnt * (DP / V); i += 128) {
      const int r = i / (DP / V), d = (i % (DP / V)) * V;
      float q[V] = {}, k[V] = {};
      if (d < p.dp) {
        const T* head = proj + static_cast<long long>(row0 + t0 + r) * p.ldp + h * p.dp;
        const float2* table = p.table + static_cast<long long>(pos + t0 + r) * p.hp;
        rotated_piece<T>(head, d, p.hp, table, q);
        rotated_piece<T>(head + p.off_k, d, p.hp, table, k);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) {
        sq[r][d + e] = q[e] * p.in_scale;
        sk[r][d + e] = k[e] * p.k_scale;
      }
    }
    for (int i = tid; i < cnt * kScanCols; i += 128) {
      const int r = i / kScanCols, c = blockIdx.x * kScanCols + i % kScanCols;
      sv[r][i % kScanCols] = c < p.vp ? to_f32<T>(proj[static_cast<long long>(row0 + t0 + r) * p.ldp + p.off_v + h * p.vp + c]) : 0.f;
    }
    __syncthreads();
    for (int r = 0; r < cnt; ++r) {
      const float4 v = *reinterpret_cast<const float4*>(&sv[r][warp * 4]);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < RL; ++i) {
        const float k = sk[r][lane + 32 * i], q = sq[r][lane + 32 * i];
        S[i].x = fmaf(w, S[i].x, k * v.x); S[i].y = fmaf(w, S[i].y, k * v.y);
        S[i].z = fmaf(w, S[i].z, k * v.z); S[i].w = fmaf(w, S[i].w, k * v.w);
        o.x = fmaf(S[i].x, q, o.x); o.y = fmaf(S[i].y, q, o.y);
        o.z = fmaf(S[i].z, q, o.z); o.w = fmaf(S[i].w, q, o.w);
      }
      o.x = warp_sum(o.x); o.y = warp_sum(o.y); o.z = warp_sum(o.z); o.w = warp_sum(o.w);
      if (lane == 0 && mine)
        *reinterpret_cast<float4*>(p.o + (static_cast<long long>(row0 + t0 + r) * p.H + h) * p.vp + c0) = o;
    }
  }
#pragma unroll
  for (int i = 0; i < RL; ++i) {
    const int d = lane + 32 * i;
    if (mine && d < p.dp) *reinterpret_cast<float4*>(st + static_cast<long long>(d) * p.vp + c0) = S[i];
  }
}

// out = o / rms(o) * silu(gate): one warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256)
retention_norm_kernel(RetParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const long long w = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= static_cast<long long>(p.rows) * p.H) return;
  const long long row = w / p.H;
  const int h = static_cast<int>(w % p.H);
  const float* o = p.o + w * p.vp;
  const T* gate = static_cast<const T*>(p.proj) + row * p.ldp + p.off_g + h * p.vp;
  T* out = static_cast<T*>(p.out) + row * p.ldo + h * p.vp;
  float ss = 0.f;
  for (int c = lane * 2; c < p.vp; c += 64) {
    const float2 f = *reinterpret_cast<const float2*>(o + c);
    ss = fmaf(f.x, f.x, fmaf(f.y, f.y, ss));
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.vdim) + p.eps);
  for (int c = lane * 2; c < p.vp; c += 64) {
    const float2 f = *reinterpret_cast<const float2*>(o + c);
    const float a = f.x * r * silu_f32(p.in_scale * to_f32<T>(gate[c])), b = f.y * r * silu_f32(p.in_scale * to_f32<T>(gate[c + 1]));
    if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(out + c) = pack_bf16x2(a, b);
    else *reinterpret_cast<float2*>(out + c) = make_float2(a, b);
  }
}

// ------------------------------------------------------------------ decoded tokens
// CTA = (row, head), eight warps. LPR lanes share a row of the state (four columns each), so a warp holds 32 / LPR rows at
// once; columns beyond 4 LPR are further rounds.
template <typename T, int LPR, int RPT>
__global__ void __launch_bounds__(256)
retention_step_kernel(RetParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>, kGroups = 256 / LPR, kCols = LPR * 4;
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                          // [dp]
  float* sk = sq + p.dp;                   // [dp]
  float* so = sk + p.dp;                   // [vp]
  float* part = so + p.vp;                 // [kGroups][kCols]
  float* red = part + kGroups * kCols;     // [8]
  const int row = blockIdx.x, h = blockIdx.y, slot = p.slots[row];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const T* x = static_cast<const T*>(p.proj) + row * p.ldp;
  T* out = static_cast<T*>(p.out) + row * p.ldo + h * p.vp;
  if (slot < 0) {
    for (int c = tid; c < p.vp; c += 256) out[c] = from_f32<T>(0.f);
    return;
  }
  const int pos = p.positions[row];
  float* st = p.state + (static_cast<long long>(slot) * p.H + h) * p.dp * p.vp;
  const int grp = tid / LPR, gl = tid % LPR;
  float4 S[RPT];
  auto fetch = [&](int c) {
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = grp + kGroups * i;
      S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (pos > 0 && d < p.dp && c < p.vp) S[i] = __ldcs(reinterpret_cast<const float4*>(st + static_cast<long long>(d) * p.vp + c));
    }
  };
  fetch(gl * 4);
  const float w = decay_pow(p.log2_decay[h], 1);
  for (int i = tid; i < 2 * (p.dp / V); i += 256) {
    const bool is_k = i >= p.dp / V;
    const int d = (is_k ? i - p.dp / V : i) * V;
    float f[V];
    rotated_piece<T>(x + (is_k ? p.off_k : 0) + h * p.dp, d, p.hp, p.table + static_cast<long long>(pos) * p.hp, f);
#pragma unroll
    for (int e = 0; e < V; ++e) (is_k ? sk : sq)[d + e] = f[e] * (is_k ? p.k_scale : p.in_scale);
  }
  __syncthreads();
  float ss = 0.f;
  for (int cb = 0; cb < p.vp; cb += kCols) {
    const int c = cb + gl * 4;
    const bool ok = c < p.vp;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (ok) {
      float v[4];
      const T* vr = x + p.off_v + h * p.vp + c;
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = to_f32<T>(vr[e]);
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        const int d = grp + kGroups * i;
        if (d >= p.dp) continue;
        const float k = sk[d], q = sq[d];
        float4 s = S[i];
        s.x = fmaf(w, s.x, k * v[0]); s.y = fmaf(w, s.y, k * v[1]);
        s.z = fmaf(w, s.z, k * v[2]); s.w = fmaf(w, s.w, k * v[3]);
        o.x = fmaf(s.x, q, o.x); o.y = fmaf(s.y, q, o.y);
        o.z = fmaf(s.z, q, o.z); o.w = fmaf(s.w, q, o.w);
        __stcs(reinterpret_cast<float4*>(st + static_cast<long long>(d) * p.vp + c), s);
      }
    }
    *reinterpret_cast<float4*>(part + grp * kCols + gl * 4) = o;
    if (cb + kCols < p.vp) fetch(c + kCols);
    __syncthreads();
    for (int i = tid; i < kCols; i += 256) {
      if (cb + i >= p.vp) break;
      float a = 0.f;
#pragma unroll
      for (int k = 0; k < kGroups; ++k) a += part[k * kCols + i];
      so[cb + i] = a;
      ss = fmaf(a, a, ss);
    }
    __syncthreads();
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int k = 0; k < 8; ++k) ss += red[k];
  const float r = 1.f / sqrtf(ss / static_cast<float>(p.vdim) + p.eps);
  const T* gate = x + p.off_g + h * p.vp;
  for (int c = tid; c < p.vp; c += 256) out[c] = from_f32<T>(so[c] * r * silu_f32(p.in_scale * to_f32<T>(gate[c])));
}

template <typename K>
int opt_in_smem(K kern, PerDeviceFlag* flag, int bytes) {
  if (!flag->unset()) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e == cudaSuccess) flag->set();
  return static_cast<int>(e);
}

template <int DT, int ET, bool OUT>
int launch_span(const RetParams& p, cudaStream_t s) {
  auto kern = retention_span_kernel<DT, ET, OUT>;
  static PerDeviceFlag attr;
  if (const int e = opt_in_smem(kern, &attr, SpanCfg<DT, ET, OUT>::kSmem)) return e;
  launch_pdl(kern, dim3(p.spans, p.H, (p.vp + ET - 1) / ET), dim3(SpanCfg<DT, ET, OUT>::kThreads), SpanCfg<DT, ET, OUT>::kSmem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int launch_norm(const RetParams& p, cudaStream_t s) {
  const long long warps = static_cast<long long>(p.rows) * p.H;
  launch_pdl(retention_norm_kernel<T>, dim3(static_cast<unsigned>((warps + 7) / 8)), dim3(256), 0, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <int DT, int ET>
int run_spans(const RetParams& p, cudaStream_t s) {
  int rc = 0;
  if (p.carry) {
    if ((rc = launch_span<DT, ET, false>(p, s))) return rc;
    launch_pdl(retention_carry_kernel, dim3((p.dp * p.vp / 4 + 255) / 256, p.H, p.n_seq), dim3(256), 0, s, pdl_all_enabled(), p);
    if ((rc = static_cast<int>(cudaGetLastError()))) return rc;
  }
  if ((rc = launch_span<DT, ET, true>(p, s))) return rc;
  return p.o ? launch_norm<__nv_bfloat16>(p, s) : 0;
}

template <typename T>
int run_scan(const RetParams& p, cudaStream_t s) {
  const dim3 grid((p.vp + kScanCols - 1) / kScanCols, p.H, p.n_seq);
  const bool pdl = pdl_all_enabled();
  if (p.dp <= 64) launch_pdl(retention_scan_kernel<T, 2>, grid, dim3(128), 0, s, pdl, p);
  else if (p.dp <= 128) launch_pdl(retention_scan_kernel<T, 4>, grid, dim3(128), 0, s, pdl, p);
  else launch_pdl(retention_scan_kernel<T, 8>, grid, dim3(128), 0, s, pdl, p);
  const int rc = static_cast<int>(cudaGetLastError());
  return rc ? rc : launch_norm<T>(p, s);
}

template <typename T, int LPR, int RPT>
int launch_step(const RetParams& p, cudaStream_t s) {
  const int smem = (2 * p.dp + p.vp + 256 * 4 + 8) * 4;
  auto kern = retention_step_kernel<T, LPR, RPT>;
  if (smem > 48 * 1024) return -2;
  launch_pdl(kern, dim3(p.rows, p.H), dim3(256), smem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int run_step(const RetParams& p, cudaStream_t s) {
  if (p.vp <= 32) {            // 32 rows x 8 lanes at once
    if (p.dp <= 64) return launch_step<T, 8, 2>(p, s);
    return p.dp <= 128 ? launch_step<T, 8, 4>(p, s) : launch_step<T, 8, 8>(p, s);
  }
  if (p.vp <= 64) {            // 16 rows x 16 lanes
    if (p.dp <= 64) return launch_step<T, 16, 4>(p, s);
    return p.dp <= 128 ? launch_step<T, 16, 8>(p, s) : launch_step<T, 16, 16>(p, s);
  }
  if (p.dp <= 64) return launch_step<T, 32, 8>(p, s);
  return p.dp <= 128 ? launch_step<T, 32, 16>(p, s) : launch_step<T, 32, 32>(p, s);
}

bool read_ret(const int* v, RetParams* p) {
  p->H = v[0]; p->dp = v[1]; p->hp = v[2]; p->vp = v[3]; p->vdim = v[4]; p->off_k = v[5]; p->off_v = v[6]; p->off_g = v[7];
  p->rows = v[8]; p->n_seq = v[9]; p->spans = v[10];
  return p->H > 0 && p->H <= 65535 && p->dp > 0 && p->dp % 16 == 0 && p->dp <= 256 && p->hp >= 0 && p->hp % 8 == 0 && 2 * p->hp <= p->dp &&
         p->vdim > 0 && p->vp >= p->vdim && p->vp % 8 == 0 && p->off_k % 8 == 0 && p->off_v % 8 == 0 && p->off_g % 8 == 0 && p->rows > 0;
}

}  // namespace
}  // namespace tsb

// ints: H, dp, hp, vp, vdim, off_k, off_v, off_g, rows, n_seq, spans. Prompt rows of n_seq sequences, cut into spans of 256
// tokens from each portion's first row (tile_seq [spans], tile0 [n_seq + 1]). dtype: 0 = fp32, 1 = bf16 (projection, out).
// chunked = 1 (bf16): tensor cores; `carry` [spans, H, dp, vp] is needed when a sequence has more than one span. `o` [rows, H, vp]
// (fp32) is needed when chunked = 0 or a head's values do not fit one tile (vp > 128, or vp > 64 with dp > 128). See RetParams.
TSB_EXPORT int tsb_retention_prefill(const int* ints, const void* proj, long long ldp, float in_scale, float k_scale,
                                     const float* log2_decay, const float* table, float* state, const int* slots, const int* cu,
                                     const int* pos0, const int* tile_seq, const int* tile0, float* carry, float* o, void* out,
                                     long long ldo, float eps, int chunked, int dtype, void* stream) {
  using namespace tsb;
  RetParams p{};
  if (!read_ret(ints, &p) || p.n_seq <= 0 || p.n_seq > 65535 || ldp % 8 || ldo % 2 || (dtype != 0 && dtype != 1)) return -2;
  p.proj = proj; p.ldp = ldp; p.in_scale = in_scale; p.k_scale = k_scale; p.log2_decay = log2_decay;
  p.table = reinterpret_cast<const float2*>(table); p.state = state; p.slots = slots; p.cu = cu; p.pos0 = pos0; p.tile_seq = tile_seq;
  p.tile0 = tile0; p.carry = carry; p.o = o; p.out = out; p.ldo = ldo; p.eps = eps;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (!chunked) {
    if (!o) return -2;
    return dtype == 1 ? run_scan<__nv_bfloat16>(p, s) : run_scan<float>(p, s);
  }
  if (dtype != 1 || p.spans <= 0 || !tile_seq || !tile0) return -2;
  const int cols = p.dp <= 128 && p.vp > 64 ? 128 : 64;
  if (p.vp <= cols) p.o = nullptr;
  else if (!o) return -2;
  if (p.dp <= 64) return cols == 64 ? run_spans<64, 64>(p, s) : run_spans<64, 128>(p, s);
  if (p.dp <= 128) return cols == 64 ? run_spans<128, 64>(p, s) : run_spans<128, 128>(p, s);
  return run_spans<256, 64>(p, s);
}

// Decoded rows: row i is the next token of the sequence in slot slots[i] (-1: padding, out = 0) at position positions[i].
TSB_EXPORT int tsb_retention_step(const int* ints, const void* proj, long long ldp, float in_scale, float k_scale, const float* log2_decay,
                                  const float* table, float* state, const int* slots, const int* positions, void* out, long long ldo,
                                  float eps, int dtype, void* stream) {
  using namespace tsb;
  RetParams p{};
  if (!read_ret(ints, &p) || ldp % 8 || (dtype != 0 && dtype != 1)) return -2;
  p.proj = proj; p.ldp = ldp; p.in_scale = in_scale; p.k_scale = k_scale; p.log2_decay = log2_decay;
  p.table = reinterpret_cast<const float2*>(table); p.state = state; p.slots = slots; p.positions = positions; p.out = out; p.ldo = ldo;
  p.eps = eps;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == 1 ? run_step<__nv_bfloat16>(p, s) : run_step<float>(p, s);
}
