// Gated delta rule (linear attention with a decaying, error-correcting state), for ragged batches of sequences.
//
// Per value head, with a state S [dim, vdim] in fp32:
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// q, k, v are short causal convolutions (per channel, then SiLU) of a packed projection; q and k are unit vectors per
// key head (q also times dim^-1/2); g = exp(-exp(A_log) softplus(a + dt_bias)), beta = sigmoid(b); the read-out is
// divided by its root mean square over vdim, scaled by a weight and by SiLU of a gate projection.
//
// Prompt rows take four launches: `delta_prepare_kernel` (convolution, unit vectors, gates; every token in parallel),
// `delta_conv_state_kernel` (the convolution's tail of each sequence goes to its slot), `delta_scan_kernel` (the
// recurrence) and `delta_gate_norm_kernel`. Decoded rows take one: `delta_step_kernel` does all of it for one token,
// streaming the state through registers once.
//
// The columns of S do not talk to each other, so the recurrence is split over value columns. In the scan eight lanes
// share a column (each holds dim / 8 rows of it in registers) and a warp walks 4 * CT columns. Both products with
// the OLD state are formed in one sweep, since S_new^T q = g (S_old^T q) + (k . q) u; that leaves two fused
// multiply-adds per element for the products and two instructions for the update, issued on register pairs
// (fma.rn.f32x2). Everything of the recurrence is fp32; nothing here uses the tensor cores.
//
// Packed projection row (element offsets, sections padded to multiples of 8):
//   [ q: Hk * dim | k: Hk * dim | v: H * vdim | gate: H * vdim | b: H | a: H ]
// A slot's convolution state holds the last taps - 1 rows of the first three sections, in the projection's type.
#include "common.cuh"

#include <algorithm>

namespace tsb {
namespace {

struct DeltaGeom {
  int Hk, H, dim, vdim;      // key heads, value heads, row and column extent of a head's state
  int dkp, vp;               // padded extents of the fp32 operands: dkp in {32, 64, 128, 256}, vp = vdim rounded up to 4
  int off_k, off_v, off_g, off_b, off_a;   // section offsets in a projection row (q starts at 0)
  int conv_c;                // columns of the convolved sections (q | k | v with their padding)
  long long ldp;             // projection row stride
};

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// ------------------------------------------------------------------ prompt rows: convolution, unit vectors, gates
struct DeltaPrepParams {
  DeltaGeom g;
  const void* proj;          // [rows, ldp]
  const float* conv_w;       // [taps, conv_c]
  const float* a_log;        // [H]
  const float* dt_bias;      // [H]
  const void* conv_state;    // [slots, taps - 1, conv_c]
  const int* cu;             // [nseq + 1] row offsets of the sequences
  const int* slots;          // [nseq]
  const int* pos0;           // [nseq] position of the first row (0: the sequence starts here)
  const int* seq_of;         // [rows]
  float* kq;                 // [rows, Hk, 2, dkp]: k, then q
  float* v;                  // [rows, H, vp]
  float4* gates;             // [rows, H]: (g, beta, k . q, 0)
  int rows;
};

template <typename T, int TAPS>
__device__ __forceinline__ float conv_at(const DeltaPrepParams& p, const T* proj, int row, int row0, long long state_row,
                                         bool has_state, int c) {
  float acc = 0.f;
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    const int r = row - (TAPS - 1) + j;
    float x = 0.f;
    if (r >= row0) x = to_f32<T>(proj[static_cast<long long>(r) * p.g.ldp + c]);
    else if (has_state)
      x = to_f32<T>(static_cast<const T*>(p.conv_state)[(state_row + (TAPS - 1) + r - row0) * p.g.conv_c + c]);
    acc = fmaf(p.conv_w[static_cast<long long>(j) * p.g.conv_c + c], x, acc);
  }
  return silu_f(acc);
}

// One warp per (row, unit). Units: the Hk key heads (q and k of the head together with its heads' gates), then blocks
// of 128 value channels.
template <typename T, int TAPS>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(DeltaPrepParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row = blockIdx.y * 8 + warp;
  if (row >= p.rows) return;
  const DeltaGeom& g = p.g;
  const int seq = p.seq_of[row];
  const int row0 = p.cu[seq];
  const bool has_state = p.pos0[seq] > 0;
  const long long state_row = static_cast<long long>(p.slots[seq]) * (TAPS - 1);
  const T* proj = static_cast<const T*>(p.proj);
  const int unit = blockIdx.x;
  if (unit < g.Hk) {
    constexpr int kMax = 8;                 // dim <= 256
    float qv[kMax], kv[kMax];
    float sqq = 0.f, skk = 0.f, sqk = 0.f;
#pragma unroll
    for (int i = 0; i < kMax; ++i) {
      const int d = lane + 32 * i;
      qv[i] = kv[i] = 0.f;
      if (d < g.dim) {
        qv[i] = conv_at<T, TAPS>(p, proj, row, row0, state_row, has_state, unit * g.dim + d);
        kv[i] = conv_at<T, TAPS>(p, proj, row, row0, state_row, has_state, g.off_k + unit * g.dim + d);
      }
      sqq = fmaf(qv[i], qv[i], sqq);
      skk = fmaf(kv[i], kv[i], skk);
      sqk = fmaf(qv[i], kv[i], sqk);
    }
    sqq = warp_sum(sqq);
    skk = warp_sum(skk);
    sqk = warp_sum(sqk);
    const float rq = 1.f / (sqrtf(sqq + 1e-6f) * sqrtf(static_cast<float>(g.dim)));
    const float rk = 1.f / sqrtf(skk + 1e-6f);
    float* out = p.kq + (static_cast<long long>(row) * g.Hk + unit) * 2 * g.dkp;
#pragma unroll
    for (int i = 0; i < kMax; ++i) {
      const int d = lane + 32 * i;
      if (d < g.dkp) {
        out[d] = kv[i] * rk;
        out[g.dkp + d] = qv[i] * rq;
      }
    }
    const int per = g.H / g.Hk;
    for (int i = lane; i < per; i += 32) {
      const int h = unit * per + i;
      const float b = to_f32<T>(proj[static_cast<long long>(row) * g.ldp + g.off_b + h]);
      const float a = to_f32<T>(proj[static_cast<long long>(row) * g.ldp + g.off_a + h]);
      const float decay = expf(-expf(p.a_log[h]) * softplus_f(a + p.dt_bias[h]));
      p.gates[static_cast<long long>(row) * g.H + h] = make_float4(decay, sigmoid_f(b), sqk * rq * rk, 0.f);
    }
  } else {
    const int c0 = (unit - g.Hk) * 128;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = c0 + lane + 32 * i;
      if (c < g.H * g.vdim)
        p.v[(static_cast<long long>(row) * g.H + c / g.vdim) * g.vp + c % g.vdim] =
            conv_at<T, TAPS>(p, proj, row, row0, state_row, has_state, g.off_v + c);
    }
  }
}

// The last taps - 1 inputs of every sequence -> its slot. Runs after the prepare kernel has read the old contents; one
// thread owns one channel of one sequence, and walks up, so a short portion may shift the slot in place.
template <typename T>
__global__ void __launch_bounds__(256)
delta_conv_state_kernel(DeltaGeom g, const T* proj, T* conv_state, const int* cu, const int* slots, const int* pos0, int tail) {
  pdl_trigger();
  pdl_grid_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int seq = blockIdx.y;
  if (c >= g.conv_c) return;
  const int row0 = cu[seq], n = cu[seq + 1] - row0;
  const int slot = slots[seq];
  if (slot < 0 || n <= 0) return;
  const bool has_state = pos0[seq] > 0;
  T* st = conv_state + static_cast<long long>(slot) * tail * g.conv_c + c;
  for (int j = 0; j < tail; ++j) {
    const int i = n - tail + j;            // token of this portion whose input belongs in place j
    T val = from_f32<T>(0.f);
    if (i >= 0) val = proj[static_cast<long long>(row0 + i) * g.ldp + c];
    else if (has_state) val = st[static_cast<long long>(j + n) * g.conv_c];
    st[static_cast<long long>(j) * g.conv_c] = val;
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
  const float* kq;           // [rows, Hk, 2, dkp]
  const float* v;            // [rows, H, vp]
  const float4* gates;       // [rows, H]
  float* state;              // [slots, H, dim, vp]
  float* o;                  // [rows, H, vp]
  const int* cu;
  const int* slots;
  const int* pos0;
};

constexpr int kScanWarps = 4;
constexpr int kScanTile = 16;    // tokens per shared-memory stage
constexpr int CT = 2;            // columns per lane
constexpr int kScanCols = kScanWarps * 4 * CT;

template <int KT>
struct ScanCfg {
  static constexpr int DK = 8 * KT;
  static constexpr int kStageFloats = kScanTile * (2 * DK + kScanCols + 4);
  static constexpr int kSmemBytes = 2 * kStageFloats * 4;
};

template <int KT>
__global__ void __launch_bounds__(kScanWarps * 32)
delta_scan_kernel(DeltaScanParams p) {
  pdl_trigger();
  pdl_grid_wait();
  using Cfg = ScanCfg<KT>;
  constexpr int DK = Cfg::DK;
  extern __shared__ __align__(16) float sm[];
  const DeltaGeom& g = p.g;
  const int seq = blockIdx.z, head = blockIdx.y;
  const int row0 = p.cu[seq], n = p.cu[seq + 1] - row0;
  const int slot = p.slots[seq];
  if (n <= 0 || slot < 0) return;
  const int hk = head / (g.H / g.Hk);
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
    constexpr int kRowVec = 2 * DK / 4;
    for (int i = threadIdx.x; i < cnt * kRowVec; i += kScanWarps * 32) {
      const int t = i / kRowVec, w = i % kRowVec;
      cp16(smem_u32(base + t * 2 * DK + w * 4), p.kq + (static_cast<long long>(row0 + t0 + t) * g.Hk + hk) * 2 * DK + w * 4, 16);
    }
    float* bv = base + kScanTile * 2 * DK;
    constexpr int kColVec = kScanCols / 4;
    for (int i = threadIdx.x; i < cnt * kColVec; i += kScanWarps * 32) {
      const int t = i / kColVec, w = i % kColVec;
      const int col = slice0 + w * 4;
      const bool ok = col < g.vp;
      cp16(smem_u32(bv + t * kScanCols + w * 4),
           p.v + (static_cast<long long>(row0 + t0 + t) * g.H + head) * g.vp + (ok ? col : 0), ok ? 16 : 0);
    }
    float* bg = bv + kScanTile * kScanCols;
    if (threadIdx.x < cnt)
      cp16(smem_u32(bg + threadIdx.x * 4), p.gates + static_cast<long long>(row0 + t0 + threadIdx.x) * g.H + head, 16);
  };
  issue(0);
  asm volatile("cp.async.commit_group;" ::: "memory");

  // which of the four sums (dk0, dk1, dq0, dq1) this lane ends up with after the exchange below
  const int own = ((lane & 4) ? 2 : 0) + ((lane & 2) ? 1 : 0);
  const int src_base = lane & ~7;
  for (int tile = 0; tile < n_tiles; ++tile) {
    if (tile + 1 < n_tiles) issue(tile + 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const float* base = sm + (tile & 1) * Cfg::kStageFloats;
    const float* bv = base + kScanTile * 2 * DK;
    const float* bg = bv + kScanTile * kScanCols;
    const int t0 = tile * kScanTile;
    const int cnt = min(kScanTile, n - t0);
#pragma unroll 2
    for (int t = 0; t < cnt; ++t) {
      const float4* kr = reinterpret_cast<const float4*>(base + t * 2 * DK);
      const float4* qr = kr + DK / 4;
      const float4 gt = *reinterpret_cast<const float4*>(bg + t * 4);
      const float2 vv = *reinterpret_cast<const float2*>(bv + t * kScanCols + lcol);
      float2 k2[KT / 2];
      float2 dk[CT], dq[CT];
#pragma unroll
      for (int c = 0; c < CT; ++c) dk[c] = dq[c] = make_float2(0.f, 0.f);
#pragma unroll
      for (int i = 0; i < KT / 4; ++i) {
        const float4 kk = kr[i * 8 + kl];
        const float4 qq = qr[i * 8 + kl];
        k2[2 * i] = make_float2(kk.x, kk.y);
        k2[2 * i + 1] = make_float2(kk.z, kk.w);
        const float2 q0 = make_float2(qq.x, qq.y), q1 = make_float2(qq.z, qq.w);
#pragma unroll
        for (int c = 0; c < CT; ++c) {
          dk[c] = fma2(S[c][2 * i], k2[2 * i], dk[c]);
          dq[c] = fma2(S[c][2 * i], q0, dq[c]);
          dk[c] = fma2(S[c][2 * i + 1], k2[2 * i + 1], dk[c]);
          dq[c] = fma2(S[c][2 * i + 1], q1, dq[c]);
        }
      }
      float a0 = dk[0].x + dk[0].y, a1 = dk[1].x + dk[1].y, a2 = dq[0].x + dq[0].y, a3 = dq[1].x + dq[1].y;
      // sum over the eight lanes of the column group: halve the number of values held per lane at each exchange
      {
        const bool hi = lane & 4;
        const float s0 = hi ? a0 : a2, s1 = hi ? a1 : a3;
        const float k0 = hi ? a2 : a0, k1 = hi ? a3 : a1;
        a0 = k0 + __shfl_xor_sync(0xffffffffu, s0, 4);
        a1 = k1 + __shfl_xor_sync(0xffffffffu, s1, 4);
      }
      {
        const bool hi = lane & 2;
        const float s0 = hi ? a0 : a1, k0 = hi ? a1 : a0;
        a0 = k0 + __shfl_xor_sync(0xffffffffu, s0, 2);
      }
      a0 += __shfl_xor_sync(0xffffffffu, a0, 1);
      const float dk0 = __shfl_sync(0xffffffffu, a0, src_base);
      const float dk1 = __shfl_sync(0xffffffffu, a0, src_base + 2);
      const float u0 = gt.y * (vv.x - gt.x * dk0);
      const float u1 = gt.y * (vv.y - gt.x * dk1);
      const float2 g2 = make_float2(gt.x, gt.x);
      const float2 uu0 = make_float2(u0, u0), uu1 = make_float2(u1, u1);
#pragma unroll
      for (int i = 0; i < KT / 2; ++i) {
        S[0][i] = fma2(S[0][i], g2, mul2(k2[i], uu0));
        S[1][i] = fma2(S[1][i], g2, mul2(k2[i], uu1));
      }
      if ((lane & 5) == 4) {               // lanes 4 and 6 of each group hold the two read-outs
        const int c = own - 2;
        if (col0 + c < g.vdim)
          p.o[(static_cast<long long>(row0 + t0 + t) * g.H + head) * g.vp + col0 + c] =
              fmaf(gt.x, a0, gt.z * (c ? u1 : u0));
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
// One warp per (row, head): y = o / rms(o) * weight * silu(gate), in the projection's type; columns past H * vdim of
// the output row are zeroed by the last head's warp.
template <typename T>
__global__ void __launch_bounds__(256)
delta_gate_norm_kernel(DeltaGeom g, const float* o, const T* proj, const float* weight, T* y, long long ldy, int y_cols,
                       int rows, float eps) {
  pdl_trigger();
  pdl_grid_wait();
  const long long w = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= static_cast<long long>(rows) * g.H) return;
  const int row = static_cast<int>(w / g.H), h = static_cast<int>(w % g.H);
  const float* orow = o + w * g.vp;
  const T* gate = proj + static_cast<long long>(row) * g.ldp + g.off_g + h * g.vdim;
  T* yr = y + row * ldy + h * g.vdim;
  float ss = 0.f;
  for (int c = lane; c < g.vdim; c += 32) ss = fmaf(orow[c], orow[c], ss);
  ss = warp_sum(ss);
  const float r = 1.f / sqrtf(ss / static_cast<float>(g.vdim) + eps);
  for (int c = lane; c < g.vdim; c += 32) yr[c] = from_f32<T>(orow[c] * r * weight[c] * silu_f(to_f32<T>(gate[c])));
  if (h == g.H - 1)
    for (int c = g.H * g.vdim + lane; c < y_cols; c += 32) y[row * ldy + c] = from_f32<T>(0.f);
}

// ------------------------------------------------------------------ decoded rows: one token per sequence, one launch
struct DeltaStepParams {
  DeltaGeom g;
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
};

constexpr int kStepThreads = 256;
constexpr int kStepWarps = kStepThreads / 32;

// CTA = (sequence, key head): it owns the head's q / k channels and all value heads that read them. A warp holds RPW
// rows of a 128-column block of S: dim / 8 rounded up.
template <typename T, int RPW>
__global__ void __launch_bounds__(kStepThreads)
delta_step_kernel(DeltaStepParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const DeltaGeom& g = p.g;
  extern __shared__ __align__(16) float sm[];
  const int per = g.H / g.Hk;
  float* sq = sm;                          // [dkp]
  float* sk = sq + g.dkp;                  // [dkp]
  float* sv = sk + g.dkp;                  // [per * vp]
  float* so = sv + per * g.vp;             // [per * vp]
  float* part = so + per * g.vp;           // [8 warps][2][128]
  float* red = part + kStepWarps * 256;    // [8 warps][3]
  const int row = blockIdx.x, hk = blockIdx.y;
  const int slot = p.slots[row];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  T* y = static_cast<T*>(p.y) + row * p.ldy;
  if (hk == g.Hk - 1)
    for (int c = g.H * g.vdim + tid; c < p.y_cols; c += kStepThreads) y[c] = from_f32<T>(0.f);
  if (slot < 0) {
    for (int c = tid; c < per * g.vdim; c += kStepThreads) y[hk * per * g.vdim + c] = from_f32<T>(0.f);
    return;
  }
  const bool has_state = p.pos[row] > 0;
  const T* proj = static_cast<const T*>(p.proj) + row * g.ldp;
  const int tail = p.taps - 1;
  T* cs = static_cast<T*>(p.conv_state) + static_cast<long long>(slot) * tail * g.conv_c;
  auto conv = [&](int c) -> float {
    float acc = 0.f;
    for (int j = 0; j < tail; ++j) {
      float x = has_state ? to_f32<T>(cs[static_cast<long long>(j) * g.conv_c + c]) : 0.f;
      acc = fmaf(p.conv_w[static_cast<long long>(j) * g.conv_c + c], x, acc);
      if (j > 0) cs[static_cast<long long>(j - 1) * g.conv_c + c] = from_f32<T>(x);
    }
    const T cur = proj[c];
    if (tail > 0) cs[static_cast<long long>(tail - 1) * g.conv_c + c] = cur;
    return silu_f(fmaf(p.conv_w[static_cast<long long>(tail) * g.conv_c + c], to_f32<T>(cur), acc));
  };
  for (int d = tid; d < g.dkp; d += kStepThreads) {
    sq[d] = d < g.dim ? conv(hk * g.dim + d) : 0.f;
    sk[d] = d < g.dim ? conv(g.off_k + hk * g.dim + d) : 0.f;
  }
  for (int c = tid; c < per * g.vdim; c += kStepThreads)
    sv[(c / g.vdim) * g.vp + c % g.vdim] = conv(g.off_v + hk * per * g.vdim + c);
  __syncthreads();
  float sqq = 0.f, skk = 0.f, sqk = 0.f;
  for (int d = tid; d < g.dim; d += kStepThreads) {
    sqq = fmaf(sq[d], sq[d], sqq);
    skk = fmaf(sk[d], sk[d], skk);
    sqk = fmaf(sq[d], sk[d], sqk);
  }
  sqq = warp_sum(sqq);
  skk = warp_sum(skk);
  sqk = warp_sum(sqk);
  if (lane == 0) {
    red[warp * 3] = sqq;
    red[warp * 3 + 1] = skk;
    red[warp * 3 + 2] = sqk;
  }
  __syncthreads();
  sqq = skk = sqk = 0.f;
#pragma unroll
  for (int w = 0; w < kStepWarps; ++w) {
    sqq += red[w * 3];
    skk += red[w * 3 + 1];
    sqk += red[w * 3 + 2];
  }
  const float rq = 1.f / (sqrtf(sqq + 1e-6f) * sqrtf(static_cast<float>(g.dim)));
  const float rk = 1.f / sqrtf(skk + 1e-6f);
  const float kq = sqk * rq * rk;

  for (int hh = 0; hh < per; ++hh) {
    const int h = hk * per + hh;
    const float bb = to_f32<T>(proj[g.off_b + h]), aa = to_f32<T>(proj[g.off_a + h]);
    const float decay = expf(-expf(p.a_log[h]) * softplus_f(aa + p.dt_bias[h]));
    const float beta = sigmoid_f(bb);
    float* st = p.state + (static_cast<long long>(slot) * g.H + h) * g.dim * g.vp;
    for (int cb = 0; cb < g.vp; cb += 128) {
      const int col = cb + lane * 4;
      const bool col_ok = col < g.vp;
      float4 S[RPW];
#pragma unroll
      for (int i = 0; i < RPW; ++i) {
        const int k = warp + kStepWarps * i;
        S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (has_state && col_ok && k < g.dim) S[i] = *reinterpret_cast<const float4*>(st + static_cast<long long>(k) * g.vp + col);
      }
      float4 dk = make_float4(0.f, 0.f, 0.f, 0.f), dq = dk;
#pragma unroll
      for (int i = 0; i < RPW; ++i) {
        const int k = warp + kStepWarps * i;
        const float kk = k < g.dim ? sk[k] * rk : 0.f, qq = k < g.dim ? sq[k] * rq : 0.f;
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
            const float kk = sk[k] * rk;
            float4 s = S[i];
            s.x = fmaf(s.x, decay, kk * u.x);
            s.y = fmaf(s.y, decay, kk * u.y);
            s.z = fmaf(s.z, decay, kk * u.z);
            s.w = fmaf(s.w, decay, kk * u.w);
            *reinterpret_cast<float4*>(st + static_cast<long long>(k) * g.vp + col) = s;
          }
        }
      }
      __syncthreads();
    }
  }
  // read-out norm and gate: one warp per value head
  for (int hh = warp; hh < per; hh += kStepWarps) {
    const float* orow = so + hh * g.vp;
    const int c0 = (hk * per + hh) * g.vdim;
    float ss = 0.f;
    for (int c = lane; c < g.vdim; c += 32) ss = fmaf(orow[c], orow[c], ss);
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / static_cast<float>(g.vdim) + p.eps);
    for (int c = lane; c < g.vdim; c += 32)
      y[c0 + c] = from_f32<T>(orow[c] * r * p.norm_w[c] * silu_f(to_f32<T>(proj[g.off_g + c0 + c])));
  }
}

// geom: 12 ints in the order of DeltaGeom (without ldp)
bool read_geom(const int* v, long long ldp, DeltaGeom* g) {
  g->Hk = v[0]; g->H = v[1]; g->dim = v[2]; g->vdim = v[3]; g->dkp = v[4]; g->vp = v[5];
  g->off_k = v[6]; g->off_v = v[7]; g->off_g = v[8]; g->off_b = v[9]; g->off_a = v[10]; g->conv_c = v[11];
  g->ldp = ldp;
  const bool dk_ok = g->dkp == 32 || g->dkp == 64 || g->dkp == 128 || g->dkp == 256;
  return g->Hk > 0 && g->H > 0 && g->H % g->Hk == 0 && g->dim > 0 && g->vdim > 0 && dk_ok && g->dim <= g->dkp &&
         g->vp >= g->vdim && g->vp % 4 == 0 && g->conv_c > 0 && ldp >= g->off_a + g->H;
}

template <typename T>
int launch_prepare(const DeltaPrepParams& p, int taps, cudaStream_t s) {
  const DeltaGeom& g = p.g;
  const dim3 grid(g.Hk + (g.H * g.vdim + 127) / 128, (p.rows + 7) / 8);
  const bool pdl = pdl_all_enabled();
#define TSB_PREP(N) case N: launch_pdl(delta_prepare_kernel<T, N>, grid, dim3(256), 0, s, pdl, p); break
  switch (taps) {
    TSB_PREP(1); TSB_PREP(2); TSB_PREP(3); TSB_PREP(4); TSB_PREP(5); TSB_PREP(6); TSB_PREP(7); TSB_PREP(8);
    default: return -2;
  }
#undef TSB_PREP
  return static_cast<int>(cudaGetLastError());
}

template <int KT>
int launch_scan(const DeltaScanParams& p, int nseq, cudaStream_t s) {
  auto kern = delta_scan_kernel<KT>;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, ScanCfg<KT>::kSmemBytes);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  const dim3 grid((p.g.vdim + kScanCols - 1) / kScanCols, p.g.H, nseq);
  launch_pdl(kern, grid, dim3(kScanWarps * 32), ScanCfg<KT>::kSmemBytes, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int RPW>
int launch_step(const DeltaStepParams& p, int rows, cudaStream_t s) {
  const int per = p.g.H / p.g.Hk;
  const int smem = (2 * p.g.dkp + 2 * per * p.g.vp + kStepWarps * 256 + kStepWarps * 3 + 8) * 4;
  if (smem > 200 * 1024) return -2;
  auto kern = delta_step_kernel<T, RPW>;
  static PerDeviceFlag attr;
  if (attr.unset()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return static_cast<int>(e);
    attr.set();
  }
  launch_pdl(kern, dim3(rows, p.g.Hk), dim3(kStepThreads), smem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace
}  // namespace tsb

// Prompt rows [rows, ldp] of nseq sequences. dtype: 0 = fp32, 1 = bf16 (projection, convolution state, y). `kq`, `v`,
// `gates`, `o` are fp32 scratch of rows * Hk * 2 * dkp, rows * H * vp, rows * H * 4 and rows * H * vp elements (16-byte
// aligned; the padding columns of v must be zero). See the structures above for the rest.
TSB_EXPORT int tsb_delta_prefill(const void* proj, long long ldp, const int* geom, const float* conv_w, const float* a_log,
                                 const float* dt_bias, const float* norm_w, void* conv_state, float* state, const int* cu,
                                 const int* slots, const int* pos0, const int* seq_of, float* kq, float* v, float* gates,
                                 float* o, void* y, long long ldy, int y_cols, int rows, int nseq, int taps, float eps,
                                 int dtype, void* stream) {
  using namespace tsb;
  DeltaGeom g;
  if (!read_geom(geom, ldp, &g) || rows <= 0 || nseq <= 0 || nseq > 65535 || taps < 1 || taps > 8 || (rows + 7) / 8 > 65535 ||
      (dtype != 0 && dtype != 1) || y_cols < g.H * g.vdim)
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  DeltaPrepParams pp{g, proj, conv_w, a_log, dt_bias, conv_state, cu, slots, pos0, seq_of, kq, v,
                     reinterpret_cast<float4*>(gates), rows};
  int rc = dtype == 1 ? launch_prepare<__nv_bfloat16>(pp, taps, s) : launch_prepare<float>(pp, taps, s);
  if (rc) return rc;
  const bool pdl = pdl_all_enabled();
  if (taps > 1) {
    const dim3 grid((g.conv_c + 255) / 256, nseq);
    if (dtype == 1)
      launch_pdl(delta_conv_state_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl, g, static_cast<const __nv_bfloat16*>(proj),
                 static_cast<__nv_bfloat16*>(conv_state), cu, slots, pos0, taps - 1);
    else
      launch_pdl(delta_conv_state_kernel<float>, grid, dim3(256), 0, s, pdl, g, static_cast<const float*>(proj),
                 static_cast<float*>(conv_state), cu, slots, pos0, taps - 1);
    rc = static_cast<int>(cudaGetLastError());
    if (rc) return rc;
  }
  DeltaScanParams sp{g, kq, v, reinterpret_cast<const float4*>(gates), state, o, cu, slots, pos0};
  switch (g.dkp) {
    case 32: rc = launch_scan<4>(sp, nseq, s); break;
    case 64: rc = launch_scan<8>(sp, nseq, s); break;
    case 128: rc = launch_scan<16>(sp, nseq, s); break;
    default: rc = launch_scan<32>(sp, nseq, s); break;
  }
  if (rc) return rc;
  const unsigned blocks = static_cast<unsigned>((static_cast<long long>(rows) * g.H + 7) / 8);
  if (dtype == 1)
    launch_pdl(delta_gate_norm_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, s, pdl, g, o,
               static_cast<const __nv_bfloat16*>(proj), norm_w, static_cast<__nv_bfloat16*>(y), ldy, y_cols, rows, eps);
  else
    launch_pdl(delta_gate_norm_kernel<float>, dim3(blocks), dim3(256), 0, s, pdl, g, o, static_cast<const float*>(proj), norm_w,
               static_cast<float*>(y), ldy, y_cols, rows, eps);
  return static_cast<int>(cudaGetLastError());
}

// Decoded rows: row i is the next token of the sequence in slot slots[i] (-1: padding, y = 0) at position pos[i].
TSB_EXPORT int tsb_delta_step(const void* proj, long long ldp, const int* geom, const float* conv_w, const float* a_log,
                              const float* dt_bias, const float* norm_w, void* conv_state, float* state, const int* slots,
                              const int* pos, void* y, long long ldy, int y_cols, int rows, int taps, float eps, int dtype,
                              void* stream) {
  using namespace tsb;
  DeltaGeom g;
  if (!read_geom(geom, ldp, &g) || rows <= 0 || g.Hk > 65535 || taps < 1 || (dtype != 0 && dtype != 1) ||
      y_cols < g.H * g.vdim)
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  DeltaStepParams p{g, proj, conv_w, a_log, dt_bias, norm_w, conv_state, state, slots, pos, y, ldy, y_cols, taps, eps};
#define TSB_STEP(R) return dtype == 1 ? launch_step<__nv_bfloat16, R>(p, rows, s) : launch_step<float, R>(p, rows, s)
  switch (g.dkp) {
    case 32: TSB_STEP(4);
    case 64: TSB_STEP(8);
    case 128: TSB_STEP(16);
    default: TSB_STEP(32);
  }
#undef TSB_STEP
}
