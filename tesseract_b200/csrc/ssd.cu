// State-space duality (a matrix state per head with a scalar decay per token), for ragged batches:
//
//   S_t = exp(-exp(A_log) dt) S_(t-1) + (dt x_t) B_t^T,  y_t = S_t C_t + D x_t                      per head, S [vdim][state]
//   t = y * silu(z), then normed in equal parts (part_norm_kernel)
//
// x, B and C pass a short causal convolution with bias and SiLU (ssd_conv_kernel, which also turns the dt projection into dt and
// the logarithm of the decay); heads share the B and C of their group. The state and what decays it are fp32.
#include "linear_state.cuh"
#include "ragged_conv.cuh"

#include <algorithm>

namespace tsb {
namespace {

constexpr int kBlk = 4;            // tokens of a portion that a thread of the convolution takes

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
  void* out;                 // [rows, ldo]
};

__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// A thread takes 16 bytes of columns of one decoded row or of up to kBlk tokens of a portion; the last column blocks take the
// heads' step sizes.
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
  uint4 in[TAIL + kBlk];
#pragma unroll
  for (int r = 0; r < TAIL + kBlk; ++r) {
    const int t = r - TAIL;                      // token relative to the first row
    in[r] = make_uint4(0u, 0u, 0u, 0u);
    if (t >= cnt) continue;
    if (before + t >= 0) in[r] = *reinterpret_cast<const uint4*>(proj + static_cast<long long>(t) * p.ld + p.off_x + c);
    else if (old && slot >= 0) in[r] = *reinterpret_cast<const uint4*>(st + static_cast<long long>(TAIL + before + t) * p.conv_c);
  }
  float w[TAPS][V], b[V];
#pragma unroll
  for (int i = 0; i < V; i += 4) {
    *reinterpret_cast<float4*>(&b[i]) = *reinterpret_cast<const float4*>(p.conv_b + c + i);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) *reinterpret_cast<float4*>(&w[j][i]) = *reinterpret_cast<const float4*>(p.conv_w + j * p.conv_c + c + i);
  }
  T* out = static_cast<T*>(p.xbc) + static_cast<long long>(row) * p.conv_c + c;
#pragma unroll
  for (int t = 0; t < kBlk; ++t) {
    if (t >= cnt) break;
    float y[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      float a = b[i];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) a = fmaf(w[j][i], to_f32<T>(reinterpret_cast<const T*>(&in[t + j])[i]), a);
      y[i] = silu_f32(a);
    }
    st16<T>(out + static_cast<long long>(t) * p.conv_c, y);
  }
  if (decode && slot >= 0) {
#pragma unroll
    for (int j = 0; j < TAIL; ++j) *reinterpret_cast<uint4*>(st + static_cast<long long>(j) * p.conv_c) = in[j + 1];
  }
}

// ------------------------------------------------------------------ prompts token by token (fp32 models, wide heads)
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
  const T* z = static_cast<const T*>(p.proj) + static_cast<long long>(row0) * p.ld + h * p.vp;
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
        for (int j = 0; j < 4; ++j) {
          const float y = fmaf(skip, to_f32<T>(x[static_cast<long long>(t) * p.conv_c + e + j]), o[j]);
          out[static_cast<long long>(t) * p.ldo + e + j] = from_f32<T>(y * silu_f32(to_f32<T>(z[static_cast<long long>(t) * p.ld + e + j])));
        }
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
  state_step<LPR, PPL, RPT, true>(p.state + (static_cast<long long>(slot) * p.H + h) * p.vp * p.np, p.vp, p.np, p.positions[row] <= 0, sq, sk, sw,
                                  sv, so);
  __syncthreads();
  const T* z = static_cast<const T*>(p.proj) + static_cast<long long>(row) * p.ld + h * p.vp;
  for (int e = tid; e < p.vp; e += 256) out[e] = from_f32<T>(fmaf(p.d[h], sv[e], so[e]) * silu_f32(to_f32<T>(z[e])));
}

// In place: every part of a row's logical columns over its root mean square, times weight and scale. CTA = (row, part).
template <typename T>
__global__ void __launch_bounds__(256)
part_norm_kernel(T* t, long long ld, const float* weight, int vdim, int vp, int per, float eps, float scale) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ float red[8];
  const int row = blockIdx.y, j0 = blockIdx.x * per, tid = threadIdx.x, nt = blockDim.x;
  T* x = t + row * ld;
  auto column = [&](int j) { return vp == vdim ? j : j / vdim * vp + j % vdim; };
  float ss = 0.f;
  const bool vec = vp == vdim && per % 8 == 0 && sizeof(T) == 2;
  if (vec) {
    for (int j = tid * 8; j < per; j += nt * 8) {
      float f[kVec16<T>];
      ld16<T>(x + j0 + j, f);
#pragma unroll
      for (int i = 0; i < kVec16<T>; ++i) ss = fmaf(f[i], f[i], ss);
    }
  } else {
    for (int j = tid; j < per; j += nt) {
      const float f = to_f32<T>(x[column(j0 + j)]);
      ss = fmaf(f, f, ss);
    }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < nt / 32; ++w) ss += red[w];
  const float r = scale / sqrtf(ss / static_cast<float>(per) + eps);
  if (vec) {
    for (int j = tid * 8; j < per; j += nt * 8) {
      float f[kVec16<T>];
      ld16<T>(x + j0 + j, f);
#pragma unroll
      for (int i = 0; i < kVec16<T>; ++i) f[i] *= r * weight[j0 + j + i];
      st16<T>(x + j0 + j, f);
    }
  } else {
    for (int j = tid; j < per; j += nt) {
      const int c = column(j0 + j);
      x[c] = from_f32<T>(to_f32<T>(x[c]) * r * weight[c]);
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

// ints: H, vdim, vp, state, np, groups, taps, rows, n_decode, prompt sequences, blocks of 4 tokens of their portions, projection row
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

// ptrs: proj, xbc, gates, d, state, slots, cu, pos0, out, all from the first prompt row (sequence) on.
TSB_EXPORT int tsb_ssd_prefill(const int* ints, void* const* q, int dtype, void* stream) {
  using namespace tsb;
  SsdParams p{};
  if (!read_ssd(ints, &p) || p.n_seq <= 0) return -2;
  p.proj = q[0]; p.xbc = q[1]; p.gates = static_cast<float2*>(q[2]); p.d = static_cast<const float*>(q[3]); p.state = static_cast<float*>(q[4]);
  p.slots = static_cast<const int*>(q[5]); p.cu = static_cast<const int*>(q[6]); p.pos0 = static_cast<const int*>(q[7]); p.out = q[8];
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) return run_scan<__nv_bfloat16>(p, s);
  if (dtype == 0) return run_scan<float>(p, s);
  return -2;
}

// t [rows, ld] in place; see part_norm_kernel. dtype: 0 = fp32, 1 = bf16.
TSB_EXPORT int tsb_part_norm(void* t, long long ld, const float* weight, int rows, int heads, int vdim, int vp, int parts, float eps,
                             float scale, int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || heads <= 0 || vdim <= 0 || vp < vdim || parts <= 0 || (heads * vdim) % parts || (dtype != 0 && dtype != 1) ||
      (dtype == 1 && (ld % 8 || (reinterpret_cast<uintptr_t>(t) & 15))))
    return -2;
  const int per = heads * vdim / parts;
  const int nt = std::min(256, (per / 8 + 31) / 32 * 32 + 32);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  for (int r0 = 0; r0 < rows; r0 += 65535) {
    const dim3 grid(parts, std::min(rows - r0, 65535));
    if (dtype == 1)
      launch_pdl(part_norm_kernel<__nv_bfloat16>, grid, dim3(nt), 0, s, pdl_all_enabled(), static_cast<__nv_bfloat16*>(t) + r0 * ld, ld, weight, vdim,
                 vp, per, eps, scale);
    else
      launch_pdl(part_norm_kernel<float>, grid, dim3(nt), 0, s, pdl_all_enabled(), static_cast<float*>(t) + r0 * ld, ld, weight, vdim, vp, per, eps,
                 scale);
  }
  return static_cast<int>(cudaGetLastError());
}
