// Real-gated linear recurrent unit behind a short convolution (a Griffin recurrent block without its projections), for
// ragged batches of sequences. Per channel:
//
//   u_t = sum_j conv[j] x_{t - taps + 1 + j} + conv_b              (x: a projection column, plus its bias)
//   r = sigmoid(ra u + ra_b), i = sigmoid(ri u + ri_b)             (ra, ri: block-diagonal square matrices)
//   log a = -r decay, a = exp(log a), S <- a S + sqrt(1 - a^2) i u (decay: 8 softplus(lam), from the caller)
//   out = S gelu(y)                                                (y: another projection column, plus its bias)
//
// Channels are stored block by block, each block padded to kp columns (a multiple of 16; padding channels stay zero), so a
// channel has the same column everywhere: x, y, u, the state and the result. u is rounded to the projection's type, all
// that follows is fp32.
//
//   rglru_conv_kernel   u of every row; for single decoded tokens it also shifts the slot's convolution inputs
//   rglru_step_kernel   single decoded tokens: gates (per-block products), state update, read-out; one launch
//   rglru_chunk_kernel  prompts: gates of 64 tokens of a sequence, and the recurrence over them from a zero state: S_local and
//                       the running product of a, which say what the chunk does to any state it starts from
//   rglru_carry_kernel  prompts: the state at the start of every chunk, and the sequence's last state into its slot
//   rglru_apply_kernel  prompts: S_local + product * carried state, times gelu(y)
#include "head_tile.cuh"
#include "ragged_conv.cuh"

#include <algorithm>

namespace tsb {
namespace {

constexpr int kChunk = 64;      // tokens of a chunk: the row tile of the gate products

struct RglruParams {
  // geometry
  int blocks, kp, C;            // C = blocks * kp
  int off_y;                    // column of y in a projection row (x starts at 0)
  const void* proj;             // [rows, ldp]
  long long ldp;
  float in_scale;
  // weights, fp32 unless noted
  const float* x_bias;          // [C]
  const float* y_bias;          // [C]
  const float* conv_w;          // [taps, C]
  const float* conv_b;          // [C]
  const void* ra;               // [blocks, kp, kp] (out, in), the projection's type
  const void* ri;
  const float* ra_b;            // [C]
  const float* ri_b;
  const float* decay;           // [C]
  int taps;
  // state
  void* conv_state;             // [slots, taps - 1, C]: the projection's values, without scale and bias
  float* state;                 // [slots, C]
  // rows: n_dec single tokens, then the portions
  int rows, n_dec;
  const int* slots;             // [sequences], -1: padding
  const int* positions;         // [rows]
  const int* seq_of;            // [rows]
  const int* cu;                // [portions + 1], from 0
  const int* pos0;              // [portions]
  const int* tile_seq;          // [chunks]
  const int* tile0;             // [portions + 1]
  int n_seq, chunks;
  // scratch and result
  void* u;                      // [rows, C]
  float* s_local;               // [rows - n_dec, C]
  float* a_prod;                // [rows - n_dec, C]
  float* carry;                 // [chunks, C]
  void* out;                    // [rows, ldo]
  long long ldo;
};

// FAST (bf16 models): hardware exponentials and divisions, good to a few fp32 roundings; fp32 models take the exact ones.
template <bool FAST>
__device__ __forceinline__ float sigmoid_g(float x) {
  if constexpr (FAST) return __fdividef(1.f, 1.f + __expf(-x));
  return sigmoid_f32(x);
}
template <bool FAST>
__device__ __forceinline__ float gelu_tanh_g(float z) {
  constexpr float k = 0.79788456080286535588f;     // sqrt(2 / pi)
  const float w = k * fmaf(0.044715f * z * z, z, z);
  // (1 + tanh w) / 2 = 1 / (1 + exp(-2 w))
  if constexpr (FAST) return __fdividef(z, 1.f + __expf(-2.f * w));
  return 0.5f * z * (1.f + tanhf(w));
}
struct Gates {
  float a, b;                   // S <- a S + b
};
template <bool FAST>
__device__ __forceinline__ Gates rglru_gates(float r_lin, float i_lin, float decay, float u) {
  const float x = -sigmoid_g<FAST>(r_lin) * decay;
  if constexpr (FAST) {
    // 1 - a^2 = -(exp(2 x) - 1): by its Taylor series where the difference would cancel (|2 x| < 1/4: the first dropped term
    // is below 2e-6 of the sum)
    const float y = 2.f * x, a = __expf(x);
    const float series = -y * fmaf(y, fmaf(y, fmaf(y, fmaf(y, 1.f / 120.f, 1.f / 24.f), 1.f / 6.f), 0.5f), 1.f);
    const float q = y > -0.25f ? series : fmaf(-a, a, 1.f);
    return {a, sqrtf(q) * sigmoid_g<true>(i_lin) * u};
  }
  return {expf(x), sqrtf(-expm1f(2.f * x)) * sigmoid_f32(i_lin) * u};
}

// A thread takes one 16-byte piece of channels of kConvRows rows; the inputs before a row stay in registers as a window. TAPS = 0:
// any number of taps, every input loaded again.
constexpr int kConvRows = 8;

template <typename T, int TAPS>
__global__ void __launch_bounds__(256)
rglru_conv_kernel(RglruParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>, W = TAPS > 0 ? TAPS : 1;
  const unsigned per = p.C / V, idx = blockIdx.x * 256u + threadIdx.x;
  const int c = static_cast<int>(idx % per) * V;
  // decoded rows one by one, then the portions' rows kConvRows at a time
  int row = static_cast<int>(idx / per), last = row;
  if (row >= p.n_dec) {
    row = p.n_dec + (row - p.n_dec) * kConvRows;
    if (row >= p.rows) return;
    last = min(row + kConvRows, p.rows) - 1;
  }
  const int tail = p.taps - 1;
  float bias[V], cb[V], w[W][V];
#pragma unroll
  for (int i = 0; i < V; ++i) {
    cb[i] = p.conv_b[c + i];
    bias[i] = p.x_bias[c + i];
  }
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < V; ++i) w[j][i] = p.conv_w[static_cast<long long>(j) * p.C + c + i];
  }
  if constexpr (TAPS > 0) {
    // eight rows in the middle of a portion: every input is requested before the first is used
    if (row >= p.n_dec && last - row == kConvRows - 1) {
      const int seq = p.seq_of[row];
      if (p.seq_of[last] == seq && row - tail >= p.n_dec + p.cu[seq - p.n_dec]) {
        const T* x = static_cast<const T*>(p.proj) + (row - tail) * p.ldp + c;
        uint4 raw[kConvRows + TAPS - 1];
#pragma unroll
        for (int r = 0; r < kConvRows + TAPS - 1; ++r) raw[r] = *reinterpret_cast<const uint4*>(x + r * p.ldp);
        // the scale goes into the taps, the biases that they multiply into one
#pragma unroll
        for (int i = 0; i < V; ++i) {
          float sum = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS; ++j) {
            sum += w[j][i];
            w[j][i] *= p.in_scale;
          }
          cb[i] = fmaf(sum, bias[i], cb[i]);
        }
#pragma unroll
        for (int r = 0; r < kConvRows; ++r) {
          float acc[V];
#pragma unroll
          for (int i = 0; i < V; ++i) {
            acc[i] = cb[i];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) acc[i] = fmaf(w[j][i], to_f32<T>(reinterpret_cast<const T*>(&raw[r + j])[i]), acc[i]);
          }
          st16<T>(static_cast<T*>(p.u) + static_cast<long long>(row + r) * p.C + c, acc);
        }
        return;
      }
    }
  }
  float win[W][V];
  for (int first_row = row; row <= last; ++row) {
    const T* x = static_cast<const T*>(p.proj) + row * p.ldp + c;
    T* u = static_cast<T*>(p.u) + static_cast<long long>(row) * p.C + c;
    float acc[V];
    const bool decoded = row < p.n_dec;
    const int seq = decoded ? row : p.seq_of[row];
    const int slot = p.slots[seq];
    if (slot < 0) {
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = 0.f;
      st16<T>(u, acc);
      continue;
    }
    T* st = static_cast<T*>(p.conv_state) + static_cast<long long>(slot) * tail * p.C + c;
    const int start = decoded ? row : p.n_dec + p.cu[seq - p.n_dec];      // first row of this sequence in the batch
    const int pos = p.positions[row];
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] = cb[i];
    auto input = [&](int back, float (&v)[V]) {      // the input `back` tokens ago, with scale and bias
      const int at = row - back - start;             // negative: in the slot, which holds the last `tail` inputs
      if (back > pos) {                              // before the start of the sequence
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = 0.f;
        return;
      }
      if (at >= 0) ld16<T>(x - back * p.ldp, v);
      else ld16<T>(st + static_cast<long long>(tail + at) * p.C, v);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = fmaf(v[i], p.in_scale, bias[i]);
    };
    if constexpr (TAPS > 0) {
      if (row == first_row || row == start) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) input(TAPS - 1 - j, win[j]);
      } else {
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
          for (int i = 0; i < V; ++i) win[j][i] = win[j + 1][i];
        input(0, win[TAPS - 1]);
      }
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(w[j][i], win[j][i], acc[i]);
    } else {
      for (int j = 0; j <= tail; ++j) {
        input(tail - j, win[0]);
        const float* wj = p.conv_w + static_cast<long long>(j) * p.C + c;
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(wj[i], win[0][i], acc[i]);
      }
    }
    st16<T>(u, acc);
    if (decoded) {
      for (int j = 0; j < tail; ++j) {
        uint4 next = *reinterpret_cast<const uint4*>(x);
        if (j + 1 < tail) next = *reinterpret_cast<const uint4*>(st + static_cast<long long>(j + 1) * p.C);
        *reinterpret_cast<uint4*>(st + static_cast<long long>(j) * p.C) = next;
      }
    }
  }
}

template <typename T, int BM>
__global__ void __launch_bounds__(128)
rglru_step_kernel(RglruParams p) {
  using Tile = HeadTile<T, BM, 2>;
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  const int n0 = blockIdx.x * 64, blk = blockIdx.y, m0 = blockIdx.z * BM;
  const int cols = min(64, p.kp - n0), rows = min(BM, p.n_dec - m0);
  const T* u = static_cast<const T*>(p.u) + static_cast<long long>(m0) * p.C + blk * p.kp;
  const long long w0 = (static_cast<long long>(blk) * p.kp + n0) * p.kp;
  const T* const w[2] = {static_cast<const T*>(p.ra) + w0, static_cast<const T*>(p.ri) + w0};
  const float* acc = Tile::run(smem, u, p.C, rows, w, p.kp, cols, p.kp);
  const int n = threadIdx.x & 63, c = blk * p.kp + n0 + n;
  if (n >= cols) return;
  const float rb = p.ra_b[c], ib = p.ri_b[c], dc = p.decay[c], yb = p.y_bias[c];
  constexpr int kPer = 8;                          // rows whose inputs are requested together
#pragma unroll
  for (int r0 = threadIdx.x >> 6; r0 < BM; r0 += 2 * kPer) {
    int slot[kPer];
    float uu[kPer], y[kPer], s[kPer];
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int m = min(r0 + 2 * i, rows - 1), row = m0 + m;
      slot[i] = p.slots[row];
      uu[i] = to_f32<T>(u[static_cast<long long>(m) * p.C + n0 + n]);
      y[i] = to_f32<T>(static_cast<const T*>(p.proj)[row * p.ldp + p.off_y + c]);
      s[i] = slot[i] >= 0 && p.positions[row] > 0 ? p.state[static_cast<long long>(slot[i]) * p.C + c] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int m = r0 + 2 * i;
      if (m >= rows) break;
      const Gates g = rglru_gates<sizeof(T) == 2>(acc[m * Tile::kLdC + n] + rb, acc[(BM + m) * Tile::kLdC + n] + ib, dc, uu[i]);
      const float next = fmaf(g.a, s[i], g.b);
      float z = 0.f;                               // (a row without a sequence)
      if (slot[i] >= 0) {
        p.state[static_cast<long long>(slot[i]) * p.C + c] = next;
        z = next * gelu_tanh_g<sizeof(T) == 2>(fmaf(y[i], p.in_scale, yb));
      }
      static_cast<T*>(p.out)[static_cast<long long>(m0 + m) * p.ldo + c] = from_f32<T>(z);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128)
rglru_chunk_kernel(RglruParams p) {
  using Tile = HeadTile<T, kChunk, 2>;
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  const int n0 = blockIdx.x * 64, blk = blockIdx.y, chunk = blockIdx.z;
  const int seq = p.tile_seq[chunk];
  const int t0 = (chunk - p.tile0[seq]) * kChunk;
  const int row0 = p.cu[seq] + t0, rows = min(kChunk, p.cu[seq + 1] - row0);     // rows of the portions, from 0
  const int cols = min(64, p.kp - n0);
  const T* u = static_cast<const T*>(p.u) + static_cast<long long>(p.n_dec + row0) * p.C + blk * p.kp;
  const long long w0 = (static_cast<long long>(blk) * p.kp + n0) * p.kp;
  const T* const w[2] = {static_cast<const T*>(p.ra) + w0, static_cast<const T*>(p.ri) + w0};
  const int tid = threadIdx.x, n = tid & 63, c = blk * p.kp + n0 + n;
  const bool ok = n < cols;
  // this thread's inputs of the gates, requested ahead of the products: rows (tid / 64) + 2 i of one channel
  T uu[kChunk / 2];
  {
    const T* uc = u + n0 + (ok ? n : 0);
#pragma unroll
    for (int i = 0; i < kChunk / 2; ++i) uu[i] = uc[static_cast<long long>(min((tid >> 6) + 2 * i, rows - 1)) * p.C];
  }
  float* acc = Tile::run(smem, u, p.C, rows, w, p.kp, cols, p.kp);
  float* sa = acc;
  float* sb = acc + kChunk * Tile::kLdC;
  {
    const float rb = ok ? p.ra_b[c] : 0.f, ib = ok ? p.ri_b[c] : 0.f, dc = ok ? p.decay[c] : 0.f;
#pragma unroll
    for (int i = 0; i < kChunk / 2; ++i) {         // (rows past the end compute on zeros and are not used)
      const int at = ((tid >> 6) + 2 * i) * Tile::kLdC + n;
      const Gates g = rglru_gates<sizeof(T) == 2>(sa[at] + rb, sb[at] + ib, dc, to_f32<T>(uu[i]));
      sa[at] = g.a;
      sb[at] = g.b;
    }
  }
  __syncthreads();
  // two halves of the chunk at once, each from a zero state
  constexpr int kHalf = kChunk / 2;
  const int h0 = (tid >> 6) * kHalf, cnt = min(kHalf, rows - h0);
  float s = 0.f, a = 1.f;
#pragma unroll 8
  for (int m = 0; m < cnt; ++m) {
    const int at = (h0 + m) * Tile::kLdC + n;
    const float am = sa[at];
    s = fmaf(am, s, sb[at]);
    a *= am;
    sa[at] = a;
    sb[at] = s;
  }
  __syncthreads();
  if (!ok) return;
  const bool second = h0 > 0;
  const float s_in = second ? sb[(kHalf - 1) * Tile::kLdC + n] : 0.f, a_in = second ? sa[(kHalf - 1) * Tile::kLdC + n] : 1.f;
#pragma unroll 4
  for (int m = 0; m < cnt; ++m) {
    const int at = (h0 + m) * Tile::kLdC + n;
    const long long o = static_cast<long long>(row0 + h0 + m) * p.C + c;
    p.s_local[o] = fmaf(sa[at], s_in, sb[at]);
    p.a_prod[o] = sa[at] * a_in;
  }
}

__global__ void __launch_bounds__(64)
rglru_carry_kernel(RglruParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const int c = blockIdx.x * 64 + threadIdx.x, seq = blockIdx.y;
  if (c >= p.C) return;
  const int row0 = p.cu[seq], n = p.cu[seq + 1] - row0;
  const int slot = p.slots[p.n_dec + seq];
  if (n <= 0 || slot < 0) return;
  float* st = p.state + static_cast<long long>(slot) * p.C + c;
  float s = p.pos0[seq] > 0 ? *st : 0.f;
  const int chunk0 = p.tile0[seq], chunks = (n + kChunk - 1) / kChunk;
  constexpr int kAhead = 8;
  for (int k0 = 0; k0 < chunks; k0 += kAhead) {
    float a[kAhead], b[kAhead];
#pragma unroll
    for (int k = 0; k < kAhead; ++k) {
      const long long o = static_cast<long long>(row0 + min((k0 + k + 1) * kChunk, n) - 1) * p.C + c;
      a[k] = p.a_prod[o];
      b[k] = p.s_local[o];
    }
#pragma unroll
    for (int k = 0; k < kAhead; ++k) {
      if (k0 + k >= chunks) break;
      p.carry[static_cast<long long>(chunk0 + k0 + k) * p.C + c] = s;
      s = fmaf(a[k], s, b[k]);
    }
  }
  *st = s;
}

// 64 threads of 4 channels, four groups of rows.
template <typename T>
__global__ void __launch_bounds__(256)
rglru_apply_kernel(RglruParams p) {
  pdl_trigger();
  pdl_grid_wait();
  const int c = (blockIdx.x * 64 + (threadIdx.x & 63)) * 4, chunk = blockIdx.y;
  if (c >= p.C) return;
  const int seq = p.tile_seq[chunk];
  const int row0 = p.cu[seq] + (chunk - p.tile0[seq]) * kChunk, rows = min(kChunk, p.cu[seq + 1] - row0);
  const float4 in = *reinterpret_cast<const float4*>(p.carry + static_cast<long long>(chunk) * p.C + c);
  const float4 yb = *reinterpret_cast<const float4*>(p.y_bias + c);
#pragma unroll 2
  for (int m = threadIdx.x >> 6; m < rows; m += 4) {
    const long long o = static_cast<long long>(row0 + m) * p.C + c, row = p.n_dec + row0 + m;
    const float4 s = __ldcs(reinterpret_cast<const float4*>(p.s_local + o)), a = __ldcs(reinterpret_cast<const float4*>(p.a_prod + o));
    const T* yp = static_cast<const T*>(p.proj) + row * p.ldp + p.off_y + c;
    float y[4];
    if constexpr (sizeof(T) == 2) {
      const uint2 r = *reinterpret_cast<const uint2*>(yp);
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] = to_f32<T>(reinterpret_cast<const T*>(&r)[i]);
    } else {
      const float4 r = *reinterpret_cast<const float4*>(yp);
      y[0] = r.x; y[1] = r.y; y[2] = r.z; y[3] = r.w;
    }
    const float z0 = fmaf(a.x, in.x, s.x) * gelu_tanh_g<sizeof(T) == 2>(fmaf(y[0], p.in_scale, yb.x));
    const float z1 = fmaf(a.y, in.y, s.y) * gelu_tanh_g<sizeof(T) == 2>(fmaf(y[1], p.in_scale, yb.y));
    const float z2 = fmaf(a.z, in.z, s.z) * gelu_tanh_g<sizeof(T) == 2>(fmaf(y[2], p.in_scale, yb.z));
    const float z3 = fmaf(a.w, in.w, s.w) * gelu_tanh_g<sizeof(T) == 2>(fmaf(y[3], p.in_scale, yb.w));
    T* out = static_cast<T*>(p.out) + row * p.ldo + c;
    if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(out) = make_uint2(pack_bf16x2(z0, z1), pack_bf16x2(z2, z3));
    else *reinterpret_cast<float4*>(out) = make_float4(z0, z1, z2, z3);
  }
}

template <typename K>
int opt_in_smem(K kern, PerDeviceFlag* flag, int bytes) {
  if (!flag->unset()) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e == cudaSuccess) flag->set();
  return static_cast<int>(e);
}

template <typename T, int BM>
int launch_step(const RglruParams& p, cudaStream_t s) {
  using Tile = HeadTile<T, BM, 2>;
  auto kern = rglru_step_kernel<T, BM>;
  static PerDeviceFlag attr;
  if (const int e = opt_in_smem(kern, &attr, Tile::kSmem)) return e;
  const dim3 grid((p.kp + 63) / 64, p.blocks, (p.n_dec + BM - 1) / BM);
  launch_pdl(kern, grid, dim3(128), Tile::kSmem, s, pdl_all_enabled(), p);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int run_rglru(const RglruParams& p, cudaStream_t s) {
  const bool pdl = pdl_all_enabled();
  const long long pieces = static_cast<long long>(p.rows) * (p.C / kVec16<T>);
  if (pieces > 0x7fffff00LL) return -2;
  const long long threads = (p.n_dec + (p.rows - p.n_dec + kConvRows - 1) / kConvRows) * static_cast<long long>(p.C / kVec16<T>);
  const dim3 cgrid(static_cast<unsigned>((threads + 255) / 256));
  switch (p.taps) {
    case 2: launch_pdl(rglru_conv_kernel<T, 2>, cgrid, dim3(256), 0, s, pdl, p); break;
    case 3: launch_pdl(rglru_conv_kernel<T, 3>, cgrid, dim3(256), 0, s, pdl, p); break;
    case 4: launch_pdl(rglru_conv_kernel<T, 4>, cgrid, dim3(256), 0, s, pdl, p); break;
    default: launch_pdl(rglru_conv_kernel<T, 0>, cgrid, dim3(256), 0, s, pdl, p); break;
  }
  int rc = static_cast<int>(cudaGetLastError());
  if (rc) return rc;
  if (p.n_dec > 0) {
    rc = p.n_dec <= 128 ? launch_step<T, 16>(p, s) : launch_step<T, 64>(p, s);
    if (rc) return rc;
  }
  if (p.rows > p.n_dec) {
    if (p.taps > 1) {
      launch_pdl(conv_state_kernel<T>, dim3((p.C + 255) / 256, p.n_seq), dim3(256), 0, s, pdl,
                 static_cast<const T*>(p.proj) + p.n_dec * p.ldp, p.ldp, p.C, static_cast<T*>(p.conv_state), p.cu, p.slots + p.n_dec,
                 p.pos0, p.taps - 1);
      rc = static_cast<int>(cudaGetLastError());
      if (rc) return rc;
    }
    using Tile = HeadTile<T, kChunk, 2>;
    auto kern = rglru_chunk_kernel<T>;
    static PerDeviceFlag attr;
    if (const int e = opt_in_smem(kern, &attr, Tile::kSmem)) return e;
    launch_pdl(kern, dim3((p.kp + 63) / 64, p.blocks, p.chunks), dim3(128), Tile::kSmem, s, pdl, p);
    launch_pdl(rglru_carry_kernel, dim3((p.C + 63) / 64, p.n_seq), dim3(64), 0, s, pdl, p);
    launch_pdl(rglru_apply_kernel<T>, dim3((p.C + 255) / 256, p.chunks), dim3(256), 0, s, pdl, p);
    rc = static_cast<int>(cudaGetLastError());
  }
  return rc;
}

}  // namespace
}  // namespace tsb

// One mixer over a ragged batch: rows [0, n_dec) are single tokens of the sequences slots[0 .. n_dec), the rest are portions
// cut into chunks of 64 tokens from each portion's first row. ints: blocks, kp, off_y, taps, rows, n_dec, n_seq, chunks.
// dtype: 0 = fp32, 1 = bf16. Scratch: u [rows, C] in the projection's type; s_local, a_prod [rows - n_dec, C] and carry
// [chunks, C] in fp32. See RglruParams.
TSB_EXPORT int tsb_rglru(const int* ints, float in_scale, const void* proj, long long ldp, const float* x_bias, const float* y_bias,
                         const float* conv_w, const float* conv_b, const void* ra, const void* ri, const float* ra_b, const float* ri_b,
                         const float* decay, void* conv_state, float* state, const int* slots, const int* positions, const int* seq_of,
                         const int* cu, const int* pos0, const int* tile_seq, const int* tile0, void* u, float* s_local, float* a_prod,
                         float* carry, void* out, long long ldo, int dtype, void* stream) {
  using namespace tsb;
  RglruParams p{};
  p.blocks = ints[0]; p.kp = ints[1]; p.off_y = ints[2]; p.taps = ints[3]; p.rows = ints[4]; p.n_dec = ints[5]; p.n_seq = ints[6];
  p.chunks = ints[7];
  p.C = p.blocks * p.kp;
  if (p.blocks <= 0 || p.blocks > 65535 || p.kp <= 0 || p.kp % 16 || p.taps < 1 || p.rows <= 0 || p.n_dec < 0 || p.n_dec > p.rows ||
      p.n_seq < 0 || p.n_seq > 65535 || p.chunks > 65535 || p.off_y % 8 || ldp % 8 || ldo % 4 || (p.n_dec + 15) / 16 > 65535 ||
      (p.rows > p.n_dec && (p.n_seq < 1 || p.chunks < 1 || !cu || !pos0 || !tile_seq || !tile0 || !seq_of || !s_local || !a_prod || !carry)))
    return -2;
  p.proj = proj; p.ldp = ldp; p.in_scale = in_scale; p.x_bias = x_bias; p.y_bias = y_bias; p.conv_w = conv_w; p.conv_b = conv_b;
  p.ra = ra; p.ri = ri; p.ra_b = ra_b; p.ri_b = ri_b; p.decay = decay; p.conv_state = conv_state; p.state = state; p.slots = slots;
  p.positions = positions; p.seq_of = seq_of; p.cu = cu; p.pos0 = pos0; p.tile_seq = tile_seq; p.tile0 = tile0; p.u = u;
  p.s_local = s_local; p.a_prod = a_prod; p.carry = carry; p.out = out; p.ldo = ldo;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) return run_rglru<__nv_bfloat16>(p, s);
  if (dtype == 0) return run_rglru<float>(p, s);
  return -2;
}
