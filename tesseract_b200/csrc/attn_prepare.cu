// What happens to a packed projection row [q: H heads | k: Hkv | v: Hkv | ..] before attention: biases, a norm of q and k (per
// head, or over all heads at once), rotation by position, queries that grow louder with it, values mixed with those of an earlier layer; q goes to a buffer of its
// own, k and v to the token's pool slot and, for prompt rows, to the key axis of the tensor-core kernel.
//
// One CTA per row. LPH lanes share a head (16 bytes each, PPL times), so a warp takes 32 / LPH heads at once. Everything between
// load and store is fp32.
#include "warp_mma.cuh"

namespace tsb {
namespace {

struct PrepareParams {
  int rows, H, Hkv, D, dim, hp, off_k, off_v, norm, bs, n_decode, ld, D_first;    // norm: 0 none, 1 unit heads, 2 heads with a weight, 3 whole
  float eps, vmix;
  float q_coef, q_every;      // q *= 1 + q_coef ln(floor((position + 1) / q_every) + 1); q_coef = 0: not
  const void* proj;
  const float* bias;          // [off_v + Hkv * D] or null
  const float* q_norm;
  const float* k_norm;
  const float2* table;        // [positions, hp] or null
  const int* positions;
  const int* slots;
  void* q;                    // [rows, H, D]
  void* k_pool;               // [blocks, Hkv, bs, D]
  void* v_pool;
  const void* v_first;        // [blocks, Hkv, bs, D_first] or null
  void* stage;                // [keys, 2 Hkv, D] or null
  const int* stage_rows;      // [rows - n_decode]
};

// V consecutive floats (16-byte aligned), multiplied in.
template <int V>
__device__ __forceinline__ void scale_by(float (&f)[V], float r, const float* w) {
  if (!w) {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] *= r;
    return;
  }
#pragma unroll
  for (int i = 0; i < V; i += 4) {
    const float4 a = *reinterpret_cast<const float4*>(w + i);
    f[i] *= r * a.x; f[i + 1] *= r * a.y; f[i + 2] *= r * a.z; f[i + 3] *= r * a.w;
  }
}

template <typename T, int LPH, int PPL>
__global__ void __launch_bounds__(256)
attn_prepare_kernel(PrepareParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec16<T>;
  __shared__ float red[2][8];
  const int row = blockIdx.x, tid = threadIdx.x, gl = tid % LPH, first = tid / LPH, step = blockDim.x / LPH;
  const T* x = static_cast<const T*>(p.proj) + static_cast<long long>(row) * p.ld;
  const int units = p.H + 2 * p.Hkv, D = p.D;
  auto load = [&](int col, float (&f)[V]) {         // V columns of the row, with their biases
    ld16<T>(x + col, f);
    if (p.bias) {
#pragma unroll
      for (int i = 0; i < V; i += 4) {
        const float4 b = *reinterpret_cast<const float4*>(p.bias + col + i);
        f[i] += b.x; f[i + 1] += b.y; f[i + 2] += b.z; f[i + 3] += b.w;
      }
    }
  };
  float whole_q = 0.f, whole_k = 0.f;
  if (p.norm == 3) {
    float sq = 0.f, sk = 0.f;
    for (int c = tid * V; c < (p.H + p.Hkv) * D; c += blockDim.x * V) {
      const bool is_k = c >= p.H * D;
      float f[V], s = 0.f;
      load(is_k ? p.off_k + c - p.H * D : c, f);
#pragma unroll
      for (int i = 0; i < V; ++i) s = fmaf(f[i], f[i], s);
      if (is_k) sk += s;
      else sq += s;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((tid & 31) == 0) {
      red[0][tid >> 5] = sq;
      red[1][tid >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
    for (int w = 0; w < static_cast<int>(blockDim.x) / 32; ++w) {
      sq += red[0][w];
      sk += red[1][w];
    }
    whole_q = 1.f / sqrtf(sq / static_cast<float>(p.H * p.dim) + p.eps);
    whole_k = 1.f / sqrtf(sk / static_cast<float>(p.Hkv * p.dim) + p.eps);
  }
  const int slot = p.slots[row];
  const long long page = slot >= 0 ? static_cast<long long>(slot / p.bs) * p.Hkv * p.bs + slot % p.bs : 0;
  const int stage_row = p.stage && row >= p.n_decode ? p.stage_rows[row - p.n_decode] : -1;
  const float2* turn = p.table && p.hp > 0 ? p.table + static_cast<long long>(max(p.positions[row], 0)) * p.hp : nullptr;
  const float loud = p.q_coef != 0.f ? 1.f + p.q_coef * logf(floorf(static_cast<float>(max(p.positions[row], 0) + 1) / p.q_every) + 1.f) : 1.f;
  constexpr int U = PPL == 1 ? 2 : 1;               // heads whose loads are requested together
  for (int u0 = 0; u0 < units; u0 += U * step) {    // (every lane takes every turn: the sums below are shuffles)
    float f[U][PPL][V], ss[U];
    int kind[U], head[U], col[U];
#pragma unroll
    for (int q = 0; q < U; ++q) {
      const int u = u0 + q * step + first;
      kind[q] = u < p.H ? 0 : u < p.H + p.Hkv ? 1 : u < units ? 2 : 3;      // q, k, v, nothing
      head[q] = kind[q] == 0 ? u : kind[q] == 1 ? u - p.H : u - p.H - p.Hkv;
      col[q] = (kind[q] == 0 ? 0 : kind[q] == 1 ? p.off_k : p.off_v) + head[q] * D;
#pragma unroll
      for (int k = 0; k < PPL; ++k) {
        const int d = (gl + k * LPH) * V;
#pragma unroll
        for (int i = 0; i < V; ++i) f[q][k][i] = 0.f;
        if (kind[q] < 3 && d < D) load(col[q] + d, f[q][k]);
      }
    }
#pragma unroll
    for (int q = 0; q < U; ++q) {
      ss[q] = 0.f;
#pragma unroll
      for (int k = 0; k < PPL; ++k)
#pragma unroll
        for (int i = 0; i < V; ++i) ss[q] = fmaf(f[q][k][i], f[q][k][i], ss[q]);
      if (p.norm == 1 || p.norm == 2) {
#pragma unroll
        for (int o = LPH / 2; o; o >>= 1) ss[q] += __shfl_xor_sync(0xffffffffu, ss[q], o);
      }
    }
#pragma unroll
    for (int q = 0; q < U; ++q) {
      if (kind[q] == 3) continue;
      const float rs = p.norm == 3 ? (kind[q] == 0 ? whole_q : whole_k) : 1.f / sqrtf(ss[q] / static_cast<float>(p.dim) + p.eps);
      const float* w = p.norm < 2 ? nullptr : (kind[q] == 0 ? p.q_norm : p.k_norm) + (p.norm == 3 ? head[q] * D : 0);
#pragma unroll
      for (int k = 0; k < PPL; ++k) {
        const int d = (gl + k * LPH) * V;
        if (d >= D) continue;
        float(&x8)[V] = f[q][k];
        if (kind[q] == 2) {
          if (p.v_first) {
            float v0[V] = {};
            if (slot >= 0 && d < p.D_first)
              ld16<T>(static_cast<const T*>(p.v_first) + (page + static_cast<long long>(head[q]) * p.bs) * p.D_first + d, v0);
#pragma unroll
            for (int i = 0; i < V; ++i) x8[i] = (1.f - p.vmix) * x8[i] + p.vmix * v0[i];
          }
        } else {
          if (p.norm) scale_by<V>(x8, rs, w ? w + d : nullptr);
          if (turn && d < 2 * p.hp) {
            const bool second = d >= p.hp;
            const int i0 = second ? d - p.hp : d, other = second ? i0 : d + p.hp;
            float g[V];
            load(col[q] + other, g);
            if (p.norm) scale_by<V>(g, rs, w ? w + other : nullptr);
#pragma unroll
            for (int i = 0; i < V; i += 2) {
              const float4 cs = *reinterpret_cast<const float4*>(turn + i0 + i);
              const float s0 = second ? cs.y : -cs.y, s1 = second ? cs.w : -cs.w;
              x8[i] = x8[i] * cs.x + g[i] * s0;
              x8[i + 1] = x8[i + 1] * cs.z + g[i + 1] * s1;
            }
          }
        }
        if (kind[q] == 0) {
#pragma unroll
          for (int i = 0; i < V; ++i) x8[i] *= loud;
          st16<T>(static_cast<T*>(p.q) + (static_cast<long long>(row) * p.H + head[q]) * D + d, x8);
          continue;
        }
        if (slot >= 0) st16<T>(static_cast<T*>(kind[q] == 1 ? p.k_pool : p.v_pool) + (page + static_cast<long long>(head[q]) * p.bs) * D + d, x8);
        if (stage_row >= 0)
          st16<T>(static_cast<T*>(p.stage) + (static_cast<long long>(stage_row) * 2 * p.Hkv + (kind[q] == 1 ? 0 : p.Hkv) + head[q]) * D + d, x8);
      }
    }
  }
}

template <typename T>
int launch_prepare(const PrepareParams& p, cudaStream_t s) {
  const int pieces = p.D / kVec16<T>;
  const int lph = pieces <= 8 ? 8 : pieces <= 16 ? 16 : 32;
  const int lanes = (p.H + 2 * p.Hkv) * lph;
  const int nt = lanes >= 256 ? 256 : (lanes + 31) / 32 * 32;
  const bool pdl = pdl_all_enabled();
#define TSB_PREP(L, N) launch_pdl(attn_prepare_kernel<T, L, N>, dim3(p.rows), dim3(nt), 0, s, pdl, p)
  if (lph == 8) TSB_PREP(8, 1);
  else if (lph == 16) TSB_PREP(16, 1);
  else if (pieces <= 32) TSB_PREP(32, 1);
  else TSB_PREP(32, 2);
#undef TSB_PREP
  return static_cast<int>(cudaGetLastError());
}

}  // namespace
}  // namespace tsb

// ints: rows, H, Hkv, D, dim, hp, off_k, off_v, norm, bs, n_decode, row stride, head size of v_first; floats: eps, vmix, q_coef, q_every; ptrs: proj, bias, q_norm, k_norm,
// table, positions, slots, q, k_pool, v_pool, v_first, stage, stage_rows (see PrepareParams). dtype: 0 = fp32, 1 = bf16. D is a
// multiple of 32, up to 256; rows and sections start on 16 bytes.
TSB_EXPORT int tsb_attn_prepare(const int* v, const float* f, void* const* q, int dtype, void* stream) {
  using namespace tsb;
  PrepareParams p{v[0], v[1], v[2], v[3], v[4], v[5], v[6], v[7], v[8], v[9], v[10], v[11], v[12], f[0], f[1], f[2], f[3], q[0], static_cast<const float*>(q[1]),
                  static_cast<const float*>(q[2]), static_cast<const float*>(q[3]), static_cast<const float2*>(q[4]),
                  static_cast<const int*>(q[5]), static_cast<const int*>(q[6]), q[7], q[8], q[9], q[10], q[11], static_cast<const int*>(q[12])};
  if (p.rows <= 0 || p.H <= 0 || p.Hkv <= 0 || p.D <= 0 || p.D % 32 || p.D > 256 || p.dim <= 0 || p.dim > p.D || p.hp % 8 || 2 * p.hp > p.D ||
      p.off_k % 8 || p.off_v % 8 || p.ld % 8 || p.norm < 0 || p.norm > 3 || (p.norm >= 2 && (!p.q_norm || !p.k_norm)) || p.bs <= 0 ||
      (p.q_coef != 0.f && !(p.q_every > 0.f)) || (p.stage && !p.stage_rows) || (p.v_first && (p.D_first <= 0 || p.D_first % 8)) || (reinterpret_cast<uintptr_t>(p.proj) & 15))
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) return launch_prepare<__nv_bfloat16>(p, s);
  if (dtype == 0) return launch_prepare<float>(p, s);
  return -2;
}
