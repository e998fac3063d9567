// Paged attention pieces for ragged batches: portions of prompts beside single decoded tokens, with an optional mask (chunks or
// a window) and the other score forms of attn_form.cuh.
//
//   ragged_append_kernel   adds the projection biases to a packed [q | k | v] row, writes q to a buffer of its own, and
//                          stores k and v in the pool slot of the token and, for prompt rows, in the contiguous key axis
//                          that the tcgen05 attention kernel reads (`stage`).
//   stage_gather_kernel    copies keys and values that earlier portions left in the pool to the key axis.
//   ragged_attn_kernel     attention of each row over the pool: one warp per (row, head), fp32 arithmetic. Serves fp32
//                          models and head sizes that the tensor-core kernels do not take.
#include "attn_form.cuh"

#include <algorithm>

namespace tsb {
namespace {

template <typename T>
constexpr int kVec = 16 / sizeof(T);

template <typename T>
__device__ __forceinline__ void load16(const T* p, float (&f)[kVec<T>]) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const T* e = reinterpret_cast<const T*>(&a);
#pragma unroll
  for (int i = 0; i < kVec<T>; ++i) f[i] = to_f32<T>(e[i]);
}
template <typename T>
__device__ __forceinline__ uint4 pack16(const float (&f)[kVec<T>]) {
  uint4 a;
  T* e = reinterpret_cast<T*>(&a);
#pragma unroll
  for (int i = 0; i < kVec<T>; ++i) e[i] = from_f32<T>(f[i]);
  return a;
}

template <typename T>
__global__ void __launch_bounds__(256)
ragged_append_kernel(const T* qkv, long long ld, const float* bias, const int* slots, T* q_out, T* k_pool, T* v_pool, T* stage,
                     const int* stage_rows, int stage_from, int rows, int H, int Hkv, int D, int bs) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec<T>;
  const int vph = D / V;                       // vectors per head
  const int vpr = (H + 2 * Hkv) * vph;
  const unsigned idx = blockIdx.x * 256u + threadIdx.x;   // (the launch checks that the count fits)
  const int row = static_cast<int>(idx / vpr), w = static_cast<int>(idx % vpr);
  if (row >= rows) return;
  const int head = w / vph, d = (w % vph) * V;
  const T* src = qkv + row * ld + head * D + d;
  float f[V];
  load16<T>(src, f);
  if (bias) {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] += bias[head * D + d + i];
  }
  const uint4 val = pack16<T>(f);
  if (head < H) {
    *reinterpret_cast<uint4*>(q_out + (static_cast<long long>(row) * H + head) * D + d) = val;
    return;
  }
  const int hk = (head - H) % Hkv;
  const bool is_v = head >= H + Hkv;
  const int slot = slots[row];
  if (slot >= 0) {
    T* pool = is_v ? v_pool : k_pool;
    *reinterpret_cast<uint4*>(pool + ((static_cast<long long>(slot / bs) * Hkv + hk) * bs + slot % bs) * D + d) = val;
  }
  if (stage && row >= stage_from) {
    const int sr = stage_rows[row - stage_from];
    *reinterpret_cast<uint4*>(stage + (static_cast<long long>(sr) * 2 * Hkv + (head - H)) * D + d) = val;
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
stage_gather_kernel(const T* k_pool, const T* v_pool, T* stage, const int* dst_rows, const int* src_slots, int n, int Hkv, int D,
                    int bs) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int V = kVec<T>;
  const int vph = D / V, vpr = 2 * Hkv * vph;
  const unsigned idx = blockIdx.x * 256u + threadIdx.x;
  const int i = static_cast<int>(idx / vpr), w = static_cast<int>(idx % vpr);
  if (i >= n) return;
  const int head = w / vph, d = (w % vph) * V;
  const int slot = src_slots[i];
  const T* pool = head < Hkv ? k_pool : v_pool;
  const int hk = head < Hkv ? head : head - Hkv;
  *reinterpret_cast<uint4*>(stage + (static_cast<long long>(dst_rows[i]) * 2 * Hkv + head) * D + d) =
      *reinterpret_cast<const uint4*>(pool + ((static_cast<long long>(slot / bs) * Hkv + hk) * bs + slot % bs) * D + d);
}

struct RaggedAttnParams {
  const void* q;          // [rows, ld_q], head h at h * D
  const void* k_pool;
  const void* v_pool;
  const int* tables;      // [sequences, table_ld]
  const int* seq_of;      // [rows] (null: row i is sequence i)
  const int* pos;         // [rows], < 0: no keys (padding)
  void* o;                // [rows, gate.ldo], head h at h * D
  long long ld_q;
  int rows, H, Hkv, bs, nb, table_ld;
  AttnForm form;
  AttnGate gate;
  int* status;
};

// EPL = D / 32 consecutive dimensions per lane. Keys are taken four at a time to overlap their loads and reductions.
template <typename T, int EPL>
__global__ void __launch_bounds__(128)
ragged_attn_kernel(RaggedAttnParams p) {
  pdl_trigger();
  pdl_grid_wait();
  constexpr int D = EPL * 32;
  const long long w = blockIdx.x * 4ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= static_cast<long long>(p.rows) * p.H) return;
  const int row = static_cast<int>(w / p.H), h = static_cast<int>(w % p.H);
  const int hk = h / (p.H / p.Hkv);
  const int* table = p.tables + static_cast<long long>(p.seq_of ? p.seq_of[row] : row) * p.table_ld;
  const T* qr = static_cast<const T*>(p.q) + row * p.ld_q + h * D;
  float q[EPL], o[EPL];
#pragma unroll
  for (int i = 0; i < EPL; ++i) {
    q[i] = to_f32<T>(qr[lane + 32 * i]);
    o[i] = 0.f;
  }
  const int pos = p.pos[row];
  int t = pos >= 0 ? p.form.first(pos) : 0;
  const float slope = p.form.slopes ? p.form.slopes[h] : 0.f;
  float m = -INFINITY, l = 0.f;
  for (; t <= pos; t += 4) {
    float s[4];
    long long base[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int tt = min(t + j, pos);
      int blk = table[tt / p.bs];
      if (blk < 0 || blk >= p.nb) {
        if (p.status) atomicCAS(p.status, kStatusOk, kStatusBadIndex);
        blk = 0;
      }
      base[j] = ((static_cast<long long>(blk) * p.Hkv + hk) * p.bs + tt % p.bs) * D;
      s[j] = 0.f;
#pragma unroll
      for (int i = 0; i < EPL; ++i) s[j] = fmaf(q[i], to_f32<T>(static_cast<const T*>(p.k_pool)[base[j] + lane + 32 * i]), s[j]);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float f = warp_sum(s[j]) * p.form.scale;
      if (p.form.softcap > 0.f) f = p.form.softcap * tanhf(f / p.form.softcap);
      s[j] = t + j <= pos ? fmaf(-slope, static_cast<float>(pos - t - j), f) : -INFINITY;
    }
    const float mn = fmaxf(fmaxf(fmaxf(s[0], s[1]), fmaxf(s[2], s[3])), m);
    const float corr = m == -INFINITY ? 0.f : expf(m - mn);
    l *= corr;
#pragma unroll
    for (int i = 0; i < EPL; ++i) o[i] *= corr;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float e = s[j] == -INFINITY ? 0.f : expf(s[j] - mn);
      l += e;
#pragma unroll
      for (int i = 0; i < EPL; ++i) o[i] = fmaf(e, to_f32<T>(static_cast<const T*>(p.v_pool)[base[j] + lane + 32 * i]), o[i]);
    }
    m = mn;
  }
  if (p.form.sink && l > 0.f) l += expf(p.form.sink[h] - m);      // (an overflow leaves nothing of the keys, as it should)
  const float inv = l > 0.f ? 1.f / l : 0.f;
  T* orow = static_cast<T*>(p.o) + row * p.gate.ldo + h * D;
#pragma unroll
  for (int i = 0; i < EPL; ++i) orow[lane + 32 * i] = from_f32<T>(o[i] * inv * p.gate.factor<T>(row, h, D, lane + 32 * i));
}

template <typename T>
int launch_ragged_attn(const RaggedAttnParams& p, int D, cudaStream_t s) {
  const unsigned blocks = static_cast<unsigned>((static_cast<long long>(p.rows) * p.H + 3) / 4);
  const bool pdl = pdl_all_enabled();
#define TSB_RA(N) case N: launch_pdl(ragged_attn_kernel<T, N>, dim3(blocks), dim3(128), 0, s, pdl, p); break
  switch (D / 32) {
    TSB_RA(1); TSB_RA(2); TSB_RA(3); TSB_RA(4); TSB_RA(5); TSB_RA(6); TSB_RA(7); TSB_RA(8);
    default: return -2;
  }
#undef TSB_RA
  return static_cast<int>(cudaGetLastError());
}

}  // namespace
}  // namespace tsb

// qkv [rows, ld] = packed [q: H heads | k: Hkv | v: Hkv] of D, bf16 (dtype 1) or fp32 (0); bias fp32 [(H + 2 Hkv) D] or
// null; q_out [rows, H, D]. Pools [blocks, Hkv, bs, D]; slots[row] = block * bs + offset (-1: no slot). Rows from stage_from on also go to
// stage [*, 2 Hkv, D] at stage_rows[row - stage_from] when stage is given. D % 8 == 0, 16-byte aligned bases and rows.
TSB_EXPORT int tsb_ragged_append(const void* qkv, long long ld, const float* bias, const int* slots, void* q_out, void* k_pool, void* v_pool,
                                 void* stage, const int* stage_rows, int stage_from, int rows, int H, int Hkv, int D, int bs,
                                 int dtype, void* stream) {
  using namespace tsb;
  if (rows <= 0 || H <= 0 || Hkv <= 0 || D <= 0 || D % 8 || bs <= 0 || ld % 8 || (stage && !stage_rows)) return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const long long vecs = static_cast<long long>(rows) * (H + 2 * Hkv) * D / (dtype == 1 ? 8 : 4);
  if (vecs > 0x7fffffffLL) return -2;
  const dim3 grid(static_cast<unsigned>((vecs + 255) / 256));
  if (dtype == 1)
    launch_pdl(ragged_append_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const __nv_bfloat16*>(qkv), ld,
               bias, slots, static_cast<__nv_bfloat16*>(q_out), static_cast<__nv_bfloat16*>(k_pool), static_cast<__nv_bfloat16*>(v_pool),
               static_cast<__nv_bfloat16*>(stage), stage_rows, stage_from, rows, H, Hkv, D, bs);
  else if (dtype == 0)
    launch_pdl(ragged_append_kernel<float>, grid, dim3(256), 0, s, pdl_all_enabled(), static_cast<const float*>(qkv), ld, bias, slots,
               static_cast<float*>(q_out), static_cast<float*>(k_pool), static_cast<float*>(v_pool), static_cast<float*>(stage), stage_rows, stage_from, rows,
               H, Hkv, D, bs);
  else
    return -2;
  return static_cast<int>(cudaGetLastError());
}

// stage[dst_rows[i]] = (keys, values) of pool slot src_slots[i], i < n (bf16).
TSB_EXPORT int tsb_stage_gather(const void* k_pool, const void* v_pool, void* stage, const int* dst_rows, const int* src_slots,
                                int n, int Hkv, int D, int bs, void* stream) {
  using namespace tsb;
  if (n <= 0 || Hkv <= 0 || D <= 0 || D % 8 || bs <= 0) return -2;
  const long long vecs = static_cast<long long>(n) * 2 * Hkv * D / 8;
  if (vecs > 0x7fffffffLL) return -2;
  launch_pdl(stage_gather_kernel<__nv_bfloat16>, dim3(static_cast<unsigned>((vecs + 255) / 256)), dim3(256), 0,
             static_cast<cudaStream_t>(stream), pdl_all_enabled(), static_cast<const __nv_bfloat16*>(k_pool),
             static_cast<const __nv_bfloat16*>(v_pool), static_cast<__nv_bfloat16*>(stage), dst_rows, src_slots, n, Hkv, D, bs);
  return static_cast<int>(cudaGetLastError());
}

// o[row, h, :] = attention of row's query over the positions it sees of its sequence in the pool, the row's own key included.
// D is a multiple of 32, up to 256. ints, floats, ptrs: see attn_form.cuh.
TSB_EXPORT int tsb_ragged_attn(const void* q, long long ld_q, const void* k_pool, const void* v_pool, const int* tables,
                               int table_ld, const int* seq_of, const int* pos, void* o, int rows, int H, int Hkv, int D, int bs,
                               int nb, const long long* ints, const float* floats, const void* const* ptrs, int dtype, void* stream) {
  using namespace tsb;
  RaggedAttnParams p{q, k_pool, v_pool, tables, seq_of, pos, o, ld_q, rows, H, Hkv, bs, nb, table_ld, {}, {}, device_status_word()};
  if (rows <= 0 || H <= 0 || Hkv <= 0 || H % Hkv || D <= 0 || D % 32 || D > 256 || bs <= 0 || nb <= 0 ||
      !read_attn_form(ints, floats, ptrs, &p.form, &p.gate))
    return -2;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == 1) return launch_ragged_attn<__nv_bfloat16>(p, D, s);
  if (dtype == 0) return launch_ragged_attn<float>(p, D, s);
  return -2;
}
