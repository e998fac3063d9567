// Warp-level tensor-core and async-copy helpers shared by the kernels of hybrid decoders: ldmatrix, the bf16 m16n8k16
// product with fp32 sums, 16-byte cp.async, and the split of an fp32 pair into two bf16 pairs whose sum carries 16 bits.
//
// Fragments of mma.m16n8k16 (g = lane / 4, t = lane % 4): A a0 = (row g, k 2t..), a1 = (row g + 8, k 2t..),
// a2 = (row g, k 2t + 8..), a3 = (row g + 8, k 2t + 8..); B b0 = (k 2t.., col g), b1 = (k 2t + 8.., col g);
// C c0, c1 = (row g, col 2t, 2t + 1), c2, c3 = (row g + 8, ...).
#pragma once

#include "common.cuh"

namespace tsb {

__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmat_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmat_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// Addresses (per lane, in bytes from the tile's start) for 16 x 16 blocks of a row-major bf16 tile with `ld` elements a row.
//   frag_a:       A from [row][k]: block at (row, k)
//   frag_a_trans: A from [k][row] (ldmat_x4_trans): block at (k, row)
//   frag_b:       two B blocks of 8 columns from [col][k] (ldmat_x4): b0, b1 of columns 0..7, then of 8..15
//   frag_b_trans: the same from [k][col] (ldmat_x4_trans)
__device__ __forceinline__ uint32_t frag_a(int lane, int row, int k, int ld) {
  return static_cast<uint32_t>((row + ((lane >> 3) & 1) * 8 + (lane & 7)) * ld + k + (lane >> 4) * 8) * 2;
}
__device__ __forceinline__ uint32_t frag_a_trans(int lane, int k, int row, int ld) {
  return static_cast<uint32_t>((k + (lane >> 4) * 8 + (lane & 7)) * ld + row + ((lane >> 3) & 1) * 8) * 2;
}
__device__ __forceinline__ uint32_t frag_b(int lane, int col, int k, int ld) {
  return static_cast<uint32_t>((col + (lane >> 4) * 8 + (lane & 7)) * ld + k + ((lane >> 3) & 1) * 8) * 2;
}
__device__ __forceinline__ uint32_t frag_b_trans(int lane, int k, int col, int ld) {
  return static_cast<uint32_t>((k + ((lane >> 3) & 1) * 8 + (lane & 7)) * ld + col + (lane >> 4) * 8) * 2;
}

// 16-byte async copy; bytes = 0 zero-fills the destination (src must still be a readable address).
__device__ __forceinline__ void cp_async_16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_8(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// (x, y) = hi + lo with both halves bf16.
__device__ __forceinline__ void split_bf16x2(float x, float y, uint32_t* hi, uint32_t* lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  *hi = *reinterpret_cast<const uint32_t*>(&h);
  *lo = pack_bf16x2(x - __low2float(h), y - __high2float(h));
}

// 16 bytes of T as floats and back.
template <typename T>
constexpr int kVec16 = 16 / sizeof(T);
template <typename T>
__device__ __forceinline__ void ld16(const T* p, float (&f)[kVec16<T>]) {
  const uint4 a = *reinterpret_cast<const uint4*>(p);
  const T* e = reinterpret_cast<const T*>(&a);
#pragma unroll
  for (int i = 0; i < kVec16<T>; ++i) f[i] = to_f32<T>(e[i]);
}
template <typename T>
__device__ __forceinline__ void st16(T* p, const float (&f)[kVec16<T>]) {
  uint4 a;
  T* e = reinterpret_cast<T*>(&a);
#pragma unroll
  for (int i = 0; i < kVec16<T>; ++i) e[i] = from_f32<T>(f[i]);
  *reinterpret_cast<uint4*>(p) = a;
}

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f32(float x) { return x / (1.f + expf(-x)); }

// One 16-byte piece of a head laid out [u: hp | v: hp | rest], rotated: pair (u_i, v_i) turns by the angle whose
// (cos, sin) is table[i]. `head` is the head's start, d0 the piece's first column; hp is a multiple of the piece.
template <typename T>
__device__ __forceinline__ void rotated_piece(const T* head, int d0, int hp, const float2* table, float (&f)[kVec16<T>]) {
  constexpr int V = kVec16<T>;
  if (d0 >= 2 * hp) {
    ld16<T>(head + d0, f);
    return;
  }
  const bool second = d0 >= hp;
  const int i0 = second ? d0 - hp : d0;
  float u[V], v[V];
  ld16<T>(head + i0, u);
  ld16<T>(head + i0 + hp, v);
#pragma unroll
  for (int i = 0; i < V; i += 2) {
    const float4 cs = *reinterpret_cast<const float4*>(table + i0 + i);
    f[i] = second ? v[i] * cs.x + u[i] * cs.y : u[i] * cs.x - v[i] * cs.y;
    f[i + 1] = second ? v[i + 1] * cs.z + u[i + 1] * cs.w : u[i + 1] * cs.z - v[i + 1] * cs.w;
  }
}

}  // namespace tsb
