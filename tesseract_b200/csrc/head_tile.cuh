// One tile of "every head (or block) has its own matrix": C[w][m][n] = sum_k x[m, k] W_w[n, k] for BM rows and 64 output
// columns, with NW matrices sharing the input. 128 threads; bf16 operands go through mma.sync, fp32 ones through FMAs.
// The fp32 sums end up in shared memory (leading dimension kLdC) and every thread may read all of them.
#pragma once

#include "warp_mma.cuh"

namespace tsb {

template <typename T, int BM, int NW>
struct HeadTile {
  static constexpr int kThreads = 128, BN = 64;
  static constexpr int kStep = sizeof(T) == 2 ? 64 : 32;                // k columns per stage
  static constexpr int kLd = kStep + 16 / static_cast<int>(sizeof(T));
  // few rows: latency decides, most of K is in flight at once; many rows and two matrices: residency decides
  static constexpr int kStages = BM == 16 ? 5 : NW == 2 ? 2 : 4;
  static constexpr int kStageElems = (BM + NW * BN) * kLd;
  static constexpr int kLdC = BN + 4;
  static constexpr int kRing = kStages * kStageElems * static_cast<int>(sizeof(T));
  static constexpr int kOut = NW * BM * kLdC * 4;
  static constexpr int kSmem = kRing > kOut ? kRing : kOut;

  // x: first row of the tile (row stride ldx, `rows` of them exist); w[i]: first matrix row of the tile (row stride ldw,
  // `cols` of them exist); 64 rows of either are less than 2^31 elements apart. K is a multiple of 16; all starts and strides are multiples of 16 bytes.
  static __device__ __forceinline__ float* run(uint8_t* smem, const T* x, long long ldx, int rows, const T* const (&w)[NW],
                                               long long ldw, int cols, int K) {
    const int ldx32 = static_cast<int>(ldx);
    return run_rows(smem, [&](int r) -> const T* { return r < rows ? x + r * ldx32 : nullptr; }, w, ldw, cols, K);
  }
  // The same with rows anywhere: x_row(r) is row r of the tile, or null for zeros.
  template <typename Row>
  static __device__ __forceinline__ float* run_rows(uint8_t* smem, Row x_row, const T* const (&w)[NW], long long ldw, int cols, int K) {
    constexpr int V = kVec16<T>, kPieces = kStep / V;
    T* ring = reinterpret_cast<T*>(smem);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int steps = (K + kStep - 1) / kStep;
    // a thread copies the same 16-byte column of every kPass-th row of the input and of the matrices
    constexpr int kPass = kThreads / kPieces, kRowsX = BM / kPass > 0 ? BM / kPass : 1, kRowsW = BN / kPass;
    const int pr = tid / kPieces, pk = (tid % kPieces) * V;
    const int ldw32 = static_cast<int>(ldw);
    const T* xr[kRowsX];
#pragma unroll
    for (int i = 0; i < kRowsX; ++i) xr[i] = BM >= kPass || pr < BM ? x_row(pr + i * kPass) : nullptr;
    auto issue = [&](int s) {
      T* st = ring + (s % kStages) * kStageElems + pr * kLd + pk;
      const int k = s * kStep + pk;
      const bool in_k = k < K;
#pragma unroll
      for (int i = 0; i < kRowsX; ++i) {
        if (BM < kPass && pr >= BM) break;
        const bool ok = in_k && xr[i] != nullptr;
        cp_async_16(smem_u32(st + i * kPass * kLd), ok ? xr[i] + k : w[0], ok ? 16 : 0);
      }
#pragma unroll
      for (int i = 0; i < NW; ++i)
#pragma unroll
        for (int j = 0; j < kRowsW; ++j) {
          const int n = pr + j * kPass;
          const bool ok = in_k && n < cols;
          cp_async_16(smem_u32(st + (BM + i * BN + j * kPass) * kLd), ok ? w[i] + n * ldw32 + k : w[i], ok ? 16 : 0);
        }
    };
    // bf16: a warp owns 32 rows x 32 columns (BM = 64) or 16 x 16 (BM = 16); fp32: 8 x 16 threads, rows and columns interleaved
    constexpr int kMB = BM == 64 ? 2 : 1, kNB = BM == 64 ? 4 : 2, kNT = kMB * kNB;      // blocks of 16 rows, of 8 columns
    constexpr int kRowsT = BM / 8;
    float acc[NW][sizeof(T) == 2 ? kNT : kRowsT][4];
#pragma unroll
    for (int i = 0; i < NW; ++i)
#pragma unroll
      for (int j = 0; j < (sizeof(T) == 2 ? kNT : kRowsT); ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
    const int row0 = BM == 64 ? (warp & 1) * 32 : 0, col0 = BM == 64 ? (warp >> 1) * 32 : warp * 16;
    const int tm = tid >> 4, tn = tid & 15;
#pragma unroll
    for (int s = 0; s < kStages - 1; ++s) {
      if (s < steps) issue(s);
      cp_commit();
    }
    for (int s = 0; s < steps; ++s) {
      if constexpr (kStages > 2) {
        cp_wait<kStages - 2>();
        __syncthreads();
        if (s + kStages - 1 < steps) issue(s + kStages - 1);
        cp_commit();
      } else {                            // (with two stages the buffer to fill is the one just read)
        __syncthreads();
        if (s + 1 < steps) issue(s + 1);
        cp_commit();
        cp_wait<1>();
        __syncthreads();
      }
      const T* sx = ring + (s % kStages) * kStageElems;
      if constexpr (sizeof(T) == 2) {
        const uint32_t ax = smem_u32(sx);
#pragma unroll
        for (int kk = 0; kk < kStep / 16; ++kk) {
          uint32_t a[kMB][4];
#pragma unroll
          for (int m = 0; m < kMB; ++m) ldmat_x4(a[m], ax + frag_a(lane, row0 + m * 16, kk * 16, kLd));
#pragma unroll
          for (int i = 0; i < NW; ++i) {
            const uint32_t bx = smem_u32(sx + (BM + i * BN) * kLd);
#pragma unroll
            for (int j = 0; j < kNB; j += 2) {
              uint32_t b[4];
              ldmat_x4(b, bx + frag_b(lane, col0 + j * 8, kk * 16, kLd));
#pragma unroll
              for (int m = 0; m < kMB; ++m) {
                mma_bf16(acc[i][m * kNB + j], a[m], b[0], b[1]);
                mma_bf16(acc[i][m * kNB + j + 1], a[m], b[2], b[3]);
              }
            }
          }
        }
      } else {
#pragma unroll 4
        for (int k = 0; k < kStep; ++k) {
          float xv[kRowsT];
#pragma unroll
          for (int r = 0; r < kRowsT; ++r) xv[r] = to_f32<T>(sx[(tm + 8 * r) * kLd + k]);
#pragma unroll
          for (int i = 0; i < NW; ++i)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
              const float wv = to_f32<T>(sx[(BM + i * BN + tn + 16 * c) * kLd + k]);
#pragma unroll
              for (int r = 0; r < kRowsT; ++r) acc[i][r][c] = fmaf(xv[r], wv, acc[i][r][c]);
            }
        }
      }
    }
    cp_wait<0>();
    __syncthreads();
    float* out = reinterpret_cast<float*>(smem);
#pragma unroll
    for (int i = 0; i < NW; ++i) {
      float* o = out + i * BM * kLdC;
      if constexpr (sizeof(T) == 2) {
        const int g = lane >> 2, t = lane & 3;
#pragma unroll
        for (int j = 0; j < kNT; ++j) {
          float* c = o + (row0 + j / kNB * 16 + g) * kLdC + col0 + j % kNB * 8 + 2 * t;
          *reinterpret_cast<float2*>(c) = make_float2(acc[i][j][0], acc[i][j][1]);
          *reinterpret_cast<float2*>(c + 8 * kLdC) = make_float2(acc[i][j][2], acc[i][j][3]);
        }
      } else {
#pragma unroll
        for (int r = 0; r < kRowsT; ++r)
#pragma unroll
          for (int c = 0; c < 4; ++c) o[(tm + 8 * r) * kLdC + tn + 16 * c] = acc[i][r][c];
      }
    }
    __syncthreads();
    return out;
  }
};

}  // namespace tsb
