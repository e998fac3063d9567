// Shared by the mixers with a short causal convolution: what a sequence's slot keeps of it.
#pragma once

#include "common.cuh"

namespace tsb {

// The last `tail` inputs of every sequence -> its slot [tail, C]. Runs after the convolution has read the old contents; one
// thread owns one channel of one sequence, and walks up, so a short portion may shift the slot in place.
template <typename T>
__global__ void __launch_bounds__(256)
conv_state_kernel(const T* x, long long ldx, int C, T* conv_state, const int* cu, const int* slots, const int* pos0, int tail) {
  pdl_trigger();
  pdl_grid_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int seq = blockIdx.y;
  if (c >= C) return;
  const int row0 = cu[seq], n = cu[seq + 1] - row0;
  const int slot = slots[seq];
  if (slot < 0 || n <= 0) return;
  const bool has_state = pos0[seq] > 0;
  T* st = conv_state + static_cast<long long>(slot) * tail * C + c;
  for (int j = 0; j < tail; ++j) {
    const int i = n - tail + j;            // token of this portion whose input belongs in place j
    T val = from_f32<T>(0.f);
    if (i >= 0) val = x[static_cast<long long>(row0 + i) * ldx + c];
    else if (has_state) val = st[static_cast<long long>(j + n) * C];
    st[static_cast<long long>(j) * C] = val;
  }
}

}  // namespace tsb
