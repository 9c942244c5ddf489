// One token of a short causal convolution (short_conv.cu) inside a decode kernel.
#pragma once
#include "gemm_api.h"
#include "io.cuh"

namespace dlv {

// activated channel c of the token at position pos, whose own input is x; ring [taps, C] of the sequence. The result is rounded to the type of the
// rows, as the prompt's convolution leaves it.
template <typename TIO>
__device__ __forceinline__ float conv_step(float x, const float* __restrict__ w, const float* __restrict__ b, const float* ring, int taps, int C, int c, int pos) {
  float acc = (b != nullptr ? b[c] : 0.f) + w[static_cast<size_t>(taps - 1) * C + c] * x;
#pragma unroll 4
  for (int back = 1; back < taps; ++back)
    if (pos - back >= 0) acc += w[static_cast<size_t>(taps - 1 - back) * C + c] * ring[static_cast<size_t>((pos - back) % taps) * C + c];
  const float y = acc / (1.f + __expf(-acc));
  if constexpr (sizeof(TIO) == 2) return bf2f(f2bf(y));
  else return y;
}

}  // namespace dlv
