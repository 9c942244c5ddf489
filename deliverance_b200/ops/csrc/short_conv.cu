// Causal convolution over time, one filter of a few taps per channel, then silu: the input stage of recurrent mixers.
//   out[t, c] = silu(b[c] + sum_j w[j, c] x[t - taps + 1 + j, c]),  zeros in front of the sequence.
// The inputs of a sequence's last positions live in its state slot as a ring [taps, C], position p at row p mod taps. Rows in front of position 0 are
// never read, so a slot needs no clearing. The ring is brought up to date by a second launch (prompts: its old rows are read by the first tokens);
// decode kernels do it in place, because the row a token writes is the only one of the ring that no token of its step reads.
#include "common.cuh"
#include "gemm_api.h"
#include "io.cuh"

namespace dlv {

constexpr int kConvRows = 8;  // rows per thread (of four channels): their inputs are loaded at once

template <typename TIO, int TAPS>
__global__ void __launch_bounds__(128) short_conv_kernel(const ConvArgs a) {
  pdl_wait();
  pdl_trigger();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4;
  if (c >= a.C) return;
  const int r0 = blockIdx.y * kConvRows, n = min(kConvRows, a.rows - r0);
  const TIO* p = static_cast<const TIO*>(a.p) + c;
  TIO* out = static_cast<TIO*>(a.out) + c;
  float w[TAPS][4], b[4] = {};
#pragma unroll
  for (int j = 0; j < TAPS; ++j) io_ld4(a.w + static_cast<size_t>(j) * a.C + c, w[j]);
  if (a.b != nullptr) io_ld4(a.b + c, b);
  auto put = [&](int r, const float (&x)[TAPS][4]) {  // x[j]: the input that filter row j multiplies
    float y[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float acc = b[e];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc += w[j][e] * x[j][e];
      y[e] = __fdividef(acc, 1.f + __expf(-acc));
    }
    io_st4(out + static_cast<size_t>(r) * a.C, y);
  };
  const int seq0 = a.row_seq[r0], first0 = a.q_start[seq0];
  if (n == kConvRows && a.row_seq[r0 + n - 1] == seq0 && r0 - (TAPS - 1) >= first0) {  // all inputs are rows of this batch
    float x[kConvRows + TAPS - 1][4];
#pragma unroll
    for (int i = 0; i < kConvRows + TAPS - 1; ++i) io_ld4(p + static_cast<long long>(r0 - (TAPS - 1) + i) * a.ld, x[i]);
#pragma unroll
    for (int i = 0; i < kConvRows; ++i) put(r0 + i, reinterpret_cast<const float (&)[TAPS][4]>(x[i]));
    return;
  }
  for (int r = r0; r < r0 + n; ++r) {
    const int s = a.row_seq[r], first = a.q_start[s], pos = a.positions[first] + r - first;
    const float* ring = a.ring + static_cast<size_t>(a.slots[s]) * TAPS * a.C + c;
    float x[TAPS][4];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int back = TAPS - 1 - j;
      if (r - back >= first) io_ld4(p + static_cast<long long>(r - back) * a.ld, x[j]);
      else if (pos - back >= 0) io_ld4(ring + static_cast<size_t>((pos - back) % TAPS) * a.C, x[j]);
      else x[j][0] = x[j][1] = x[j][2] = x[j][3] = 0.f;
    }
    put(r, x);
  }
}

// the last inputs of every sequence, one (sequence, ring row) per grid row
template <typename TIO>
__global__ void __launch_bounds__(128) short_conv_ring_kernel(const ConvArgs a) {
  pdl_wait();
  pdl_trigger();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8, s = blockIdx.y / a.taps, back = blockIdx.y % a.taps, n = a.q_len[s];
  if (c >= a.C || back >= n) return;
  const int r = a.q_start[s] + n - 1 - back, pos = a.positions[r];
  float x[8];
  io_ld8(static_cast<const TIO*>(a.p) + static_cast<long long>(r) * a.ld + c, x);
  io_st8(a.ring + (static_cast<size_t>(a.slots[s]) * a.taps + pos % a.taps) * a.C + c, x);
}

template <typename TIO>
static cudaError_t launch_short_conv_t(const ConvArgs& a, cudaStream_t st) {
  const unsigned gx = static_cast<unsigned>((a.C / 8 + 127) / 128);
  const dim3 grid(static_cast<unsigned>((a.C / 4 + 127) / 128), static_cast<unsigned>((a.rows + kConvRows - 1) / kConvRows));
  cudaError_t e = cudaErrorInvalidValue;
#define DLV_CONV(N) case N: e = launch_pdl(short_conv_kernel<TIO, N>, grid, dim3(128), 0, st, a); break
  switch (a.taps) {
    DLV_CONV(1);
    DLV_CONV(2);
    DLV_CONV(3);
    DLV_CONV(4);
    DLV_CONV(5);
    DLV_CONV(6);
    DLV_CONV(7);
    DLV_CONV(8);
  }
#undef DLV_CONV
  if (e != cudaSuccess) return e;
  return launch_pdl(short_conv_ring_kernel<TIO>, dim3(gx, static_cast<unsigned>(a.num_seqs * a.taps)), dim3(128), 0, st, a);
}

int launch_short_conv(const ConvArgs& a, bool is_f32, cudaStream_t st) {
  if (a.rows == 0 || a.num_seqs == 0) return 0;
  if (a.taps < 1 || a.taps > kMaxTaps || a.C % 8 != 0 || (a.rows + kConvRows - 1) / kConvRows > 65535 || a.num_seqs * a.taps > 65535) return 1;
  return (is_f32 ? launch_short_conv_t<float>(a, st) : launch_short_conv_t<__nv_bfloat16>(a, st)) == cudaSuccess ? 0 : 2;
}

}  // namespace dlv
