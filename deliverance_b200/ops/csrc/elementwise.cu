// Memory-bound fused elementwise / normalisation kernels (bf16 activations, fp32 math).
//   rmsnorm, residual-add + rmsnorm (Gemma "1 + w" offset, Granite residual multiplier), LayerNorm,
//   act(gate) * up on a concatenated projection, embedding gather (+ scale, + positional / token-type tables),
//   per-head q/k RMSNorm + HF half-rotation RoPE + paged KV-cache write in one pass.
// Reference math: core/.../generator/RmsNorm.java:107-121, TransformerBlock.java:265-276, LayerNorm.java:20-151,
// CausalSelfAttention.java:315-372,429-446, Qwen3CausalSelfAttention.java:74-92, EmbedInput.java:26-44,
// native/src/main/c/simd/vector_simd.c:185-213 (the fused activation; here the product stays bf16, no int8 requant).
#include "gemm_api.h"
#include "io.cuh"

namespace dlv {

// ------------------------------------------------------------------------------------------------ RMSNorm
// One CTA per row. x, residual, y: bf16 [T, H]; H % 8 == 0. When residual != nullptr: residual += x * res_mult first
// (written back) and the norm runs on the updated residual.
__global__ void __launch_bounds__(256) rmsnorm_kernel(const __nv_bfloat16* __restrict__ x, __nv_bfloat16* residual,
                                                      const __nv_bfloat16* __restrict__ w, __nv_bfloat16* __restrict__ y,
                                                      int H, float eps, float offset, float res_mult) {
  pdl_wait();     // no-op unless launched with programmatic stream serialization: the kernel in front has completed
  pdl_trigger();  // the next kernel may start its prologue (and a GEMM its weight prefetch) under this kernel's tail
  extern __shared__ float row[];  // H floats
  __shared__ float red[32];
  const size_t base = static_cast<size_t>(blockIdx.x) * H;
  float ss = 0.f;
  for (int i = threadIdx.x * 8; i < H; i += blockDim.x * 8) {
    uint4 xv = *reinterpret_cast<const uint4*>(x + base + i);
    const uint32_t* xu = reinterpret_cast<const uint32_t*>(&xv);
    float v[8];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float2 f = unpack_bf162(xu[j]);
      v[2 * j] = f.x;
      v[2 * j + 1] = f.y;
    }
    if (residual != nullptr) {
      uint4 rv = *reinterpret_cast<const uint4*>(residual + base + i);
      const uint32_t* ru = reinterpret_cast<const uint32_t*>(&rv);
      uint4 ov;
      uint32_t* ou = reinterpret_cast<uint32_t*>(&ov);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float2 f = unpack_bf162(ru[j]);
        float a = f.x + v[2 * j] * res_mult, b = f.y + v[2 * j + 1] * res_mult;
        ou[j] = pack_bf162(a, b);
        float2 back = unpack_bf162(ou[j]);  // the norm sees the stored (rounded) residual
        v[2 * j] = back.x;
        v[2 * j + 1] = back.y;
      }
      *reinterpret_cast<uint4*>(residual + base + i) = ov;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      row[i + j] = v[j];
      ss += v[j] * v[j];
    }
  }
  ss = block_sum(ss, red);
  const float inv = rsqrtf(ss / H + eps);
  for (int i = threadIdx.x * 8; i < H; i += blockDim.x * 8) {
    uint4 wv = *reinterpret_cast<const uint4*>(w + i);
    const uint32_t* wu = reinterpret_cast<const uint32_t*>(&wv);
    uint4 ov;
    uint32_t* ou = reinterpret_cast<uint32_t*>(&ov);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float2 f = unpack_bf162(wu[j]);
      ou[j] = pack_bf162(row[i + 2 * j] * inv * (f.x + offset), row[i + 2 * j + 1] * inv * (f.y + offset));
    }
    *reinterpret_cast<uint4*>(y + base + i) = ov;
  }
}

// ------------------------------------------------------------------------------------------------ LayerNorm
__global__ void __launch_bounds__(256) layernorm_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ w,
                                                        const __nv_bfloat16* __restrict__ b, __nv_bfloat16* __restrict__ y, int H,
                                                        float eps) {
  pdl_wait();     // no-op unless launched with programmatic stream serialization: the kernel in front has completed
  pdl_trigger();  // the next kernel may start its prologue (and a GEMM its weight prefetch) under this kernel's tail
  extern __shared__ float row[];
  __shared__ float red[32];
  const size_t base = static_cast<size_t>(blockIdx.x) * H;
  float s = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float v = bf2f(x[base + i]);
    row[i] = v;
    s += v;
  }
  const float mean = block_sum(s, red) / H;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float d = row[i] - mean;
    ss += d * d;
  }
  const float inv = rsqrtf(block_sum(ss, red) / H + eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float v = (row[i] - mean) * inv * bf2f(w[i]) + (b ? bf2f(b[i]) : 0.f);
    y[base + i] = f2bf(v);
  }
}

// ------------------------------------------------------------------------------------------------ act(gate) * up
__device__ __forceinline__ float act_apply(float g, int act) {
  switch (act) {
    case 0: return g / (1.f + __expf(-g));                                                     // silu
    case 1: return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));  // gelu tanh
    case 2: return 0.5f * g * (1.f + erff(g * 0.7071067811865475f));                            // gelu erf
    case 3: return fmaxf(g, 0.f);
    case 5: return fmaxf(g, 0.f) * fmaxf(g, 0.f);  // squared relu
    default: return tanhf(g);
  }
}

// in: [T, 2*I] (gate | up), out: [T, I]; I % 8 == 0
__global__ void __launch_bounds__(256) act_mul_kernel(const __nv_bfloat16* __restrict__ in, __nv_bfloat16* __restrict__ out, int I,
                                                      int act, long long total_vec) {
  pdl_wait();     // no-op unless launched with programmatic stream serialization: the kernel in front has completed
  pdl_trigger();  // the next kernel may start its prologue (and a GEMM its weight prefetch) under this kernel's tail
  const long long idx = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (idx >= total_vec) return;
  const int per_row = I / 8;
  const long long t = idx / per_row;
  const int c = static_cast<int>(idx % per_row) * 8;
  const __nv_bfloat16* g = in + t * 2 * I + c;
  uint4 gv = *reinterpret_cast<const uint4*>(g);
  uint4 uv = *reinterpret_cast<const uint4*>(g + I);
  const uint32_t* gu = reinterpret_cast<const uint32_t*>(&gv);
  const uint32_t* uu = reinterpret_cast<const uint32_t*>(&uv);
  uint4 ov;
  uint32_t* ou = reinterpret_cast<uint32_t*>(&ov);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    float2 a = unpack_bf162(gu[j]), b = unpack_bf162(uu[j]);
    ou[j] = pack_bf162(act_apply(a.x, act) * b.x, act_apply(a.y, act) * b.y);
  }
  *reinterpret_cast<uint4*>(out + t * I + c) = ov;
}

// unary activation (MLPs without an up projection): a thread takes eight elements
template <typename TIO>
__global__ void __launch_bounds__(256) act_kernel(const TIO* __restrict__ in, TIO* __restrict__ out, int act, long long n) {
  pdl_wait();     // no-op unless launched with programmatic stream serialization: the kernel in front has completed
  pdl_trigger();  // the next kernel may start its prologue (and a GEMM its weight prefetch) under this kernel's tail
  const long long i = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) * 8;
  if (i + 8 <= n) {
    float v[8];
    io_ld8(in + i, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = act_apply(v[e], act);
    io_st8(out + i, v);
  } else {
    for (long long k = i; k < n; ++k) io_st(out + k, act_apply(io_ld(in + k), act));
  }
}

// ------------------------------------------------------------------------------------------------ embedding
// out[t] = table[ids[t]] * scale (+ pos_table[pos[t]]) (+ type_table[types[t]]); H % 8 == 0
__global__ void __launch_bounds__(128) embedding_kernel(const __nv_bfloat16* __restrict__ table, const int* __restrict__ ids,
                                                        const __nv_bfloat16* __restrict__ pos_table, const int* __restrict__ pos,
                                                        const __nv_bfloat16* __restrict__ type_table, const int* __restrict__ types,
                                                        __nv_bfloat16* __restrict__ out, int H, int vocab, float scale) {
  pdl_wait();     // no-op unless launched with programmatic stream serialization: the kernel in front has completed
  pdl_trigger();  // the next kernel may start its prologue (and a GEMM its weight prefetch) under this kernel's tail
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) id = 0;  // host validates ids; never read out of the table
  const __nv_bfloat16* src = table + static_cast<size_t>(id) * H;
  const __nv_bfloat16* ps = pos_table ? pos_table + static_cast<size_t>(pos[t]) * H : nullptr;
  const __nv_bfloat16* ts = type_table ? type_table + static_cast<size_t>(types ? types[t] : 0) * H : nullptr;
  for (int i = threadIdx.x * 8; i < H; i += blockDim.x * 8) {
    uint4 v = *reinterpret_cast<const uint4*>(src + i);
    const uint32_t* vu = reinterpret_cast<const uint32_t*>(&v);
    float f[8];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float2 a = unpack_bf162(vu[j]);
      f[2 * j] = a.x * scale;
      f[2 * j + 1] = a.y * scale;
    }
    if (ps) {
      uint4 pv = *reinterpret_cast<const uint4*>(ps + i);
      const uint32_t* pu = reinterpret_cast<const uint32_t*>(&pv);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float2 a = unpack_bf162(pu[j]);
        f[2 * j] += a.x;
        f[2 * j + 1] += a.y;
      }
    }
    if (ts) {
      uint4 pv = *reinterpret_cast<const uint4*>(ts + i);
      const uint32_t* pu = reinterpret_cast<const uint32_t*>(&pv);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float2 a = unpack_bf162(pu[j]);
        f[2 * j] += a.x;
        f[2 * j + 1] += a.y;
      }
    }
    uint4 o;
    uint32_t* ou = reinterpret_cast<uint32_t*>(&o);
#pragma unroll
    for (int j = 0; j < 4; ++j) ou[j] = pack_bf162(f[2 * j], f[2 * j + 1]);
    *reinterpret_cast<uint4*>(out + static_cast<size_t>(t) * H + i) = o;
  }
}

// ------------------------------------------------------------------------------------------------ q/k norm + RoPE + KV write
// qkv: [T, (H + 2 KV) * D] bf16. One warp per (token, head). q heads are normalised/rotated in place; k heads are
// normalised/rotated and written to the paged cache; v heads are copied to the cache.
// cache layout: [num_blocks, KV, block_size, D]; slot = block * block_size + offset; slot < 0 skips the cache write.
template <int D>
__global__ void __launch_bounds__(256) rope_kv_kernel(__nv_bfloat16* __restrict__ qkv, const int* __restrict__ positions,
                                                      const long long* __restrict__ slots, const __nv_bfloat16* __restrict__ q_norm_w,
                                                      const __nv_bfloat16* __restrict__ k_norm_w, const float* __restrict__ cos_t,
                                                      const float* __restrict__ sin_t, __nv_bfloat16* __restrict__ k_cache,
                                                      __nv_bfloat16* __restrict__ v_cache, int T, int H, int KV, int block_size,
                                                      int rot_half, float eps, float norm_offset, int max_pos) {
  pdl_wait();     // no-op unless launched with programmatic stream serialization: the kernel in front has completed
  pdl_trigger();  // the next kernel may start its prologue (and a GEMM its weight prefetch) under this kernel's tail
  const int warp_global = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  const int heads = H + 2 * KV;
  if (warp_global >= T * heads) return;
  const int t = warp_global / heads, h = warp_global % heads;
  __nv_bfloat16* src = qkv + static_cast<size_t>(t) * heads * D + static_cast<size_t>(h) * D;
  constexpr int HALF = D / 2;
  constexpr int PER = HALF / 32 > 0 ? HALF / 32 : 1;  // pairs per lane (D >= 64)
  const bool is_q = h < H, is_k = !is_q && h < H + KV;
  const long long slot = slots ? slots[t] : -1;
  const int kvh = is_q ? 0 : (is_k ? h - H : h - H - KV);
  __nv_bfloat16* dst = nullptr;
  if (!is_q && slot >= 0) {
    const long long blk = slot / block_size, off = slot % block_size;
    __nv_bfloat16* cache = is_k ? k_cache : v_cache;
    dst = cache + ((blk * KV + kvh) * block_size + off) * D;
  }
  float a[PER], b[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int d = lane + 32 * i;
    a[i] = d < HALF ? bf2f(src[d]) : 0.f;
    b[i] = d < HALF ? bf2f(src[d + HALF]) : 0.f;
  }
  if (!is_q && !is_k) {  // v: plain copy
    if (dst) {
#pragma unroll
      for (int i = 0; i < PER; ++i) {
        const int d = lane + 32 * i;
        if (d < HALF) {
          dst[d] = f2bf(a[i]);
          dst[d + HALF] = f2bf(b[i]);
        }
      }
    }
    return;
  }
  const __nv_bfloat16* nw = is_q ? q_norm_w : k_norm_w;
  if (nw != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) ss += a[i] * a[i] + b[i] * b[i];
    ss = warp_sum(ss);
    const float inv = rsqrtf(ss / D + eps);
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int d = lane + 32 * i;
      if (d < HALF) {
        // round through bf16 like a separate norm kernel would
        a[i] = bf2f(f2bf(a[i] * inv * (bf2f(nw[d]) + norm_offset)));
        b[i] = bf2f(f2bf(b[i] * inv * (bf2f(nw[d + HALF]) + norm_offset)));
      }
    }
  }
  if (cos_t != nullptr) {
    int pos = positions[t];
    pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int d = lane + 32 * i;
      if (d < rot_half) {
        const float c = cos_t[static_cast<size_t>(pos) * rot_half + d], s = sin_t[static_cast<size_t>(pos) * rot_half + d];
        const float x0 = a[i], x1 = b[i];
        a[i] = x0 * c - x1 * s;
        b[i] = x1 * c + x0 * s;
      }
    }
  }
  __nv_bfloat16* out = is_q ? src : dst;
  if (out) {
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int d = lane + 32 * i;
      if (d < HALF) {
        out[d] = f2bf(a[i]);
        out[d + HALF] = f2bf(b[i]);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ fp32 residual stream
// Models that keep the residual stream in fp32: embedding with a hashed-bigram table, residual add + one or two LayerNorms of the same
// row, gated activation with row pitches. TIO: bf16 or fp32 activations.

// out[t] = table[ids[t]] * scale + bigram[row]; row = (prev * mul_prev + id * mul_cur) mod buckets, or `buckets` (the extra last row) when the
// token has no predecessor (prev < 0); out2 (optional, pitch ld2): the same row in the table's type
template <typename TIO>
__global__ void __launch_bounds__(128) bigram_embedding_kernel(const TIO* __restrict__ table, const TIO* __restrict__ bigram, const int* __restrict__ ids,
                                                               const int* __restrict__ prev, float* __restrict__ out, int W, int vocab, int buckets,
                                                               long long mul_prev, long long mul_cur, float scale, TIO* __restrict__ out2,
                                                               long long ld2) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) id = 0;  // host validates ids; never read out of the table
  const TIO* src = table + static_cast<size_t>(id) * W;
  const TIO* bg = nullptr;
  if (bigram != nullptr) {
    const long long pv = prev[t];
    long long row = pv < 0 ? buckets : (pv * mul_prev + static_cast<long long>(id) * mul_cur) % buckets;
    if (row < 0) row += buckets;
    bg = bigram + row * W;
  }
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    const float v = io_ld(src + i) * scale + (bg != nullptr ? io_ld(bg + i) : 0.f);
    out[static_cast<size_t>(t) * W + i] = v;
    if (out2 != nullptr) io_st(out2 + t * ld2 + i, v);
  }
}

// residual += delta (when given; written back), then y1 = LayerNorm(residual; w1, b1) and, when w2 is given, y2 = LayerNorm(residual; w2, b2)
// from the same statistics. Columns W .. y_pitch of the outputs are zeroed. One CTA per row.
template <typename TIO>
__global__ void __launch_bounds__(256) add_layernorm_kernel(float* __restrict__ residual, const float* __restrict__ delta, const float* __restrict__ w1,
                                                            const float* __restrict__ b1, TIO* __restrict__ y1, const float* __restrict__ w2,
                                                            const float* __restrict__ b2, TIO* __restrict__ y2, int W, int y_pitch, float eps) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  const size_t base = static_cast<size_t>(blockIdx.x) * W, yb = static_cast<size_t>(blockIdx.x) * y_pitch;
  const bool vec = (W & 3) == 0;  // rows start on 16 bytes then
  float s = 0.f;
  if (vec) {
    for (int i = threadIdx.x * 4; i < W; i += blockDim.x * 4) {
      float4 v = *reinterpret_cast<const float4*>(residual + base + i);
      if (delta != nullptr) {
        const float4 d = *reinterpret_cast<const float4*>(delta + base + i);
        v.x += d.x; v.y += d.y; v.z += d.z; v.w += d.w;
        *reinterpret_cast<float4*>(residual + base + i) = v;
      }
      *reinterpret_cast<float4*>(row + i) = v;
      s += (v.x + v.y) + (v.z + v.w);
    }
  } else {
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
      float v = residual[base + i];
      if (delta != nullptr) {
        v += delta[base + i];
        residual[base + i] = v;
      }
      row[i] = v;
      s += v;
    }
  }
  const float mean = block_sum(s, red) / W;  // (its barriers also publish the row)
  float ss = 0.f;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    const float d = row[i] - mean;
    ss += d * d;
  }
  const float inv = rsqrtf(block_sum(ss, red) / W + eps);
  auto norm4 = [&](int i, const float* w, const float* b, TIO* y) {
    const float4 v = *reinterpret_cast<const float4*>(row + i), wv = *reinterpret_cast<const float4*>(w + i), bv = *reinterpret_cast<const float4*>(b + i);
    const float o0 = (v.x - mean) * inv * wv.x + bv.x, o1 = (v.y - mean) * inv * wv.y + bv.y, o2 = (v.z - mean) * inv * wv.z + bv.z,
                o3 = (v.w - mean) * inv * wv.w + bv.w;
    if constexpr (sizeof(TIO) == 2) *reinterpret_cast<uint2*>(y + yb + i) = make_uint2(pack_bf162(o0, o1), pack_bf162(o2, o3));
    else *reinterpret_cast<float4*>(y + yb + i) = make_float4(o0, o1, o2, o3);
  };
  if (vec && (y_pitch & 3) == 0) {
    for (int i = threadIdx.x * 4; i < W; i += blockDim.x * 4) {
      if (y1 != nullptr) norm4(i, w1, b1, y1);
      if (y2 != nullptr) norm4(i, w2, b2, y2);
    }
    for (int i = W + threadIdx.x; i < y_pitch; i += blockDim.x) {
      if (y1 != nullptr) io_st(y1 + yb + i, 0.f);
      if (y2 != nullptr) io_st(y2 + yb + i, 0.f);
    }
    return;
  }
  for (int i = threadIdx.x; i < y_pitch; i += blockDim.x) {
    const float n = i < W ? (row[i] - mean) * inv : 0.f;
    if (y1 != nullptr) io_st(y1 + yb + i, i < W ? n * w1[i] + b1[i] : 0.f);
    if (y2 != nullptr) io_st(y2 + yb + i, i < W ? n * w2[i] + b2[i] : 0.f);
  }
}

// out[t, c] = act(in[t, c]) * in[t, I + c]
template <typename TIO>
__global__ void __launch_bounds__(256) gated_act_kernel(const TIO* __restrict__ in, long long ld_in, TIO* __restrict__ out, long long ld_out, int I, int act,
                                                        long long total) {
  pdl_wait();
  pdl_trigger();
  const long long idx = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (idx >= total) return;
  const int per_row = I / 8;
  const long long t = idx / per_row;
  const int c = static_cast<int>(idx % per_row) * 8;
  const TIO* g = in + t * ld_in + c;
  TIO* o = out + t * ld_out + c;
  if constexpr (sizeof(TIO) == 2) {
    const uint4 gv = *reinterpret_cast<const uint4*>(g), uv = *reinterpret_cast<const uint4*>(g + I);
    const uint32_t* gu = reinterpret_cast<const uint32_t*>(&gv);
    const uint32_t* uu = reinterpret_cast<const uint32_t*>(&uv);
    uint32_t ou[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 a = unpack_bf162(gu[j]), b = unpack_bf162(uu[j]);
      ou[j] = pack_bf162(act_apply(a.x, act) * b.x, act_apply(a.y, act) * b.y);
    }
    *reinterpret_cast<uint4*>(o) = make_uint4(ou[0], ou[1], ou[2], ou[3]);
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = act_apply(g[j], act) * g[I + j];
  }
}

// ------------------------------------------------------------------------------------------------ sandwich norm
// Norm behind a sublayer, scaled residual add and norm in front of the next sublayer in one pass over a row of the fp32 residual stream:
//   residual += mult * LayerNorm(sub; w_sub)   (skipped without sub)
//   y = LayerNorm(residual; w_next)            (the residual itself without w_next), columns W .. y_width zeroed
// RMS: RMS norms instead of LayerNorms. A weight may be one number for all columns (sub_one, next_one).
// sub is one row [T, ld_sub] or, with pos, the weighted sum of k rows of an expert-ordered buffer: sum_j wts[t, j] * sub[pos[t, j]], formed
// in fp32 in slot order. One CTA per row; the row lives in registers (NV groups of four columns per thread), both variances are means of
// squared deviations.
struct SandwichArgs {
  float* residual;
  const void* sub;
  long long ld_sub;
  const int* pos;
  const float* wts;
  int k;
  const float* w_sub;
  float mult;
  const float* w_next;
  void* y;
  long long ld_y;
  int W, y_width;
  float eps;
  int vec;  // rows, pitches and pointers allow four-column accesses
  int sub_one, next_one;
};

template <typename TSUB, typename TIO, int NV, int NT, bool RMS>
__global__ void __launch_bounds__(NT) sandwich_norm_kernel(const SandwichArgs a) {
  __shared__ float red[32];
  const int t = blockIdx.x, W = a.W;
  float* res = a.residual + static_cast<size_t>(t) * W;
  TIO* y = static_cast<TIO*>(a.y) + t * a.ld_y;
  const TSUB* sub = static_cast<const TSUB*>(a.sub);
  float v[NV][4];
  auto col = [&](int n) { return (n * NT + static_cast<int>(threadIdx.x)) * 4; };
  pdl_wait();
  pdl_trigger();
  auto load = [&](auto* p, int c, float* o) {
    if (a.vec) {
      if (c < W) io_ld4(p + c, o);
      else o[0] = o[1] = o[2] = o[3] = 0.f;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] = c + e < W ? io_ld(p + c + e) : 0.f;
    }
  };
  auto deviation = [&](float mean) {  // sum of squared deviations of the real columns
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float d = v[n][e] - mean;
        ss += col(n) + e < W ? d * d : 0.f;
      }
    return ss;
  };
  if (sub != nullptr) {
    float r[NV][4];
#pragma unroll
    for (int n = 0; n < NV; ++n) load(res, col(n), r[n]);
    if (a.pos == nullptr) {
#pragma unroll
      for (int n = 0; n < NV; ++n) load(sub + t * a.ld_sub, col(n), v[n]);
    } else {
#pragma unroll
      for (int n = 0; n < NV; ++n) v[n][0] = v[n][1] = v[n][2] = v[n][3] = 0.f;
      for (int j = 0; j < a.k; ++j) {
        const float wt = a.wts[static_cast<size_t>(t) * a.k + j];
        const TSUB* row = sub + a.pos[static_cast<size_t>(t) * a.k + j] * a.ld_sub;
#pragma unroll
        for (int n = 0; n < NV; ++n) {
          float o[4];
          load(row, col(n), o);
#pragma unroll
          for (int e = 0; e < 4; ++e) v[n][e] += wt * o[e];
        }
      }
    }
    float mean = 0.f;
    if constexpr (!RMS) {
      float s = 0.f;
#pragma unroll
      for (int n = 0; n < NV; ++n) s += (v[n][0] + v[n][1]) + (v[n][2] + v[n][3]);
      mean = block_sum(s, red) / W;
    }
    const float inv = rsqrtf(block_sum(deviation(mean), red) / W + a.eps) * a.mult;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      float w[4];
      if (a.sub_one) w[0] = w[1] = w[2] = w[3] = a.w_sub[0];
      else load(a.w_sub, col(n), w);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[n][e] = r[n][e] + (v[n][e] - mean) * inv * w[e];
      if (a.vec) {
        if (col(n) < W) io_st4(res + col(n), v[n]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (col(n) + e < W) res[col(n) + e] = v[n][e];
          else v[n][e] = 0.f;
        }
      }
      if (a.vec && col(n) >= W) v[n][0] = v[n][1] = v[n][2] = v[n][3] = 0.f;
    }
  } else {
#pragma unroll
    for (int n = 0; n < NV; ++n) load(res, col(n), v[n]);
  }
  float mean = 0.f, inv = 1.f;
  if (a.w_next != nullptr) {
    if constexpr (!RMS) {
      float s = 0.f;
#pragma unroll
      for (int n = 0; n < NV; ++n) s += (v[n][0] + v[n][1]) + (v[n][2] + v[n][3]);
      mean = block_sum(s, red) / W;
    }
    inv = rsqrtf(block_sum(deviation(mean), red) / W + a.eps);
  }
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    float o[4] = {v[n][0], v[n][1], v[n][2], v[n][3]};
    if (a.w_next != nullptr) {
      float w[4];
      if (a.next_one) w[0] = w[1] = w[2] = w[3] = a.w_next[0];
      else load(a.w_next, col(n), w);
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] = col(n) + e < W ? (v[n][e] - mean) * inv * w[e] : 0.f;
    }
    if (a.vec) {
      if (col(n) < a.y_width) io_st4(y + col(n), o);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (col(n) + e < a.y_width) io_st(y + col(n) + e, o[e]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ pair rotation + KV write
// qkv rows [q (H * dk) | k (KV * dk) | v (KV * dv)], dk and dv multiples of 8. The first 2 * half columns of every query and key head are
// rotated in neighbouring pairs (2 i, 2 i + 1); queries in place, keys on their way into the cache, values are copied. A thread takes
// eight columns; query columns that are not rotated are not touched.
template <typename TIO>
__global__ void __launch_bounds__(256) rope_pairs_kv_kernel(TIO* __restrict__ qkv, long long ld, const int* __restrict__ positions,
                                                            const long long* __restrict__ slots, const float* __restrict__ cos_t,
                                                            const float* __restrict__ sin_t, TIO* __restrict__ k_cache, TIO* __restrict__ v_cache, int T, int H,
                                                            int KV, int dk, int dv, int page, int half, int max_pos) {
  pdl_wait();
  pdl_trigger();
  const int rot = (2 * half + 7) / 8, ck = dk / 8, cv = dv / 8;
  const int nq = H * rot, nk = KV * ck, per = nq + nk + KV * cv;
  const long long idx = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (idx >= static_cast<long long>(T) * per) return;
  const int t = static_cast<int>(idx / per);
  int c = static_cast<int>(idx % per);
  const TIO* src;
  TIO* dst;
  int d0 = 0;  // first column inside the head (rotated parts only)
  bool rotate = false;
  if (c < nq) {
    d0 = (c % rot) * 8;
    dst = qkv + t * ld + static_cast<long long>(c / rot) * dk + d0;
    src = dst;
    rotate = true;
  } else {
    const long long slot = slots[t];
    if (slot < 0) return;
    const long long blk = slot / page, off = slot % page;
    c -= nq;
    if (c < nk) {
      d0 = (c % ck) * 8;
      src = qkv + t * ld + static_cast<long long>(H) * dk + static_cast<long long>(c) * 8;
      dst = k_cache + ((blk * KV + c / ck) * page + off) * dk + d0;
      rotate = d0 < 2 * half;
    } else {
      c -= nk;
      src = qkv + t * ld + static_cast<long long>(H + KV) * dk + static_cast<long long>(c) * 8;
      dst = v_cache + ((blk * KV + c / cv) * page + off) * dv + (c % cv) * 8;
    }
  }
  float x[8];
  io_ld4(src, x);
  io_ld4(src + 4, x + 4);
  if (rotate) {
    int pos = positions[t];
    pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = d0 / 2 + e;
      if (i < half) {
        const float cs = cos_t[static_cast<size_t>(pos) * half + i], sn = sin_t[static_cast<size_t>(pos) * half + i];
        const float u = x[2 * e], w = x[2 * e + 1];
        x[2 * e] = u * cs - w * sn;
        x[2 * e + 1] = w * cs + u * sn;
      }
    }
  }
  io_st4(dst, x);
  io_st4(dst + 4, x + 4);
}

// ------------------------------------------------------------------------------------------------ per-head norm, half rotation, KV write
// Projection rows p: queries at column 0 (H heads of dk columns), keys at off_k (KV heads of dk), values at off_v (KV heads of dv; off_v = off_k
// when the values are the projected keys). Queries and keys: optional RMS norm over the head (dim real columns), then the pairs
// (i, i + half), i < half, are rotated; queries in place, keys into the cache. Values go to the cache as projected or, with v_first,
// blended with another row of the same token: (1 - lam) v + lam v_first.
// LPH lanes of a warp own one (row, head), eight columns per lane and step. The partners of eight rotated columns lie in another lane's
// registers when `half` is a multiple of eight and the head is one step wide (LANES); otherwise the head passes through shared memory.
template <typename TIO, int LPH, bool LANES>
__global__ void __launch_bounds__(256) rope_heads_kv_kernel(const RopeHeadsArgs a) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) float hsm[];
  const bool tied = a.off_v == a.off_k;
  const int heads = a.H + a.KV + (tied ? 0 : a.KV);
  const int sub = threadIdx.x % LPH, grp = threadIdx.x / LPH;
  const unsigned idx = blockIdx.x * (256u / LPH) + grp;
  const bool active = idx < static_cast<unsigned>(a.T) * heads;  // (all lanes reach the shuffles and warp barriers below)
  const int t = active ? static_cast<int>(idx / heads) : 0, h = active ? static_cast<int>(idx % heads) : 0;
  const bool is_q = h < a.H, is_v = h >= a.H + a.KV;
  const int kvh = is_q ? 0 : (is_v ? h - a.H - a.KV : h - a.H);
  TIO* row = static_cast<TIO*>(a.p) + t * a.ld;
  long long at = 0;  // row of the caches
  bool store = active;
  if (!is_q) {
    const long long slot = a.slots[t];
    store = active && slot >= 0;
    const unsigned su = static_cast<unsigned>(store ? slot : 0), page = static_cast<unsigned>(a.page);  // (the caches hold fewer than 2^32 rows)
    at = a.wide ? static_cast<long long>(su) * a.KV + kvh : (static_cast<long long>(su / page) * a.KV + kvh) * a.page + su % page;
  }
  float* s = hsm + grp * a.dk;
  const TIO* src = row + (is_q ? h * a.dk : (is_v ? a.off_v + kvh * a.dv : a.off_k + kvh * a.dk));
  TIO* vdst = static_cast<TIO*>(a.v_cache) + at * a.dv;
  const float* nw = is_v ? nullptr : (is_q ? a.q_norm : a.k_norm);
  const int width = is_v ? a.dv : a.dk;
  float ss = 0.f, x[8] = {};
  for (int c = sub * 8; c < width; c += LPH * 8) {
    io_ld8(src + c, x);
    if (is_v || (!is_q && tied)) {
      if (a.v_first != nullptr) {
        float f[8];
        io_ld8(static_cast<const TIO*>(a.v_first) + t * a.ld_first + kvh * a.dv + c, f);
        float y[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] = (1.f - a.lam) * x[e] + a.lam * f[e];
        if (store) io_st8(vdst + c, y);
      } else if (store) {
        io_st8(vdst + c, x);
      }
    }
    if (!is_v) {
      if constexpr (!LANES) {
        *reinterpret_cast<float4*>(s + c) = make_float4(x[0], x[1], x[2], x[3]);
        *reinterpret_cast<float4*>(s + c + 4) = make_float4(x[4], x[5], x[6], x[7]);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += x[e] * x[e];
    }
  }
#pragma unroll
  for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  float other[8];  // LANES: the partners of this lane's columns
  if constexpr (LANES) {
    const int hc = a.half / 8, from = sub < hc ? sub + hc : (sub < 2 * hc ? sub - hc : sub);
#pragma unroll
    for (int e = 0; e < 8; ++e) other[e] = __shfl_sync(0xffffffffu, x[e], from, LPH);
  } else {
    __syncwarp();
  }
  if (is_v || !store) return;
  const float inv = nw != nullptr ? rsqrtf(ss / a.dim + a.eps) : 1.f;
  int pos = a.positions[t];
  pos = pos < 0 ? 0 : (pos >= a.max_pos ? a.max_pos - 1 : pos);
  const float* cs = a.cos_t + static_cast<size_t>(pos) * a.half;
  const float* sn = a.sin_t + static_cast<size_t>(pos) * a.half;
  TIO* dst = is_q ? row + h * a.dk : static_cast<TIO*>(a.k_cache) + at * a.dk;
  const int end = is_q && nw == nullptr ? min(a.dk, (2 * a.half + 7) / 8 * 8) : a.dk;  // queries that nothing changes stay where they are
  if constexpr (LANES) {
    const int c = sub * 8;
    if (c >= end) return;
    float w[8];
    if (nw != nullptr) {
      io_ld8(nw + c, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] *= inv * w[e];
    }
    if (c < 2 * a.half) {
      const bool low = c < a.half;
      const int i = low ? c : c - a.half;
      if (nw != nullptr) {
        io_ld8(nw + (low ? c + a.half : i), w);
#pragma unroll
        for (int e = 0; e < 8; ++e) other[e] *= inv * w[e];
      }
      float co[8], si[8];
      io_ld8(cs + i, co);
      io_ld8(sn + i, si);
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] = low ? x[e] * co[e] - other[e] * si[e] : x[e] * co[e] + other[e] * si[e];
    }
    io_st8(dst + c, x);
    return;
  }
  for (int c = sub * 8; c < end; c += LPH * 8) {
    float y[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const int d = c + e;
      float v = s[d] * inv;
      if (nw != nullptr) v *= nw[d];
      if (d < 2 * a.half) {
        const bool low = d < a.half;
        const int i = low ? d : d - a.half, o = low ? d + a.half : i;
        float w = s[o] * inv;
        if (nw != nullptr) w *= nw[o];
        v = low ? v * cs[i] - w * sn[i] : v * cs[i] + w * sn[i];
      }
      y[e] = v;
    }
    io_st8(dst + c, y);
  }
}

template <typename TIO>
static int launch_rope_heads_t(const RopeHeadsArgs& a, cudaStream_t st) {
  const int chunks = (a.dk > a.dv ? a.dk : a.dv) / 8;
  const long long n = static_cast<long long>(a.T) * (a.H + (a.off_v == a.off_k ? 1 : 2) * a.KV);
  const bool lanes = a.half % 8 == 0 && a.dk <= 256;
  auto go = [&](auto by_lanes, auto by_memory, int lph) {
    const int per = 256 / lph;
    const dim3 grid(static_cast<unsigned>((n + per - 1) / per));
    const cudaError_t e = lanes ? launch_pdl(by_lanes, grid, dim3(256), 0, st, a)
                                : launch_pdl(by_memory, grid, dim3(256), static_cast<size_t>(per) * a.dk * sizeof(float), st, a);
    return e == cudaSuccess ? 0 : 2;
  };
  if (chunks <= 4) return go(rope_heads_kv_kernel<TIO, 4, true>, rope_heads_kv_kernel<TIO, 4, false>, 4);
  if (chunks <= 8) return go(rope_heads_kv_kernel<TIO, 8, true>, rope_heads_kv_kernel<TIO, 8, false>, 8);
  if (chunks <= 16) return go(rope_heads_kv_kernel<TIO, 16, true>, rope_heads_kv_kernel<TIO, 16, false>, 16);
  return go(rope_heads_kv_kernel<TIO, 32, true>, rope_heads_kv_kernel<TIO, 32, false>, 32);
}

// ------------------------------------------------------------------------------------------------ launchers
void launch_rmsnorm(const void* x, void* residual, const void* w, void* y, int T, int H, float eps, float offset,
                    float res_mult, cudaStream_t st) {
  if (T == 0) return;
  launch_pdl(rmsnorm_kernel, dim3(T), dim3(256), H * sizeof(float), st, static_cast<const __nv_bfloat16*>(x), static_cast<__nv_bfloat16*>(residual),
                                                    static_cast<const __nv_bfloat16*>(w), static_cast<__nv_bfloat16*>(y), H, eps,
                                                    offset, res_mult);
}
void launch_layernorm(const void* x, const void* w, const void* b, void* y, int T, int H, float eps, cudaStream_t st) {
  if (T == 0) return;
  layernorm_kernel<<<T, 256, H * sizeof(float), st>>>(static_cast<const __nv_bfloat16*>(x), static_cast<const __nv_bfloat16*>(w),
                                                      static_cast<const __nv_bfloat16*>(b), static_cast<__nv_bfloat16*>(y), H, eps);
}
void launch_act_mul(const void* in, void* out, long long T, int I, int act, cudaStream_t st) {
  const long long total = T * (I / 8);
  if (total == 0) return;
  launch_pdl(act_mul_kernel, dim3(static_cast<unsigned>((total + 255) / 256)), dim3(256), 0, st, static_cast<const __nv_bfloat16*>(in),
                                                                             static_cast<__nv_bfloat16*>(out), I, act, total);
}
void launch_act(const void* in, void* out, long long n, int act, bool is_f32, cudaStream_t st) {
  if (n == 0) return;
  const dim3 grid(static_cast<unsigned>((n + 2047) / 2048));
  if (is_f32) launch_pdl(act_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(in), static_cast<float*>(out), act, n);
  else launch_pdl(act_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<const __nv_bfloat16*>(in), static_cast<__nv_bfloat16*>(out), act, n);
}
void launch_embedding(const void* table, const int* ids, const void* pos_table, const int* pos, const void* type_table,
                      const int* types, void* out, int T, int H, int vocab, float scale, cudaStream_t st) {
  if (T == 0) return;
  launch_pdl(embedding_kernel, dim3(T), dim3(128), 0, st, static_cast<const __nv_bfloat16*>(table), ids, static_cast<const __nv_bfloat16*>(pos_table), pos,
                                      static_cast<const __nv_bfloat16*>(type_table), types, static_cast<__nv_bfloat16*>(out), H, vocab,
                                      scale);
}
void launch_bigram_embedding(const void* table, const void* bigram, const int* ids, const int* prev, float* out, int rows, int W, int vocab, int buckets,
                             long long mul_prev, long long mul_cur, float scale, void* out2, long long ld2, bool is_f32, cudaStream_t st) {
  if (rows == 0) return;
  if (is_f32)
    launch_pdl(bigram_embedding_kernel<float>, dim3(rows), dim3(128), 0, st, static_cast<const float*>(table), static_cast<const float*>(bigram), ids, prev,
               out, W, vocab, buckets, mul_prev, mul_cur, scale, static_cast<float*>(out2), ld2);
  else
    launch_pdl(bigram_embedding_kernel<__nv_bfloat16>, dim3(rows), dim3(128), 0, st, static_cast<const __nv_bfloat16*>(table),
               static_cast<const __nv_bfloat16*>(bigram), ids, prev, out, W, vocab, buckets, mul_prev, mul_cur, scale,
               static_cast<__nv_bfloat16*>(out2), ld2);
}
void launch_add_layernorm(float* residual, const float* delta, const float* w1, const float* b1, void* y1, const float* w2, const float* b2, void* y2,
                          int rows, int W, int y_pitch, float eps, bool is_f32, cudaStream_t st) {
  if (rows == 0) return;
  if (is_f32)
    launch_pdl(add_layernorm_kernel<float>, dim3(rows), dim3(256), W * sizeof(float), st, residual, delta, w1, b1, static_cast<float*>(y1), w2, b2,
               static_cast<float*>(y2), W, y_pitch, eps);
  else
    launch_pdl(add_layernorm_kernel<__nv_bfloat16>, dim3(rows), dim3(256), W * sizeof(float), st, residual, delta, w1, b1, static_cast<__nv_bfloat16*>(y1), w2,
               b2, static_cast<__nv_bfloat16*>(y2), W, y_pitch, eps);
}
void launch_gated_act(const void* in, long long ld_in, void* out, long long ld_out, int rows, int I, int act, bool is_f32, cudaStream_t st) {
  const long long total = static_cast<long long>(rows) * (I / 8);
  if (total == 0) return;
  const dim3 grid(static_cast<unsigned>((total + 255) / 256));
  if (is_f32) launch_pdl(gated_act_kernel<float>, grid, dim3(256), 0, st, static_cast<const float*>(in), ld_in, static_cast<float*>(out), ld_out, I, act, total);
  else
    launch_pdl(gated_act_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<const __nv_bfloat16*>(in), ld_in, static_cast<__nv_bfloat16*>(out), ld_out, I,
               act, total);
}
template <typename TSUB, typename TIO, bool RMS>
static void sandwich_dispatch_t(const SandwichArgs& a, int rows, cudaStream_t st) {
  const int width = a.W > a.y_width ? a.W : a.y_width;
  if (width <= 512) launch_pdl(sandwich_norm_kernel<TSUB, TIO, 1, 128, RMS>, dim3(rows), dim3(128), 0, st, a);
  else if (width <= 1024) launch_pdl(sandwich_norm_kernel<TSUB, TIO, 1, 256, RMS>, dim3(rows), dim3(256), 0, st, a);
  else if (width <= 2048) launch_pdl(sandwich_norm_kernel<TSUB, TIO, 2, 256, RMS>, dim3(rows), dim3(256), 0, st, a);
  else if (width <= 4096) launch_pdl(sandwich_norm_kernel<TSUB, TIO, 4, 256, RMS>, dim3(rows), dim3(256), 0, st, a);
  else launch_pdl(sandwich_norm_kernel<TSUB, TIO, 4, 1024, RMS>, dim3(rows), dim3(1024), 0, st, a);  // up to 16384 columns
}
template <typename TSUB, typename TIO>
static void sandwich_dispatch(const SandwichArgs& a, int rows, bool rms, cudaStream_t st) {
  if (rms) sandwich_dispatch_t<TSUB, TIO, true>(a, rows, st);
  else sandwich_dispatch_t<TSUB, TIO, false>(a, rows, st);
}
void launch_sandwich_norm(float* residual, const void* sub, long long ld_sub, bool sub_f32, const int* pos, const float* wts, int k, const float* w_sub,
                          bool sub_one, float mult, const float* w_next, bool next_one, bool rms, void* y, long long ld_y, int rows, int W, int y_width, float eps,
                          bool vec, bool is_f32, cudaStream_t st) {
  if (rows == 0) return;
  const SandwichArgs a = {residual, sub, ld_sub, pos, wts, k, w_sub, mult, w_next, y, ld_y, W, y_width, eps, vec ? 1 : 0, sub_one ? 1 : 0, next_one ? 1 : 0};
  if (is_f32 && sub_f32) sandwich_dispatch<float, float>(a, rows, rms, st);
  else if (is_f32) sandwich_dispatch<__nv_bfloat16, float>(a, rows, rms, st);
  else if (sub_f32) sandwich_dispatch<float, __nv_bfloat16>(a, rows, rms, st);
  else sandwich_dispatch<__nv_bfloat16, __nv_bfloat16>(a, rows, rms, st);
}
void launch_rope_pairs_kv(void* qkv, long long ld, const int* positions, const long long* slots, const float* cos_t, const float* sin_t, void* k_cache,
                          void* v_cache, int T, int H, int KV, int dk, int dv, int page, int half, int max_pos, bool is_f32, cudaStream_t st) {
  const long long n = static_cast<long long>(T) * (H * ((2 * half + 7) / 8) + KV * (dk / 8 + dv / 8));
  if (n == 0) return;
  const dim3 grid(static_cast<unsigned>((n + 255) / 256));
  if (is_f32)
    launch_pdl(rope_pairs_kv_kernel<float>, grid, dim3(256), 0, st, static_cast<float*>(qkv), ld, positions, slots, cos_t, sin_t, static_cast<float*>(k_cache),
               static_cast<float*>(v_cache), T, H, KV, dk, dv, page, half, max_pos);
  else
    launch_pdl(rope_pairs_kv_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<__nv_bfloat16*>(qkv), ld, positions, slots, cos_t, sin_t,
               static_cast<__nv_bfloat16*>(k_cache), static_cast<__nv_bfloat16*>(v_cache), T, H, KV, dk, dv, page, half, max_pos);
}
int launch_rope_heads_kv(const RopeHeadsArgs& a, bool is_f32, cudaStream_t st) {
  if (a.T == 0) return 0;
  if (a.dk > 1024 || a.dk % 8 != 0 || a.dv % 8 != 0 || static_cast<long long>(a.T) * (a.H + 2 * a.KV) > 0x7fffffffll) return 1;  // (the heads of a block share 48 KB)
  return is_f32 ? launch_rope_heads_t<float>(a, st) : launch_rope_heads_t<__nv_bfloat16>(a, st);
}
int launch_rope_kv(void* qkv, const int* positions, const long long* slots, const void* qn, const void* kn, const float* cos_t,
                   const float* sin_t, void* k_cache, void* v_cache, int T, int H, int KV, int D, int block_size, int rot_half,
                   float eps, float norm_offset, int max_pos, cudaStream_t st) {
  if (T == 0) return 0;
  const long long warps = static_cast<long long>(T) * (H + 2 * KV);
  const unsigned grid = static_cast<unsigned>((warps + 7) / 8);
#define DLV_ROPE(DD)                                                                                                         \
  launch_pdl(rope_kv_kernel<DD>, dim3(grid), dim3(256), 0, st, static_cast<__nv_bfloat16*>(qkv), positions, slots,                                \
                                           static_cast<const __nv_bfloat16*>(qn), static_cast<const __nv_bfloat16*>(kn), cos_t, \
                                           sin_t, static_cast<__nv_bfloat16*>(k_cache), static_cast<__nv_bfloat16*>(v_cache), T, \
                                           H, KV, block_size, rot_half, eps, norm_offset, max_pos)
  switch (D) {
    case 64: DLV_ROPE(64); break;
    case 128: DLV_ROPE(128); break;
    case 256: DLV_ROPE(256); break;
    default: return 1;
  }
#undef DLV_ROPE
  return 0;
}

}  // namespace dlv
