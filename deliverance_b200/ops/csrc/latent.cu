// Latent attention: the cache holds one compressed vector c (R values, RMS-normed) and one rotated key part (dr values) per token, shared
// by all query heads. Per head h the unrotated key is Wuk_h c and the value Wuv_h c; a score is (q_n . Wuk_h c + q_r . k_r) * scale.
//
// Two evaluation orders of the same product:
//   prompts   keys and values of the visible range are expanded once per step (gather -> GEMM) and go through the tcgen05 prefill kernel
//             (attention_tc.cu, latent layout): few operations per (query, key) pair;
//   decode    Wuk_h is moved to the query side (q' = Wuk_h^T q_n, "absorbed") and Wuv_h behind the weighted sum, so that all heads of a
//             row read the same R + dr cached values per key once: few bytes per key.
//
// Projection row p (one GEMM): [H heads x dk: q unrotated (dn, padded to dn_pad = a multiple of 64) | q rotated (padded likewise)] [latent R]
// [rotated key dr] [gate H x dv], blocks padded to 8 columns; padding columns are exact zeros (zero weight rows).
// Cache: c [pages, 1, page, Rp] and r [pages, 1, page, drp], Rp / drp = R / dr padded to 16 with zeros.
#include <stdexcept>
#include <string>

#include "common.cuh"
#include "gemm_api.h"

namespace dlv {

namespace {

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(sz) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x2(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ float ld1(const __nv_bfloat16* p) { return bf2f(*p); }
__device__ __forceinline__ float ld1(const float* p) { return *p; }
__device__ __forceinline__ void st1(__nv_bfloat16* p, float v) { *p = f2bf(v); }
__device__ __forceinline__ void st1(float* p, float v) { *p = v; }
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float* f) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const uint32_t* u = reinterpret_cast<const uint32_t*>(&v);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 a = unpack_bf162(u[j]);
    f[2 * j] = a.x;
    f[2 * j + 1] = a.y;
  }
}
__device__ __forceinline__ void load8(const float* p, float* f) {
  *reinterpret_cast<float4*>(f) = *reinterpret_cast<const float4*>(p);
  *reinterpret_cast<float4*>(f + 4) = *reinterpret_cast<const float4*>(p + 4);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float* f) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf162(f[0], f[1]), pack_bf162(f[2], f[3]), pack_bf162(f[4], f[5]), pack_bf162(f[6], f[7]));
}
__device__ __forceinline__ void store8(float* p, const float* f) {
  *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(f);
  *reinterpret_cast<float4*>(p + 4) = *reinterpret_cast<const float4*>(f + 4);
}

}  // namespace

// ------------------------------------------------------------------------------------------------ rotation, latent norm, cache write
// One warp per (row, unit): unit h < H rotates the rotated query part of head h in place; unit H norms the latent, rotates the shared key
// part and writes both to the cache rows (the projection row itself keeps its values).
template <typename T>
__global__ void __launch_bounds__(256) latent_prepare_kernel(T* __restrict__ p, long long ld, int rows, const int* __restrict__ positions,
                                                             const long long* __restrict__ slots, const float* __restrict__ norm_w,
                                                             const float* __restrict__ cos_t, const float* __restrict__ sin_t, int half, int max_pos,
                                                             T* __restrict__ c_cache, T* __restrict__ r_cache, LatentGeom g, int dn_pad, float eps) {
  pdl_wait();
  pdl_trigger();
  const int wg = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int units = g.H + 1;
  if (wg >= rows * units) return;
  const int t = wg / units, h = wg % units;
  int pos = positions[t];
  pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
  const float* ct = cos_t + static_cast<size_t>(pos) * half;
  const float* st = sin_t + static_cast<size_t>(pos) * half;
  T* row = p + static_cast<long long>(t) * ld;
  if (h < g.H) {
    T* q = row + h * g.dk + dn_pad;
    for (int i = lane; i < half; i += 32) {
      const float u = ld1(q + i), v = ld1(q + i + half), c = ct[i], s = st[i];
      st1(q + i, u * c - v * s);
      st1(q + i + half, v * c + u * s);
    }
    return;
  }
  const long long slot = slots[t];
  if (slot < 0) return;
  const T* src = row + g.off_c;
  const int R8 = (g.R + 7) & ~7;
  float ss = 0.f;
  for (int i = lane * 8; i < R8; i += 256) {
    float f[8];
    load8(src + i, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
  }
  ss = warp_sum(ss);
  const float inv = rsqrtf(ss / g.R + eps);
  T* dst = c_cache + slot * g.Rp;
  for (int i = lane * 8; i < g.Rp; i += 256) {
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (i < R8) load8(src + i, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] *= inv * norm_w[i + e];  // (norm_w is zero-padded to Rp)
    store8(dst + i, f);
  }
  const T* kr = row + g.off_r;
  T* rd = r_cache + slot * g.drp;
  for (int i = lane; i < g.drp; i += 32) {
    float v = 0.f;
    if (i < half) v = ld1(kr + i) * ct[i] - ld1(kr + i + half) * st[i];
    else if (i < 2 * half) v = ld1(kr + i) * ct[i - half] + ld1(kr + i - half) * st[i - half];
    else if (i < g.dr) v = ld1(kr + i);
    st1(rd + i, v);
  }
}

void launch_latent_prepare(void* p, long long ld, int rows, const int* positions, const long long* slots, const float* norm_w, const float* cos_t,
                           const float* sin_t, int half, int max_pos, void* c_cache, void* r_cache, const LatentGeom& g, float eps, bool is_f32,
                           cudaStream_t st) {
  if (rows == 0) return;
  const int dn_pad = (g.dn + 63) / 64 * 64;
  const long long warps = static_cast<long long>(rows) * (g.H + 1);
  const dim3 grid(static_cast<unsigned>((warps + 7) / 8));
  if (is_f32)
    launch_pdl(latent_prepare_kernel<float>, grid, dim3(256), 0, st, static_cast<float*>(p), ld, rows, positions, slots, norm_w, cos_t, sin_t, half, max_pos,
               static_cast<float*>(c_cache), static_cast<float*>(r_cache), g, dn_pad, eps);
  else
    launch_pdl(latent_prepare_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, static_cast<__nv_bfloat16*>(p), ld, rows, positions, slots, norm_w, cos_t, sin_t,
               half, max_pos, static_cast<__nv_bfloat16*>(c_cache), static_cast<__nv_bfloat16*>(r_cache), g, dn_pad, eps);
}

// ------------------------------------------------------------------------------------------------ gather of cached rows for expansion
// Sequence s: keys [key0[s], key0[s] + n_keys[s]) of cache sequence seq[s] -> rows row0[s].. of the flat buffers. One warp per row.
__global__ void __launch_bounds__(256) latent_gather_kernel(const __nv_bfloat16* __restrict__ c_cache, const __nv_bfloat16* __restrict__ r_cache,
                                                            const int* __restrict__ bt, int bt_stride, int page, const int* __restrict__ seq,
                                                            const int* __restrict__ key0, const int* __restrict__ n_keys, const int* __restrict__ row0,
                                                            __nv_bfloat16* __restrict__ c_out, int c_pitch, __nv_bfloat16* __restrict__ r_out, int r_pitch,
                                                            int Rp, int drp) {
  pdl_wait();
  pdl_trigger();
  const int s = blockIdx.y, j = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (j >= n_keys[s]) return;
  const int key = key0[s] + j;
  const long long slot = static_cast<long long>(bt[static_cast<long long>(seq[s]) * bt_stride + key / page]) * page + key % page;
  const long long out = row0[s] + j;
  for (int i = lane * 8; i < c_pitch; i += 256)
    *reinterpret_cast<uint4*>(c_out + out * c_pitch + i) = i < Rp ? *reinterpret_cast<const uint4*>(c_cache + slot * Rp + i) : make_uint4(0u, 0u, 0u, 0u);
  for (int i = lane * 8; i < r_pitch; i += 256)
    *reinterpret_cast<uint4*>(r_out + out * r_pitch + i) = i < drp ? *reinterpret_cast<const uint4*>(r_cache + slot * drp + i) : make_uint4(0u, 0u, 0u, 0u);
}

void launch_latent_gather(const void* c_cache, const void* r_cache, const int* bt, int bt_stride, int page, const int* seq, const int* key0,
                          const int* n_keys, const int* row0, int num_seqs, int max_rows, void* c_out, int c_pitch, void* r_out, int r_pitch, int Rp, int drp,
                          cudaStream_t st) {
  if (num_seqs == 0 || max_rows == 0) return;
  launch_pdl(latent_gather_kernel, dim3((max_rows + 7) / 8, num_seqs), dim3(256), 0, st, static_cast<const __nv_bfloat16*>(c_cache),
             static_cast<const __nv_bfloat16*>(r_cache), bt, bt_stride, page, seq, key0, n_keys, row0, static_cast<__nv_bfloat16*>(c_out), c_pitch,
             static_cast<__nv_bfloat16*>(r_out), r_pitch, Rp, drp);
}

// ------------------------------------------------------------------------------------------------ absorbed query
// q_lat[i][h] = [Wuk_h^T q_n (Rp) | q_r (drp)] for row i (row row_idx[i] of p). wuk [H][Rp][dn_pad]. mma.sync with 16 rows as the A operand;
// A and B use the same assignment of k elements to the instruction's k positions (lane c of a group of four owns 8 consecutive elements of
// every 32), so both operands are read with 16-byte loads. grid (H, row tiles of 16, blocks of 128 latent columns), 4 warps x 32 columns.
__global__ void __launch_bounds__(128) latent_absorb_kernel(const __nv_bfloat16* __restrict__ p, long long ld, const int* __restrict__ row_idx, int rows,
                                                            const __nv_bfloat16* __restrict__ wuk, __nv_bfloat16* __restrict__ q_lat, LatentGeom g,
                                                            int dn_pad) {
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, i0 = blockIdx.y * 16, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, c = lane & 3;
  const int CW = g.Rp + g.drp;
  const int n_base = blockIdx.z * 128 + warp * 32;
  if (n_base < g.Rp) {
    const bool va = i0 + gq < rows, vb = i0 + gq + 8 < rows;
    const int ra = va ? (row_idx ? row_idx[i0 + gq] : i0 + gq) : 0, rb = vb ? (row_idx ? row_idx[i0 + gq + 8] : i0 + gq + 8) : 0;
    const __nv_bfloat16* pa = p + ra * ld + h * g.dk + c * 8;
    const __nv_bfloat16* pb = p + rb * ld + h * g.dk + c * 8;
    float acc[4][4];
#pragma unroll
    for (int n = 0; n < 4; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll 2
    for (int k0 = 0; k0 < dn_pad; k0 += 32) {
      const uint4 xa = va ? *reinterpret_cast<const uint4*>(pa + k0) : zero;
      const uint4 xb = vb ? *reinterpret_cast<const uint4*>(pb + k0) : zero;
      const uint32_t a0[4] = {xa.x, xb.x, xa.y, xb.y}, a1[4] = {xa.z, xb.z, xa.w, xb.w};
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int r = n_base + n * 8 + gq;
        const uint4 w = n_base + n * 8 < g.Rp ? __ldg(reinterpret_cast<const uint4*>(wuk + (static_cast<size_t>(h) * g.Rp + r) * dn_pad + k0 + c * 8)) : zero;
        mma_16816(acc[n], a0, w.x, w.y);
        mma_16816(acc[n], a1, w.z, w.w);
      }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int col = n_base + n * 8 + 2 * c;
      if (n_base + n * 8 >= g.Rp) break;
      if (va) *reinterpret_cast<uint32_t*>(q_lat + (static_cast<size_t>(i0 + gq) * g.H + h) * CW + col) = pack_bf162(acc[n][0], acc[n][1]);
      if (vb) *reinterpret_cast<uint32_t*>(q_lat + (static_cast<size_t>(i0 + gq + 8) * g.H + h) * CW + col) = pack_bf162(acc[n][2], acc[n][3]);
    }
  }
  if (blockIdx.z == 0) {
    for (int e = threadIdx.x; e < 16 * g.drp; e += 128) {
      const int i = i0 + e / g.drp, d = e % g.drp;
      if (i >= rows) continue;
      const long long r = row_idx ? row_idx[i] : i;
      q_lat[(static_cast<size_t>(i) * g.H + h) * CW + g.Rp + d] = p[r * ld + h * g.dk + dn_pad + d];  // (zero beyond dr: padding columns)
    }
  }
}

void launch_latent_absorb(const void* p, long long ld, const int* row_idx, int rows, const void* wuk, void* q_lat, const LatentGeom& g, cudaStream_t st) {
  if (rows == 0) return;
  launch_pdl(latent_absorb_kernel, dim3(g.H, (rows + 15) / 16, (g.Rp + 127) / 128), dim3(128), 0, st, static_cast<const __nv_bfloat16*>(p), ld, row_idx, rows,
             static_cast<const __nv_bfloat16*>(wuk), static_cast<__nv_bfloat16*>(q_lat), g, (g.dn + 63) / 64 * 64);
}

// ------------------------------------------------------------------------------------------------ decode attention over the latent cache
// grid (rows, groups of 16 * MH heads, splits), 8 warps. All heads of the group share every cached key row: tiles of BK keys ([c | r], padded
// pitch so that ldmatrix is free of bank conflicts) arrive by cp.async in two stages; the score tile [16 MH heads x BK keys] is computed with
// the keys split over the warps, goes through shared memory for the online softmax (fp32), and the probabilities come back as bf16 A
// operand of the weighted sum, for which the warps split the latent columns (the K rows double as V). Partial sums leave in fp32, with the
// running maximum and sum of every (row, head, split); latent_expand_kernel merges them.
template <int MH, int BK>
struct LatentDecodeSmem {
  int pitch, pitch_p, pitch_s;
  int off_q, off_p, off_s, off_st, bytes;
  __host__ __device__ explicit LatentDecodeSmem(int CW) {
    pitch = (CW + 8) * 2;         // CW is a multiple of 16: an odd number of 16-byte units
    pitch_p = (BK + 8) * 2;
    pitch_s = BK + 4;             // floats
    off_q = 2 * BK * pitch;
    off_p = off_q + 16 * MH * pitch;
    off_s = off_p + 16 * MH * pitch_p;
    off_st = off_s + 16 * MH * pitch_s * 4;
    bytes = off_st + 3 * 16 * MH * 4;
  }
};

template <int NPW, int MH, int BK>  // NPW: 16-column blocks of the latent per warp
__global__ void __launch_bounds__(256) latent_decode_kernel(const __nv_bfloat16* __restrict__ q_lat, const __nv_bfloat16* __restrict__ c_cache,
                                                            const __nv_bfloat16* __restrict__ r_cache, const int* __restrict__ bt, int bt_stride,
                                                            const int* __restrict__ row_seq, const int* __restrict__ row_ctx, float* __restrict__ part_o,
                                                            float* __restrict__ part_ml, LatentGeom g, int page, float scale, int window, int splits) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t lsm[];
  const int CW = g.Rp + g.drp;
  const LatentDecodeSmem<MH, BK> L(CW);
  const uint32_t base_u = smem_u32(lsm);
  float* sS = reinterpret_cast<float*>(lsm + L.off_s);
  float* sM = reinterpret_cast<float*>(lsm + L.off_st);
  float* sL = sM + 16 * MH;
  float* sA = sL + 16 * MH;
  const int i = blockIdx.x, h0 = blockIdx.y * 16 * MH, sp = blockIdx.z;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, t4 = lane & 3;
  const int nh = min(16 * MH, g.H - h0);
  const int ctx = row_ctx[i];
  const long long bt_row = static_cast<long long>(row_seq ? row_seq[i] : i) * bt_stride;
  const int first_key = (window > 0 && ctx > window) ? ctx - window : 0;
  const int tl = first_key / BK, th = (ctx + BK - 1) / BK;
  const int per = (th - tl + splits - 1) / splits;
  const int t0 = tl + sp * per, t1 = min(th, t0 + per);

  const int cq = CW / 8, cc = g.Rp / 8;  // 16-byte chunks per row: whole, latent part
  for (int r = warp; r < 16 * MH; r += 8) {
    const __nv_bfloat16* src = q_lat + (static_cast<size_t>(i) * g.H + h0 + r) * CW;
    for (int k = lane; k < cq; k += 32)
      *reinterpret_cast<uint4*>(lsm + L.off_q + r * L.pitch + k * 16) = r < nh ? *reinterpret_cast<const uint4*>(src + k * 8) : make_uint4(0u, 0u, 0u, 0u);
  }
  if (tid < 16 * MH) {
    sM[tid] = -INFINITY;
    sL[tid] = 0.f;
  }
  auto load_tile = [&](int tile, int buf) {
#pragma unroll
    for (int e = 0; e < BK / 8; ++e) {
      const int r = warp * (BK / 8) + e, key = tile * BK + r;
      const bool valid = key < ctx;
      const long long slot = valid ? static_cast<long long>(bt[bt_row + key / page]) * page + key % page : 0;
      const uint32_t dst = base_u + (buf * BK + r) * L.pitch;
      for (int k = lane; k < cq; k += 32) {
        const __nv_bfloat16* src = k < cc ? c_cache + slot * g.Rp + k * 8 : r_cache + slot * g.drp + (k - cc) * 8;
        cp_async16(dst + k * 16, src, valid);
      }
    }
    cp_async_commit();
  };
  float o[MH][NPW][2][4];
#pragma unroll
  for (int m = 0; m < MH; ++m)
#pragma unroll
    for (int j = 0; j < NPW; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[m][j][0][e] = o[m][j][1][e] = 0.f;
  const int np = g.Rp / 16;
  if (t0 < t1) load_tile(t0, 0);
  for (int tile = t0; tile < t1; ++tile) {
    const int buf = (tile - t0) & 1;
    if (tile + 1 < t1) {
      load_tile(tile + 1, buf ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint32_t kb = base_u + buf * BK * L.pitch;
    // ---- scores: MH == 1: warp w takes 8 keys; MH == 2: warps split as 2 head groups x 4 groups of 16 keys
    if (MH == 2 || warp * 8 < BK) {
      constexpr int NT = MH == 2 ? BK / 32 : 1;
      const int m = MH == 2 ? (warp & 1) : 0, key_w = MH == 2 ? (warp >> 1) * (BK / 4) : warp * 8;
      float s[NT][4];
#pragma unroll
      for (int n = 0; n < NT; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      const uint32_t qa = base_u + L.off_q + (m * 16 + (lane & 15)) * L.pitch + (lane >> 4) * 16;
      const uint32_t ka = kb + (key_w + (NT == 2 ? (lane & 7) + (lane >> 4) * 8 : (lane & 7))) * L.pitch + ((lane >> 3) & 1) * 16;
#pragma unroll 4
      for (int ks = 0; ks < CW / 16; ++ks) {
        uint32_t a[4];
        ldmatrix_x4(qa + ks * 32, a);
        if constexpr (NT == 2) {
          uint32_t b[4];
          ldmatrix_x4(ka + ks * 32, b);
          mma_16816(s[0], a, b[0], b[1]);
          mma_16816(s[1], a, b[2], b[3]);
        } else {
          uint32_t b[2];
          ldmatrix_x2(ka + ks * 32, b);
          mma_16816(s[0], a, b[0], b[1]);
        }
      }
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int col = key_w + n * 8 + 2 * t4;
        float* d = sS + (m * 16 + gq) * L.pitch_s + col;
        *reinterpret_cast<float2*>(d) = make_float2(s[n][0], s[n][1]);
        *reinterpret_cast<float2*>(d + 8 * L.pitch_s) = make_float2(s[n][2], s[n][3]);
      }
    }
    __syncthreads();
    // ---- online softmax: 256 / (16 MH) threads per head row
    {
      constexpr int TPR = 16 / MH, KPT = BK / TPR;
      const int r = tid / TPR, c0 = tid % TPR;
      float v[KPT], mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < KPT; ++e) {
        const int col = e * TPR + c0, key = tile * BK + col;
        v[e] = (key < ctx && key >= first_key) ? sS[r * L.pitch_s + col] * scale : -INFINITY;
        mx = fmaxf(mx, v[e]);
      }
#pragma unroll
      for (int off = 1; off < TPR; off <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_old = sM[r], m_new = fmaxf(m_old, mx);
      float sum = 0.f;
      __nv_bfloat16* pr = reinterpret_cast<__nv_bfloat16*>(lsm + L.off_p + r * L.pitch_p);
#pragma unroll
      for (int e = 0; e < KPT; ++e) {
        const float w = v[e] == -INFINITY ? 0.f : __expf(v[e] - m_new);
        sum += w;
        pr[e * TPR + c0] = f2bf(w);
      }
#pragma unroll
      for (int off = 1; off < TPR; off <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      __syncwarp();
      if (c0 == 0) {
        const float alpha = m_old == -INFINITY ? 0.f : __expf(m_old - m_new);
        sA[r] = alpha;
        sM[r] = m_new;
        sL[r] = sL[r] * alpha + sum;
      }
    }
    __syncthreads();
    // ---- weighted sum: warp w owns the 16-column blocks w, w + 8, ...
#pragma unroll
    for (int m = 0; m < MH; ++m) {
      const float a0 = sA[m * 16 + gq], a1 = sA[m * 16 + gq + 8];
#pragma unroll
      for (int j = 0; j < NPW; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          o[m][j][n][0] *= a0;
          o[m][j][n][1] *= a0;
          o[m][j][n][2] *= a1;
          o[m][j][n][3] *= a1;
        }
    }
#pragma unroll
    for (int ks = 0; ks < BK / 16; ++ks) {
      uint32_t a[MH][4];
#pragma unroll
      for (int m = 0; m < MH; ++m) ldmatrix_x4(base_u + L.off_p + (m * 16 + (lane & 15)) * L.pitch_p + (lane >> 4) * 16 + ks * 32, a[m]);
#pragma unroll
      for (int j = 0; j < NPW; ++j) {
        const int blk = warp + 8 * j;
        if (blk < np) {  // warp-uniform
          uint32_t b[4];
          ldmatrix_x4_trans(kb + (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * L.pitch + blk * 32 + (lane >> 4) * 16, b);
#pragma unroll
          for (int m = 0; m < MH; ++m) {
            mma_16816(o[m][j][0], a[m], b[0], b[1]);
            mma_16816(o[m][j][1], a[m], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();  // the stage, the scores and the probabilities are overwritten by the next tile
  }
  // ---- partial results
#pragma unroll
  for (int m = 0; m < MH; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = m * 16 + gq + half * 8;
      if (r >= nh) continue;
      float* dst = part_o + ((static_cast<size_t>(i) * g.H + h0 + r) * splits + sp) * g.Rp;
#pragma unroll
      for (int j = 0; j < NPW; ++j) {
        const int blk = warp + 8 * j;
        if (blk >= np) continue;
#pragma unroll
        for (int n = 0; n < 2; ++n)
          *reinterpret_cast<float2*>(dst + blk * 16 + n * 8 + 2 * t4) = make_float2(o[m][j][n][2 * half], o[m][j][n][2 * half + 1]);
      }
    }
  if (tid < nh) {
    float* ml = part_ml + ((static_cast<size_t>(i) * g.H + h0 + tid) * splits + sp) * 2;
    ml[0] = sM[tid];
    ml[1] = sL[tid];
  }
}

template <int NPW, int MH, int BK>
static int launch_latent_decode_t(const void* q_lat, const void* c_cache, const void* r_cache, const int* bt, int bt_stride, const int* row_seq,
                                  const int* row_ctx, int rows, float* part_o, float* part_ml, const LatentGeom& g, int page, float scale, int window,
                                  int splits, cudaStream_t st) {
  const LatentDecodeSmem<MH, BK> L(g.Rp + g.drp);
  if (L.bytes > 227 * 1024) return 1;
  static PerDeviceOnce attr_once;
  if (attr_once.first()) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<NPW, MH, BK>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) throw std::runtime_error(std::string("latent decode attention: cudaFuncSetAttribute: ") + cudaGetErrorString(e));
  }
  launch_pdl(latent_decode_kernel<NPW, MH, BK>, dim3(rows, (g.H + 16 * MH - 1) / (16 * MH), splits), dim3(256), static_cast<size_t>(L.bytes), st,
             static_cast<const __nv_bfloat16*>(q_lat), static_cast<const __nv_bfloat16*>(c_cache), static_cast<const __nv_bfloat16*>(r_cache), bt, bt_stride,
             row_seq, row_ctx, part_o, part_ml, g, page, scale, window, splits);
  return 0;
}

int launch_latent_decode(const void* q_lat, const void* c_cache, const void* r_cache, const int* bt, int bt_stride, const int* row_seq, const int* row_ctx,
                         int rows, float* part_o, float* part_ml, const LatentGeom& g, int page, float scale, int window, int splits, cudaStream_t st) {
  if (rows == 0) return 0;
#define DLV_LD(N, M, B) \
  return launch_latent_decode_t<N, M, B>(q_lat, c_cache, r_cache, bt, bt_stride, row_seq, row_ctx, rows, part_o, part_ml, g, page, scale, window, splits, st)
  if (g.Rp <= 128) {
    if (g.H > 16) { DLV_LD(1, 2, 64); }
    DLV_LD(1, 1, 64);
  }
  if (g.Rp <= 256) {
    if (g.H > 16) { DLV_LD(2, 2, 64); }
    DLV_LD(2, 1, 64);
  }
  if (g.Rp <= 512) {
    if (g.H > 16 && LatentDecodeSmem<2, 64>(g.Rp + g.drp).bytes <= 227 * 1024) { DLV_LD(4, 2, 64); }
    if (LatentDecodeSmem<1, 64>(g.Rp + g.drp).bytes <= 227 * 1024) { DLV_LD(4, 1, 64); }
  }
  if (g.Rp <= 1024) { DLV_LD(8, 1, 32); }
#undef DLV_LD
  return 1;
}

// ------------------------------------------------------------------------------------------------ merge of the splits, value weights, gate
// out[row][h * dv + v] = sigmoid(gate) * sum_r wuv[h][v][r] * o_lat[r], with o_lat = the normalised sum over the splits. wuv [H][dv8][Kp].
// grid (H, row tiles of 16, blocks of 32 value columns), 4 warps x 8 columns; the merged rows are the A operand, staged in shared memory.
constexpr int kLatentMaxSplits = 64;
__global__ void __launch_bounds__(128) latent_expand_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int splits,
                                                            const int* __restrict__ row_idx, int rows, const __nv_bfloat16* __restrict__ wuv,
                                                            const __nv_bfloat16* __restrict__ p, long long ld, __nv_bfloat16* __restrict__ out, int out_pitch,
                                                            LatentGeom g) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t esm[];
  const int pitch = g.Kp + 8;
  __nv_bfloat16* sO = reinterpret_cast<__nv_bfloat16*>(esm);                 // [16][pitch]
  float* sW = reinterpret_cast<float*>(esm + 16 * pitch * 2);                // [16][splits] weights, already divided by the row's sum
  const int h = blockIdx.x, i0 = blockIdx.y * 16, n0 = blockIdx.z * 32, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, c = lane & 3;
  const int nr = min(16, rows - i0);
  if (tid < 16) {
    if (tid < nr) {
      const float* ml = part_ml + (static_cast<size_t>(i0 + tid) * g.H + h) * splits * 2;
      float m = -INFINITY;
      for (int s = 0; s < splits; ++s) m = fmaxf(m, ml[2 * s]);
      float den = 0.f;
      for (int s = 0; s < splits; ++s) {
        const float w = ml[2 * s] == -INFINITY ? 0.f : __expf(ml[2 * s] - m);
        sW[tid * splits + s] = w;
        den += w * ml[2 * s + 1];
      }
      const float inv = den > 0.f ? 1.f / den : 0.f;
      for (int s = 0; s < splits; ++s) sW[tid * splits + s] *= inv;
    }
  }
  __syncthreads();
  const int quads = g.Kp / 4;
  for (int e = tid; e < 16 * quads; e += 128) {
    const int r = e / quads, k = (e % quads) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (r < nr && k < g.Rp) {
      const float* src = part_o + (static_cast<size_t>(i0 + r) * g.H + h) * splits * g.Rp + k;
      for (int s = 0; s < splits; ++s) {
        const float w = sW[r * splits + s];
        const float4 a = *reinterpret_cast<const float4*>(src + static_cast<size_t>(s) * g.Rp);
        v.x += w * a.x;
        v.y += w * a.y;
        v.z += w * a.z;
        v.w += w * a.w;
      }
    }
    *reinterpret_cast<uint2*>(sO + r * pitch + k) = make_uint2(pack_bf162(v.x, v.y), pack_bf162(v.z, v.w));
  }
  __syncthreads();
  const int dv8 = (g.dv + 7) & ~7, nb = n0 + warp * 8;
  if (nb >= dv8) return;
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  const __nv_bfloat16* w = wuv + (static_cast<size_t>(h) * dv8 + nb + gq) * g.Kp + c * 8;
  const __nv_bfloat16* xa = sO + gq * pitch + c * 8;
#pragma unroll 4
  for (int k0 = 0; k0 < g.Kp; k0 += 32) {
    const uint4 b = __ldg(reinterpret_cast<const uint4*>(w + k0));
    const uint4 x0 = *reinterpret_cast<const uint4*>(xa + k0), x1 = *reinterpret_cast<const uint4*>(xa + 8 * pitch + k0);
    const uint32_t a0[4] = {x0.x, x1.x, x0.y, x1.y}, a1[4] = {x0.z, x1.z, x0.w, x1.w};
    mma_16816(acc, a0, b.x, b.y);
    mma_16816(acc, a1, b.z, b.w);
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int i = gq + half * 8;
    if (i >= nr) continue;
    const long long row = row_idx ? row_idx[i0 + i] : i0 + i;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int v = nb + 2 * c + e;
      if (v >= g.dv) continue;
      float y = acc[half * 2 + e];
      if (g.off_g >= 0) y /= 1.f + __expf(-bf2f(p[row * ld + g.off_g + h * g.dv + v]));
      out[row * out_pitch + h * g.dv + v] = f2bf(y);
    }
  }
}

void launch_latent_expand(const float* part_o, const float* part_ml, int splits, const int* row_idx, int rows, const void* wuv, const void* p, long long ld,
                          void* out, int out_pitch, const LatentGeom& g, cudaStream_t st) {
  if (rows == 0) return;
  const size_t smem = static_cast<size_t>(16) * (g.Kp + 8) * 2 + static_cast<size_t>(16) * splits * 4;
  if (splits > kLatentMaxSplits || smem > 48 * 1024) throw std::runtime_error("latent expand: too many splits or latent columns");
  launch_pdl(latent_expand_kernel, dim3(g.H, (rows + 15) / 16, (g.dv + 31) / 32), dim3(128), smem, st, part_o, part_ml, splits, row_idx, rows,
             static_cast<const __nv_bfloat16*>(wuv), static_cast<const __nv_bfloat16*>(p), ld, static_cast<__nv_bfloat16*>(out), out_pitch, g);
}

// ------------------------------------------------------------------------------------------------ 32-bit form
// Whole mixer core of one (row, head) in fp32: absorbed query, online softmax over the cached keys, value weights, gate. grid (rows, H).
__global__ void __launch_bounds__(256) latent_rows_f32_kernel(const float* __restrict__ p, long long ld, const int* __restrict__ row_idx,
                                                              const int* __restrict__ row_seq, const int* __restrict__ row_ctx, const float* __restrict__ wuk,
                                                              const float* __restrict__ wuv, const float* __restrict__ c_cache,
                                                              const float* __restrict__ r_cache, const int* __restrict__ bt, int bt_stride,
                                                              float* __restrict__ out, int out_pitch, LatentGeom g, int dn_pad, int page, float scale,
                                                              int window) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float fsm[];
  float* sQ = fsm;                 // [Rp + drp] absorbed query
  float* sO = sQ + g.Rp + g.drp;   // [Rp]
  float* sP = sO + g.Rp;           // [64] scores, then weights
  __shared__ long long sSlot[64];
  const int i = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const long long row = row_idx ? row_idx[i] : i;
  const int ctx = row_ctx[i];
  const long long bt_row = static_cast<long long>(row_seq ? row_seq[i] : i) * bt_stride;
  const float* q = p + row * ld + h * g.dk;
  for (int r = warp; r < g.Rp; r += 8) {
    const float* w = wuk + (static_cast<size_t>(h) * g.Rp + r) * dn_pad;
    float s = 0.f;
    for (int d = lane; d < g.dn; d += 32) s += q[d] * w[d];
    s = warp_sum(s);
    if (lane == 0) sQ[r] = s;
  }
  for (int d = tid; d < g.drp; d += 256) sQ[g.Rp + d] = q[dn_pad + d];
  for (int r = tid; r < g.Rp; r += 256) sO[r] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;  // every thread keeps the same copy
  const int first_key = (window > 0 && ctx > window) ? ctx - window : 0;
  for (int k0 = first_key; k0 < ctx; k0 += 64) {
    const int n = min(64, ctx - k0);
    __syncthreads();
    if (tid < n) sSlot[tid] = static_cast<long long>(bt[bt_row + (k0 + tid) / page]) * page + (k0 + tid) % page;
    __syncthreads();
    for (int j = warp; j < n; j += 8) {
      const float* c = c_cache + sSlot[j] * g.Rp;
      const float* kr = r_cache + sSlot[j] * g.drp;
      float s = 0.f;
      for (int r = lane; r < g.Rp; r += 32) s += sQ[r] * c[r];
      for (int d = lane; d < g.drp; d += 32) s += sQ[g.Rp + d] * kr[d];
      s = warp_sum(s);
      if (lane == 0) sP[j] = s * scale;
    }
    __syncthreads();
    float mx = m_run;
    for (int j = 0; j < n; ++j) mx = fmaxf(mx, sP[j]);
    const float alpha = m_run == -INFINITY ? 0.f : expf(m_run - mx);
    m_run = mx;
    __syncthreads();
    if (tid < n) sP[tid] = expf(sP[tid] - mx);
    __syncthreads();
    float sum = 0.f;
    for (int j = 0; j < n; ++j) sum += sP[j];
    l_run = l_run * alpha + sum;
    for (int r = tid; r < g.Rp; r += 256) {
      float a = sO[r] * alpha;
      for (int j = 0; j < n; ++j) a += sP[j] * c_cache[sSlot[j] * g.Rp + r];
      sO[r] = a;
    }
  }
  __syncthreads();
  const int dv8 = (g.dv + 7) & ~7;
  for (int v = warp; v < g.dv; v += 8) {
    const float* w = wuv + (static_cast<size_t>(h) * dv8 + v) * g.Kp;
    float s = 0.f;
    for (int r = lane; r < g.Rp; r += 32) s += sO[r] * w[r];
    s = warp_sum(s) / l_run;
    if (lane == 0) {
      if (g.off_g >= 0) s /= 1.f + expf(-p[row * ld + g.off_g + h * g.dv + v]);
      out[row * out_pitch + h * g.dv + v] = s;
    }
  }
}

int launch_latent_rows_f32(const float* p, long long ld, const int* row_idx, const int* row_seq, const int* row_ctx, int rows, const float* wuk,
                           const float* wuv, const float* c_cache, const float* r_cache, const int* bt, int bt_stride, float* out, int out_pitch,
                           const LatentGeom& g, int page, float scale, int window, cudaStream_t st) {
  if (rows == 0) return 0;
  const size_t smem = static_cast<size_t>(2 * g.Rp + g.drp + 64) * 4;
  if (smem > 46 * 1024 || g.H > 65535) return 1;
  launch_pdl(latent_rows_f32_kernel, dim3(rows, g.H), dim3(256), smem, st, p, ld, row_idx, row_seq, row_ctx, wuk, wuv, c_cache, r_cache, bt, bt_stride, out,
             out_pitch, g, (g.dn + 63) / 64 * 64, page, scale, window);
  return 0;
}

// ------------------------------------------------------------------------------------------------ fp32 projection
// out = x W^T (+ bias), true fp32 FMA. 64 x 64 tiles, 256 threads with 4 x 4 accumulators, K in steps of 16.
__global__ void __launch_bounds__(256) linear_f32_kernel(const float* __restrict__ x, int ldx, const float* __restrict__ w, const float* __restrict__ bias,
                                                         float* __restrict__ out, int ldo, int M, int N, int K) {
  pdl_wait();
  pdl_trigger();
  __shared__ float sx[16][68], sw[16][68];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    for (int e = tid; e < 64 * 16; e += 256) {
      const int r = e >> 4, k = e & 15;
      sx[k][r] = (m0 + r < M && k0 + k < K) ? x[static_cast<size_t>(m0 + r) * ldx + k0 + k] : 0.f;
      sw[k][r] = (n0 + r < N && k0 + k < K) ? w[static_cast<size_t>(n0 + r) * K + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sx[k][ty * 4]), b = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] += av[i] * bv[j];
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) out[static_cast<size_t>(m) * ldo + n] = acc[i][j] + (bias ? bias[n] : 0.f);
    }
  }
}

void launch_linear_f32(const float* x, int ldx, const float* w, const float* bias, float* out, int ldo, int M, int N, int K, cudaStream_t st) {
  if (M == 0 || N == 0) return;
  const unsigned gy = static_cast<unsigned>((M + 63) / 64);
  if (gy > 65535) throw std::runtime_error("fp32 projection: too many rows");
  launch_pdl(linear_f32_kernel, dim3((N + 63) / 64, gy), dim3(256), 0, st, x, ldx, w, bias, out, ldo, M, N, K);
}

}  // namespace dlv
