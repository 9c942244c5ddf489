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
#include <type_traits>

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

__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

}  // namespace

// ------------------------------------------------------------------------------------------------ rotation, latent norm, cache write
// One warp: norm of the latent and rotation of the shared key part of one projection row, both written to cache row `slot`.
template <typename T>
__device__ __forceinline__ void latent_cache_row(const T* __restrict__ row, long long slot, int pos, const LatentPrep& pr, const LatentGeom& g, int lane) {
  const float* ct = pr.cos_t + static_cast<size_t>(pos) * pr.half;
  const float* st = pr.sin_t + static_cast<size_t>(pos) * pr.half;
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
  const float inv = rsqrtf(ss / g.R + pr.eps);
  T* dst = static_cast<T*>(pr.c_cache) + slot * g.Rp;
  for (int i = lane * 8; i < g.Rp; i += 256) {
    float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (i < R8) load8(src + i, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] *= inv * pr.norm_w[i + e];  // (norm_w is zero-padded to Rp)
    store8(dst + i, f);
  }
  const T* kr = row + g.off_r;
  T* rd = static_cast<T*>(pr.r_cache) + slot * g.drp;
  for (int i = lane; i < g.drp; i += 32) {
    float v = 0.f;
    if (i < pr.half) v = ld1(kr + i) * ct[i] - ld1(kr + i + pr.half) * st[i];
    else if (i < 2 * pr.half) v = ld1(kr + i) * ct[i - pr.half] + ld1(kr + i - pr.half) * st[i - pr.half];
    else if (i < g.dr) v = ld1(kr + i);
    st1(rd + i, v);
  }
}
__device__ __forceinline__ int clamp_pos(int pos, int max_pos) { return pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos); }

// grid.y 0: rotates the rotated query parts in place, one thread per VEC pairs (row, head, pairs i .. i + VEC - 1); grid.y 1: one warp per row
// for the cache (the projection row itself keeps its latent and key).
template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_prepare_kernel(T* __restrict__ p, long long ld, int rows, LatentPrep pr, LatentGeom g, int dn_pad) {
  pdl_wait();
  pdl_trigger();
  if (blockIdx.y == 1) {  // (not launched for rows without a latent)
    const int t = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (t >= rows || pr.slots[t] < 0) return;
    latent_cache_row<T>(p + t * ld, pr.slots[t], clamp_pos(pr.positions[t], pr.max_pos), pr, g, threadIdx.x & 31);
    return;
  }
  const int per_head = pr.half / VEC, per_row = g.H * per_head;
  const long long idx = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (idx >= static_cast<long long>(rows) * per_row) return;
  const int t = static_cast<int>(idx / per_row), k = static_cast<int>(idx % per_row), h = k / per_head, i = (k % per_head) * VEC;
  const int pos = clamp_pos(pr.positions[t], pr.max_pos);
  T* q = p + t * ld + h * g.dk + dn_pad + i;
  const float* ct = pr.cos_t + static_cast<size_t>(pos) * pr.half + i;
  const float* st = pr.sin_t + static_cast<size_t>(pos) * pr.half + i;
  if constexpr (VEC == 8) {
    float u[8], v[8], c[8], s[8];
    load8(q, u);
    load8(q + pr.half, v);
    load8(ct, c);
    load8(st, s);
    float a[8], b[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      a[e] = u[e] * c[e] - v[e] * s[e];
      b[e] = v[e] * c[e] + u[e] * s[e];
    }
    store8(q, a);
    store8(q + pr.half, b);
  } else {
    const float u = ld1(q), v = ld1(q + pr.half), c = ct[0], s = st[0];
    st1(q, u * c - v * s);
    st1(q + pr.half, v * c + u * s);
  }
}

template <typename T>
static void launch_latent_prepare_t(void* p, long long ld, int rows, const LatentPrep& pr, const LatentGeom& g, cudaStream_t st) {
  const int dn_pad = (g.dn + 63) / 64 * 64;
  const int vec = pr.half % 8 == 0 ? 8 : 1;
  const long long rot = (static_cast<long long>(rows) * g.H * (pr.half / vec) + 255) / 256, cache = (rows + 7) / 8;
  const dim3 grid(static_cast<unsigned>(rot > cache ? rot : cache), g.off_c >= 0 ? 2 : 1);
  if (vec == 8) launch_pdl(latent_prepare_kernel<T, 8>, grid, dim3(256), 0, st, static_cast<T*>(p), ld, rows, pr, g, dn_pad);
  else launch_pdl(latent_prepare_kernel<T, 1>, grid, dim3(256), 0, st, static_cast<T*>(p), ld, rows, pr, g, dn_pad);
}

void launch_latent_prepare(void* p, long long ld, int rows, const LatentPrep& pr, const LatentGeom& g, bool is_f32, cudaStream_t st) {
  if (rows == 0) return;
  if (is_f32) launch_latent_prepare_t<float>(p, ld, rows, pr, g, st);
  else launch_latent_prepare_t<__nv_bfloat16>(p, ld, rows, pr, g, st);
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
// With `prep` (decode batches, row_idx == nullptr) the launch also does the work of latent_prepare_kernel: the query's rotated part is rotated
// on its way to q_lat, and the CTAs of one more grid column write the cache rows.
__global__ void __launch_bounds__(128) latent_absorb_kernel(const __nv_bfloat16* __restrict__ p, long long ld, const int* __restrict__ row_idx, int rows,
                                                            const __nv_bfloat16* __restrict__ wuk, __nv_bfloat16* __restrict__ q_lat, LatentGeom g,
                                                            int dn_pad, LatentPrep pr, int prep) {
  const int h = blockIdx.x, i0 = blockIdx.y * 16, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, c = lane & 3;
  if (h < g.H) {  // weights do not depend on the kernel in front: towards L2 while it finishes
    const char* w0 = reinterpret_cast<const char*>(wuk + (static_cast<size_t>(h) * g.Rp + blockIdx.z * 128) * dn_pad);
    const int bytes = min(128, g.Rp - static_cast<int>(blockIdx.z) * 128) * dn_pad * 2;
    for (int o = threadIdx.x * 128; o < bytes; o += 128 * 128) prefetch_l2(w0 + o);
  }
  pdl_wait();
  pdl_trigger();
  if (h == g.H) {
    for (int r = blockIdx.z * 4 + warp; r < 16; r += 4 * gridDim.z)
      if (i0 + r < rows && pr.slots[i0 + r] >= 0)
        latent_cache_row<__nv_bfloat16>(p + (i0 + r) * ld, pr.slots[i0 + r], clamp_pos(pr.positions[i0 + r], pr.max_pos), pr, g, lane);
    return;
  }
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
  // rotated part: 8 threads per row, columns shared out over the blocks of the grid's z direction
  const int i = i0 + (threadIdx.x >> 3);
  if (i < rows) {
    const long long r = row_idx ? row_idx[i] : i;
    const __nv_bfloat16* q = p + r * ld + h * g.dk + dn_pad;
    __nv_bfloat16* dst = q_lat + (static_cast<size_t>(i) * g.H + h) * CW + g.Rp;
    const size_t at = prep ? static_cast<size_t>(clamp_pos(pr.positions[i], pr.max_pos)) * pr.half : 0;
    for (int d = (threadIdx.x & 7) + 8 * blockIdx.z; d < g.drp; d += 8 * gridDim.z) {
      __nv_bfloat16 v = q[d];  // (zero beyond dr: padding columns)
      if (prep && d < 2 * pr.half) {
        const int k = d < pr.half ? d : d - pr.half;
        const float a = bf2f(q[k]), b = bf2f(q[k + pr.half]), cs = pr.cos_t[at + k], sn = pr.sin_t[at + k];
        v = f2bf(d < pr.half ? a * cs - b * sn : b * cs + a * sn);
      }
      dst[d] = v;
    }
  }
}

void launch_latent_absorb(const void* p, long long ld, const int* row_idx, int rows, const void* wuk, void* q_lat, const LatentGeom& g,
                          const LatentPrep* prep, cudaStream_t st) {
  if (rows == 0) return;
  const LatentPrep none = {};
  launch_pdl(latent_absorb_kernel, dim3(g.H + (prep && g.off_c >= 0 ? 1 : 0), (rows + 15) / 16, (g.Rp + 127) / 128), dim3(128), 0, st, static_cast<const __nv_bfloat16*>(p),
             ld, row_idx, rows, static_cast<const __nv_bfloat16*>(wuk), static_cast<__nv_bfloat16*>(q_lat), g, (g.dn + 63) / 64 * 64, prep ? *prep : none,
             prep ? 1 : 0);
}

// CTAs per cluster for a number of splits that is a power of two
int latent_cluster_size(int splits) { return splits >= 8 ? 8 : (splits >= 4 ? 4 : (splits >= 2 ? 2 : 1)); }
int g_latent_head_groups = 0;  // 1: groups of 16 heads only (tests, comparisons)

// ------------------------------------------------------------------------------------------------ decode attention over the latent cache
// grid (splits, rows, groups of 16 * MH heads), 8 * MH warps. All heads of the group share every cached key row: tiles of 32 keys ([c | r],
// padded pitch so that ldmatrix is free of bank conflicts) arrive by cp.async, NST - 1 tiles ahead (one bulk copy per row and part instead
// was slower, 77 against 64 us at 64 sequences of 2048 keys of 512 + 64: the copy engine starts one in about 40 ns). Per tile: the
// scores [16 MH heads x 32 keys] (a warp owns 16 heads, 8 keys and half of the k range; most of its part of the query stays in registers,
// because shared-memory bandwidth is what the tile loop runs out of first), through shared memory to the online softmax (fp32), and back as
// the bf16 A operand of the weighted sum, for which the warps split the latent columns (the K rows double as V). For MH = 1 two CTAs share
// an SM, so that the barriers of one hide under the other. The splits of a row form thread-block clusters of up to eight CTAs, which merge
// their sums through distributed shared memory: with one cluster per row the normalised bf16 result leaves (o_lat), else one fp32 partial
// (sum, maximum, denominator) per cluster.
constexpr int kLdBK = 32;
template <int MH>
struct LatentDecodeSmem {
  static constexpr int kRows = 16 * MH, kStages = MH == 1 ? 2 : 3;
  static constexpr int kPitchP = (kLdBK + 8) * 2, kPitchS = kLdBK + 4;  // bytes, floats
  int pitch, off_q, off_p, off_s, off_st, bytes;
  __host__ __device__ explicit LatentDecodeSmem(int CW) {
    pitch = (CW + 8) * 2;  // CW is a multiple of 16: an odd number of 16-byte units
    off_q = kStages * kLdBK * pitch;
    off_p = off_q + kRows * pitch;
    off_s = off_p + kRows * kPitchP;
    off_st = off_s + 2 * kRows * kPitchS * 4;
    bytes = off_st + (3 + 8) * kRows * 4;
  }
};

__device__ __forceinline__ uint32_t map_cluster(const void* p, uint32_t rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(smem_u32(p)), "r"(rank));
  return r;
}
__device__ __forceinline__ float ld_cluster_f1(const void* p, uint32_t rank) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(map_cluster(p, rank)) : "memory");
  return v;
}
__device__ __forceinline__ float4 ld_cluster_f4(const void* p, uint32_t rank) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(map_cluster(p, rank)) : "memory");
  return v;
}
__device__ __forceinline__ void cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

// NPW: 16-column blocks of the latent per warp; NQ: k16 steps of the query a warp keeps in registers
template <int NPW, int MH, int NQ>
__global__ void __launch_bounds__(256 * MH, (MH == 1 && NPW <= 4) ? 2 : 1) latent_decode_kernel(
    const __nv_bfloat16* __restrict__ q_lat, const __nv_bfloat16* __restrict__ c_cache, const __nv_bfloat16* __restrict__ r_cache, const int* __restrict__ bt,
    int bt_stride, const int* __restrict__ row_seq, const int* __restrict__ row_ctx, __nv_bfloat16* __restrict__ o_lat, float* __restrict__ part_o,
    float* __restrict__ part_ml, LatentGeom g, int page, float scale, const float* __restrict__ sink, int window, int cs) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(128) uint8_t lsm[];
  using L = LatentDecodeSmem<MH>;
  constexpr int BK = kLdBK, ROWS = L::kRows, NST = L::kStages, NT = 256 * MH, NW = 8 * MH;
  const int CW = g.Rp + g.drp;
  const L lay(CW);
  const uint32_t base_u = smem_u32(lsm);
  float* sS = reinterpret_cast<float*>(lsm + lay.off_s);
  float* sM = reinterpret_cast<float*>(lsm + lay.off_st);
  float* sL = sM + ROWS;
  float* sA = sL + ROWS;
  float* sW = sA + ROWS;  // [8][ROWS] merge weights
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, t4 = lane & 3;
  const int splits = gridDim.x, sp = blockIdx.x, i = blockIdx.y, h0 = blockIdx.z * ROWS;
  const int nh = min(ROWS, g.H - h0);
  const int ctx = row_ctx[i];
  const int* bt_row = bt + static_cast<long long>(row_seq ? row_seq[i] : i) * bt_stride;
  const int first_key = (window > 0 && ctx > window) ? ctx - window : 0;
  const int tl = first_key / BK, th = (ctx + BK - 1) / BK;
  const int per = (th - tl + splits - 1) / splits;
  const int t0 = tl + sp * per, nt = max(0, min(th, t0 + per) - t0);

  // NT / 32 threads per key row. A tile of 32 keys lies inside one page (page sizes are multiples of 32), so rows behind the context are
  // rows of the same page: finite values that the mask gives weight zero.
  const int cq = CW / 8, cc = g.Rp / 8;  // 16-byte chunks per row: whole, latent part
  const int lrow = tid / (NT / 32), lcol = tid % (NT / 32);
  // place of the next tile to load: page index, its id (fetched one tile ahead of use) and the tile's first row in it
  int pidx = t0 * BK / page, poff = t0 * BK - pidx * page, pg = nt > 0 ? bt_row[pidx] : 0;
  const uint32_t ldst = base_u + lrow * lay.pitch + lcol * 16, stage_bytes = BK * lay.pitch;
  const char* cbase = reinterpret_cast<const char*>(c_cache) + lcol * 16;
  const char* rbase = reinterpret_cast<const char*>(r_cache) + lcol * 16;
  const bool full_c = cc == 2 * NPW * (NT / 32);
  auto load_tile = [&](int j) {
    const uint32_t slot = static_cast<uint32_t>(pg * page + poff + lrow);  // (cache rows fit 31 bits: checked on the host)
    const uint32_t dst = ldst + (j % NST) * stage_bytes;
    const char* c = cbase + static_cast<unsigned long long>(slot) * static_cast<uint32_t>(g.Rp * 2);
    const char* r = rbase + static_cast<unsigned long long>(slot) * static_cast<uint32_t>(g.drp * 2);
    if (full_c) {
#pragma unroll
      for (int k = 0; k < 2 * NPW; ++k) cp_async16(dst + k * (NT / 2), c + k * (NT / 2), true);
    } else {
#pragma unroll
      for (int k = 0; k < 2 * NPW; ++k)
        if (lcol + k * (NT / 32) < cc) cp_async16(dst + k * (NT / 2), c + k * (NT / 2), true);
    }
    if (lcol < cq - cc) cp_async16(dst + cc * 16, r, true);
    if (cq - cc > NT / 32)
      for (int k = lcol + NT / 32; k < cq - cc; k += NT / 32) cp_async16(dst + (cc + k - lcol) * 16, r + (k - lcol) * 16, true);
    poff += BK;
    if (poff == page) {
      poff = 0;
      ++pidx;
      if (j + 1 < nt) pg = bt_row[pidx];
    }
  };
#pragma unroll
  for (int j = 0; j < NST - 1; ++j) {
    if (j < nt) load_tile(j);
    cp_async_commit();
  }
  for (int r = warp; r < ROWS; r += NW) {
    const __nv_bfloat16* src = q_lat + (static_cast<size_t>(i) * g.H + h0 + r) * CW;
    for (int k = lane; k < cq; k += 32)
      *reinterpret_cast<uint4*>(lsm + lay.off_q + r * lay.pitch + k * 16) = r < nh ? *reinterpret_cast<const uint4*>(src + k * 8) : make_uint4(0u, 0u, 0u, 0u);
  }
  __syncthreads();
  const int np = g.Rp / 16, nks = CW / 16;
  // score product of this warp: head group sm, keys skey .. + 7, k16 steps [ks0, ks0 + nk)
  const int sm = warp >> 3, skey = (warp & 3) * 8, skh = (warp >> 2) & 1;
  const int ks0 = skh * (nks / 2), nk = skh ? nks - nks / 2 : nks / 2;
  const uint32_t qa = base_u + lay.off_q + (sm * 16 + (lane & 15)) * lay.pitch + (lane >> 4) * 16 + ks0 * 32;
  // shared-memory addresses that only move with the stage
  const uint32_t ka0 = base_u + (skey + (lane & 7)) * lay.pitch + (lane >> 3) * 16 + ks0 * 32;  // two k16 steps per ldmatrix.x4
  const uint32_t va0 = base_u + ((lane & 7) + ((lane >> 3) & 1) * 8) * lay.pitch + (lane >> 4) * 16 + warp * 32;
  const uint32_t pa0 = base_u + lay.off_p + (lane & 15) * L::kPitchP + (lane >> 4) * 16;
  float* const sdst = sS + (skh * ROWS + sm * 16 + gq) * L::kPitchS + skey + 2 * t4;
  const bool all_blocks = np == NPW * NW;
  uint32_t soff = 0;  // byte offset of the current stage
  uint32_t qr[NQ > 0 ? NQ : 1][4];
#pragma unroll
  for (int k = 0; k < NQ; ++k)
    if (k < nk) ldmatrix_x4(qa + k * 32, qr[k]);
    else qr[k][0] = qr[k][1] = qr[k][2] = qr[k][3] = 0u;
  float o[MH][NPW][2][4];
#pragma unroll
  for (int m = 0; m < MH; ++m)
#pragma unroll
    for (int j = 0; j < NPW; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[m][j][0][e] = o[m][j][1][e] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;  // softmax state of head row tid / 16
  for (int it = 0; it < nt; ++it) {
    const int tile = t0 + it;
    cp_async_wait<NST - 2>();
    __syncthreads();  // the tile is here, and every warp is done with the stage of the previous one
    if (it + NST - 1 < nt) load_tile(it + NST - 1);
    cp_async_commit();
    {
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};  // two accumulators: half the dependent chain
      const uint32_t ka = ka0 + soff;
      const uint32_t ka2 = ka - ((lane >> 4) << 5);  // one step: ldmatrix.x2 (lanes 16.. repeat the addresses of lanes 0..)
      if (NQ > 0 && nk >= NQ) {
#pragma unroll
        for (int k = 0; k + 1 < NQ; k += 2) {
          uint32_t b[4];
          ldmatrix_x4(ka + k * 32, b);
          mma_16816(s0, qr[k], b[0], b[1]);
          mma_16816(s1, qr[k + 1], b[2], b[3]);
        }
        if constexpr (NQ % 2 == 1) {
          uint32_t b[2];
          ldmatrix_x2(ka2 + (NQ - 1) * 32, b);
          mma_16816(s0, qr[NQ - 1], b[0], b[1]);
        }
      } else {
#pragma unroll
        for (int k = 0; k < NQ; k += 2) {
          if (k + 1 < NQ && k + 1 < nk) {
            uint32_t b[4];
            ldmatrix_x4(ka + k * 32, b);
            mma_16816(s0, qr[k], b[0], b[1]);
            mma_16816(s1, qr[k + 1 < NQ ? k + 1 : k], b[2], b[3]);
          } else if (k < nk) {
            uint32_t b[2];
            ldmatrix_x2(ka2 + k * 32, b);
            mma_16816(s0, qr[k], b[0], b[1]);
          }
        }
      }
      int k = NQ;
      for (; k + 1 < nk; k += 2) {
        uint32_t a0[4], a1[4], b[4];
        ldmatrix_x4(ka + k * 32, b);
        ldmatrix_x4(qa + k * 32, a0);
        ldmatrix_x4(qa + k * 32 + 32, a1);
        mma_16816(s0, a0, b[0], b[1]);
        mma_16816(s1, a1, b[2], b[3]);
      }
      if (k < nk) {
        uint32_t a[4], b[2];
        ldmatrix_x4(qa + k * 32, a);
        ldmatrix_x2(ka2 + k * 32, b);
        mma_16816(s0, a, b[0], b[1]);
      }
      *reinterpret_cast<float2*>(sdst) = make_float2(s0[0] + s1[0], s0[1] + s1[1]);
      *reinterpret_cast<float2*>(sdst + 8 * L::kPitchS) = make_float2(s0[2] + s1[2], s0[3] + s1[3]);
    }
    __syncthreads();
    // ---- online softmax: 16 threads per head row, two neighbouring keys each. The running maximum (the same in a row's threads) follows only
    // when a score has outgrown it by more than 8: a stale one costs head-room (weights up to e^8), a new one a reduction and a pass over the
    // accumulators. The denominator stays a partial sum per thread until the end.
    bool grown;
    {
      const int r = tid >> 4, c0 = (tid & 15) * 2, key = tile * BK + c0;
      const float2 a = *reinterpret_cast<const float2*>(sS + r * L::kPitchS + c0), b = *reinterpret_cast<const float2*>(sS + (ROWS + r) * L::kPitchS + c0);
      const float v0 = (key < ctx && key >= first_key) ? (a.x + b.x) * scale : -INFINITY;
      const float v1 = (key + 1 < ctx && key + 1 >= first_key) ? (a.y + b.y) * scale : -INFINITY;
      float mx = fmaxf(v0, v1), alpha = 1.f;
      grown = __any_sync(0xffffffffu, mx > m_run + 8.f);
      if (grown) {  // warp-uniform
#pragma unroll
        for (int off = 1; off < 16; off <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        if (mx > m_run + 8.f) {
          alpha = __expf(m_run - mx);  // (exp of -infinity: 0)
          l_run *= alpha;
          m_run = mx;
        }
      }
      if ((tid & 15) == 0) sA[r] = alpha;
      const float w0 = v0 == -INFINITY ? 0.f : __expf(v0 - m_run), w1 = v1 == -INFINITY ? 0.f : __expf(v1 - m_run);
      *reinterpret_cast<uint32_t*>(lsm + lay.off_p + r * L::kPitchP + c0 * 2) = pack_bf162(w0, w1);
      l_run += w0 + w1;
    }
    // ---- weighted sum: warp w owns the 16-column blocks w, w + NW, ...
    if (__syncthreads_or(grown)) {
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
    }
    auto weighted = [&](auto whole) {
#pragma unroll
      for (int ks = 0; ks < BK / 16; ++ks) {
        uint32_t a[MH][4];
#pragma unroll
        for (int m = 0; m < MH; ++m) ldmatrix_x4(pa0 + m * 16 * L::kPitchP + ks * 32, a[m]);
        const uint32_t va = va0 + soff + ks * 16 * lay.pitch;
#pragma unroll
        for (int j = 0; j < NPW; ++j) {
          if (decltype(whole)::value || warp + NW * j < np) {  // warp-uniform
            uint32_t b[4];
            ldmatrix_x4_trans(va + j * NW * 32, b);
#pragma unroll
            for (int m = 0; m < MH; ++m) {
              mma_16816(o[m][j][0], a[m], b[0], b[1]);
              mma_16816(o[m][j][1], a[m], b[2], b[3]);
            }
          }
        }
      }
    };
    if (all_blocks) weighted(std::true_type());
    else weighted(std::false_type());
    soff = soff == (NST - 1) * stage_bytes ? 0 : soff + stage_bytes;
  }
  cp_async_wait<0>();
#pragma unroll
  for (int off = 1; off < 16; off <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, off);
  if ((tid & 15) == 0) {
    sM[tid >> 4] = m_run;
    sL[tid >> 4] = l_run;
  }
  __syncthreads();
  // ---- merge of the cluster's sums
  const int outer = splits / cs, op = sp / cs, PO = g.Rp + 4;
  float* sO = reinterpret_cast<float*>(lsm);  // [ROWS][PO] (aliases the stages)
#pragma unroll
  for (int m = 0; m < MH; ++m)
#pragma unroll
    for (int j = 0; j < NPW; ++j) {
      const int blk = warp + NW * j;
      if (blk >= np) continue;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        float* d = sO + (m * 16 + gq) * PO + blk * 16 + n * 8 + 2 * t4;
        *reinterpret_cast<float2*>(d) = make_float2(o[m][j][n][0], o[m][j][n][1]);
        *reinterpret_cast<float2*>(d + 8 * PO) = make_float2(o[m][j][n][2], o[m][j][n][3]);
      }
    }
  const int rank = sp % cs;
  if (cs > 1) cluster_barrier();
  else __syncthreads();
  if (tid < ROWS) {
    float m = -INFINITY, ms[8], l = 0.f;
#pragma unroll
    for (int s = 0; s < 8; ++s)
      if (s < cs) {
        ms[s] = cs > 1 ? ld_cluster_f1(sM + tid, s) : sM[tid];
        m = fmaxf(m, ms[s]);
      }
#pragma unroll
    for (int s = 0; s < 8; ++s)
      if (s < cs) {
        ms[s] = ms[s] == -INFINITY ? 0.f : __expf(ms[s] - m);
        l += ms[s] * (cs > 1 ? ld_cluster_f1(sL + tid, s) : sL[tid]);
      }
    if (sink != nullptr && outer == 1 && tid < nh) l += __expf(sink[h0 + tid] - m);  // (m is finite: a row sees its own key)
    const float inv = outer > 1 ? 1.f : (l > 0.f ? 1.f / l : 0.f);
#pragma unroll
    for (int s = 0; s < 8; ++s)
      if (s < cs) sW[s * ROWS + tid] = ms[s] * inv;
    if (outer > 1 && rank == 0 && tid < nh) {
      float* ml = part_ml + ((static_cast<size_t>(i) * g.H + h0 + tid) * outer + op) * 2;
      ml[0] = m;
      ml[1] = l;
    }
  }
  __syncthreads();
  const int quads = g.Rp / 4;
  for (int e = rank * NT + tid; e < nh * quads; e += cs * NT) {
    const int r = e / quads, k = (e % quads) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int s = 0; s < 8; ++s)
      if (s < cs) {
        const float w = sW[s * ROWS + r];
        const float4 a = cs > 1 ? ld_cluster_f4(sO + r * PO + k, s) : *reinterpret_cast<const float4*>(sO + r * PO + k);
        v.x += w * a.x;
        v.y += w * a.y;
        v.z += w * a.z;
        v.w += w * a.w;
      }
    const size_t head = static_cast<size_t>(i) * g.H + h0 + r;
    if (outer > 1) *reinterpret_cast<float4*>(part_o + (head * outer + op) * g.Rp + k) = v;
    else *reinterpret_cast<uint2*>(o_lat + head * g.Rp + k) = make_uint2(pack_bf162(v.x, v.y), pack_bf162(v.z, v.w));
  }
  if (cs > 1) cluster_barrier();  // nobody leaves while a peer still reads its shared memory
}

template <int NPW, int MH, int NQ>
static int launch_latent_decode_t(const LatentDecodeArgs& a, const LatentGeom& g, cudaStream_t st) {
  const LatentDecodeSmem<MH> L(g.Rp + g.drp);
  if (L.bytes > 227 * 1024) return 1;
  static PerDeviceOnce attr_once;
  if (attr_once.first()) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<NPW, MH, NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) throw std::runtime_error(std::string("latent decode attention: cudaFuncSetAttribute: ") + cudaGetErrorString(e));
  }
  const int cs = latent_cluster_size(a.splits);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(a.splits, a.rows, (g.H + 16 * MH - 1) / (16 * MH));
  cfg.blockDim = dim3(256 * MH);
  cfg.dynamicSmemBytes = static_cast<size_t>(L.bytes);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = g_pdl_enabled ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = cs;
  attr[1].val.clusterDim.y = attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = cs > 1 ? 2 : 1;
  cudaError_t e = cudaLaunchKernelEx(&cfg, latent_decode_kernel<NPW, MH, NQ>, static_cast<const __nv_bfloat16*>(a.q_lat),
                                     static_cast<const __nv_bfloat16*>(a.c_cache), static_cast<const __nv_bfloat16*>(a.r_cache), a.bt, a.bt_stride, a.row_seq,
                                     a.row_ctx, static_cast<__nv_bfloat16*>(a.o_lat), a.part_o, a.part_ml, g, a.page, a.scale, a.sink, a.window, cs);
  if (e != cudaSuccess) throw std::runtime_error(std::string("latent decode attention launch: ") + cudaGetErrorString(e));
  return 0;
}

int launch_latent_decode(const LatentDecodeArgs& a, const LatentGeom& g, cudaStream_t st) {
  if (a.rows == 0) return 0;
  if (a.page % kLdBK != 0 || a.splits % latent_cluster_size(a.splits) != 0) return 2;
  const bool two = g.H > 16 && LatentDecodeSmem<2>(g.Rp + g.drp).bytes <= 227 * 1024 && g_latent_head_groups != 1;
  if (g.Rp <= 128) return two ? launch_latent_decode_t<1, 2, 6>(a, g, st) : launch_latent_decode_t<1, 1, 6>(a, g, st);
  if (g.Rp <= 256) return two ? launch_latent_decode_t<1, 2, 9>(a, g, st) : launch_latent_decode_t<2, 1, 9>(a, g, st);
  if (g.Rp <= 512) return two ? launch_latent_decode_t<2, 2, 12>(a, g, st) : launch_latent_decode_t<4, 1, 12>(a, g, st);
  if (g.Rp <= 1024) return launch_latent_decode_t<8, 1, 0>(a, g, st);
  return 1;
}

// ------------------------------------------------------------------------------------------------ value weights, gate (and merge)
// out[row][h * dv + v] = sigmoid(gate) * sum_r wuv[h][v][r] * o_lat[r]. wuv [H][dv8][Kp]. grid (H, row tiles of 16, blocks of 32 value
// columns), 4 warps x 8 columns, operands read as in latent_absorb_kernel. MERGE: o_lat is first summed from `outer` partials per row and head
// into shared memory (few rows: a batch that needs more splits than one cluster).
template <bool MERGE>
__global__ void __launch_bounds__(128) latent_expand_kernel(const __nv_bfloat16* __restrict__ o_lat, const float* __restrict__ part_o,
                                                            const float* __restrict__ part_ml, int outer, const int* __restrict__ row_idx, int rows,
                                                            const __nv_bfloat16* __restrict__ wuv, const __nv_bfloat16* __restrict__ p, long long ld,
                                                            __nv_bfloat16* __restrict__ out, int out_pitch, LatentGeom g,
                                                            const float* __restrict__ sink) {
  const int h = blockIdx.x, i0 = blockIdx.y * 16, n0 = blockIdx.z * 32, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, c = lane & 3;
  const int dv8 = (g.dv + 7) & ~7;
  {  // weights do not depend on the kernel in front: towards L2 while it finishes
    const char* w0 = reinterpret_cast<const char*>(wuv + (static_cast<size_t>(h) * dv8 + n0) * g.Kp);
    for (int o = tid * 128; o < min(32, dv8 - n0) * g.Kp * 2; o += 128 * 128) prefetch_l2(w0 + o);
  }
  pdl_wait();
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t esm[];
  const int pitch = g.Kp + 8;
  __nv_bfloat16* sO = reinterpret_cast<__nv_bfloat16*>(esm);                 // [16][pitch]
  float* sW = reinterpret_cast<float*>(esm + 16 * pitch * 2);                // [16][outer] weights, already divided by the row's sum
  const int nr = min(16, rows - i0);
  if (MERGE) {
    if (tid < nr) {
      const float* ml = part_ml + (static_cast<size_t>(i0 + tid) * g.H + h) * outer * 2;
      float m = -INFINITY;
      for (int s = 0; s < outer; ++s) m = fmaxf(m, ml[2 * s]);
      float den = sink != nullptr ? __expf(sink[h] - m) : 0.f;
      for (int s = 0; s < outer; ++s) {
        const float w = ml[2 * s] == -INFINITY ? 0.f : __expf(ml[2 * s] - m);
        sW[tid * outer + s] = w;
        den += w * ml[2 * s + 1];
      }
      const float inv = den > 0.f ? 1.f / den : 0.f;
      for (int s = 0; s < outer; ++s) sW[tid * outer + s] *= inv;
    }
    __syncthreads();
    const int quads = g.Kp / 4;
    for (int e = tid; e < 16 * quads; e += 128) {
      const int r = e / quads, k = (e % quads) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (r < nr && k < g.Rp) {
        const float* src = part_o + (static_cast<size_t>(i0 + r) * g.H + h) * outer * g.Rp + k;
#pragma unroll 4
        for (int s = 0; s < outer; ++s) {
          const float w = sW[r * outer + s];
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
  }
  const int nb = n0 + warp * 8;
  if (nb >= dv8) return;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  const bool va = gq < nr, vb = gq + 8 < nr;
  const __nv_bfloat16* ga = o_lat + (static_cast<size_t>(i0 + (va ? gq : 0)) * g.H + h) * g.Rp + c * 8;
  const __nv_bfloat16* gb = o_lat + (static_cast<size_t>(i0 + (vb ? gq + 8 : 0)) * g.H + h) * g.Rp + c * 8;
  const __nv_bfloat16* xa = sO + gq * pitch + c * 8;
  const __nv_bfloat16* w = wuv + (static_cast<size_t>(h) * dv8 + nb + gq) * g.Kp + c * 8;
  // the epilogue's gate values travel under the product
  float gate[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
  long long orow[2];
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int i = gq + half * 8;
    orow[half] = i < nr ? (row_idx ? row_idx[i0 + i] : i0 + i) : 0;
#pragma unroll
    for (int e = 0; e < 2; ++e)
      if (g.off_g >= 0 && i < nr && nb + 2 * c + e < g.dv) gate[half][e] = bf2f(p[orow[half] * ld + g.off_g + h * g.dv + nb + 2 * c + e]);
  }
  float acc[4] = {0.f, 0.f, 0.f, 0.f}, acc2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
  for (int k0 = 0; k0 < g.Kp; k0 += 32) {
    const uint4 b = __ldg(reinterpret_cast<const uint4*>(w + k0));
    uint4 x0, x1;
    if (MERGE) {
      x0 = *reinterpret_cast<const uint4*>(xa + k0);
      x1 = *reinterpret_cast<const uint4*>(xa + 8 * pitch + k0);
    } else {
      const bool in = k0 + c * 8 < g.Rp;
      x0 = va && in ? *reinterpret_cast<const uint4*>(ga + k0) : zero;
      x1 = vb && in ? *reinterpret_cast<const uint4*>(gb + k0) : zero;
    }
    const uint32_t a0[4] = {x0.x, x1.x, x0.y, x1.y}, a1[4] = {x0.z, x1.z, x0.w, x1.w};
    mma_16816(acc, a0, b.x, b.y);
    mma_16816(acc2, a1, b.z, b.w);
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    if (gq + half * 8 >= nr) continue;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int v = nb + 2 * c + e;
      if (v >= g.dv) continue;
      float y = acc[half * 2 + e] + acc2[half * 2 + e];
      if (g.off_g >= 0) y /= 1.f + __expf(-gate[half][e]);
      out[orow[half] * out_pitch + h * g.dv + v] = f2bf(y);
    }
  }
}

void launch_latent_expand(const LatentDecodeArgs& a, const int* row_idx, const void* wuv, const void* p, long long ld, void* out, int out_pitch,
                          const LatentGeom& g, cudaStream_t st) {
  if (a.rows == 0) return;
  const int outer = a.splits / latent_cluster_size(a.splits);
  const size_t smem = outer > 1 ? static_cast<size_t>(16) * (g.Kp + 8) * 2 + static_cast<size_t>(16) * outer * 4 : 0;
  if (smem > 48 * 1024) throw std::runtime_error("latent expand: too many splits or latent columns");
  const dim3 grid(g.H, (a.rows + 15) / 16, (g.dv + 31) / 32);
  const auto *ol = static_cast<const __nv_bfloat16*>(a.o_lat), *w = static_cast<const __nv_bfloat16*>(wuv), *pp = static_cast<const __nv_bfloat16*>(p);
  auto* o = static_cast<__nv_bfloat16*>(out);
  if (outer > 1) launch_pdl(latent_expand_kernel<true>, grid, dim3(128), smem, st, ol, a.part_o, a.part_ml, outer, row_idx, a.rows, w, pp, ld, o, out_pitch, g, a.sink);
  else launch_pdl(latent_expand_kernel<false>, grid, dim3(128), smem, st, ol, a.part_o, a.part_ml, outer, row_idx, a.rows, w, pp, ld, o, out_pitch, g, a.sink);
}

// ------------------------------------------------------------------------------------------------ 32-bit form
// Whole mixer core of one (row, head) in fp32: absorbed query, online softmax over the cached keys, value weights, gate. grid (rows, H).
__global__ void __launch_bounds__(256) latent_rows_f32_kernel(const float* __restrict__ p, long long ld, const int* __restrict__ row_idx,
                                                              const int* __restrict__ row_seq, const int* __restrict__ row_ctx, const float* __restrict__ wuk,
                                                              const float* __restrict__ wuv, const float* __restrict__ c_cache,
                                                              const float* __restrict__ r_cache, const int* __restrict__ bt, int bt_stride,
                                                              float* __restrict__ out, int out_pitch, LatentGeom g, int dn_pad, int page, float scale,
                                                              int window, const float* __restrict__ sink) {
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
  if (sink != nullptr) l_run += expf(sink[h] - m_run);  // (a row sees its own key: m_run is finite)
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
                           const LatentGeom& g, int page, float scale, int window, const float* sink, cudaStream_t st) {
  if (rows == 0) return 0;
  const size_t smem = static_cast<size_t>(2 * g.Rp + g.drp + 64) * 4;
  if (smem > 46 * 1024 || g.H > 65535) return 1;
  launch_pdl(latent_rows_f32_kernel, dim3(rows, g.H), dim3(256), smem, st, p, ld, row_idx, row_seq, row_ctx, wuk, wuv, c_cache, r_cache, bt, bt_stride, out,
             out_pitch, g, (g.dn + 63) / 64 * 64, page, scale, window, sink);
  return 0;
}

// ------------------------------------------------------------------------------------------------ fp32 projection
// out = x W^T (+ bias), true fp32 FMA. 64 x 64 tiles, 256 threads with 4 x 4 accumulators, K in steps of 16.
__global__ void __launch_bounds__(256) linear_f32_kernel(const float* __restrict__ x, int ldx, const float* __restrict__ w, const float* __restrict__ bias,
                                                         float* __restrict__ out, int ldo, int M, int N, int K, const int4* __restrict__ items) {
  pdl_wait();
  pdl_trigger();
  __shared__ float sx[16][68], sw[16][68];
  int m0 = blockIdx.y * 64;
  if (items != nullptr) {  // grouped: (expert, first row, end row) per 64-row item, w stacks the experts
    const int4 it = items[blockIdx.y];
    if (it.x < 0) return;
    w += static_cast<size_t>(it.x) * N * K;
    m0 = it.y;
    M = min(it.z, it.y + 64);
  }
  const int n0 = blockIdx.x * 64, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
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
  launch_pdl(linear_f32_kernel, dim3((N + 63) / 64, gy), dim3(256), 0, st, x, ldx, w, bias, out, ldo, M, N, K, static_cast<const int4*>(nullptr));
}
void launch_grouped_linear_f32(const float* x, int ldx, const float* w, float* out, int ldo, const int* items, int n_items, int N, int K, cudaStream_t st) {
  if (n_items == 0 || N == 0) return;
  launch_pdl(linear_f32_kernel, dim3((N + 63) / 64, static_cast<unsigned>(n_items)), dim3(256), 0, st, x, ldx, w, static_cast<const float*>(nullptr), out, ldo, 0,
             N, K, reinterpret_cast<const int4*>(items));
}

}  // namespace dlv
