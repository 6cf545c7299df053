// Latent attention over a paged latent cache, forward only.
//
// A cache row holds [latent c (rank) | rotated key part (rot)] of one token, pitch ldc elements; the
// rows of page p are p * page_size ... .  Per head the score of query q and a cached token is
//     (q_n . W_uk c + q_r . k_r) * scale = ((W_uk^T q_n) . c + q_r . k_r) * scale
// and the head's output is W_uv (sum_j p_j c_j): with W_uk and W_uv moved to the query side every head
// attends to the same row, so decoding reads the cache once for all heads and expands nothing.
//
//   latent_prepare_kernel   interleaved rotation of q (in place) and of the shared key part, RMS norm of
//                           the latent; row -> cache page (and, for prompts, -> packed rows)
//   latent_absorb_kernel    q_lat = W_uk^T q_n            latent_expand_kernel   o = W_uv o_lat
//   latent_attn_any_kernel  attention of any query against its sequence's pages, any sizes, fp32 math
//   latent_decode_kernel    bf16 decode on mma.sync tiles, split over the keys, partials merged by
//                           latent_combine_kernel
#include "host_utils.h"
#include "serve_common.cuh"

namespace ob {

// ------------------------------------------------------------------------------------------------ prepare
struct LatentPrepArgs {
  void* proj;              // T [N, ldp]: q heads (dim + rot each) at 0, [c | k_r] at dkv_off (if dkv_off >= 0)
  const int* pos;          // [N] position in the sequence, -1: no token
  const int* row;          // [N] cache row of the token, -1: none
  const float* cos_t;      // [positions, pairs]
  const float* sin_t;
  const void* norm_w;      // T [rank]
  void* cache;             // T [rows, ldc]
  void* packed;            // T [N, ldc] or null
  long long ldp, ldc, cache_rows;
  int dkv_off, H, dim, rot, rank, pairs, table_rows;
  float eps;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_prepare_kernel(const LatentPrepArgs p) {
  __shared__ float red[33];
  const int n = blockIdx.x;
  const int pos = p.pos[n];
  if (pos < 0 || pos >= p.table_rows) {
    if (pos != -1 && threadIdx.x == 0) atomicCAS(p.status, 0, OB_ERR_BAD_ARG | (n << 8));
    return;
  }
  T* q = (T*)p.proj + (long long)n * p.ldp;
  const float *ct = p.cos_t + (long long)pos * p.pairs, *sn = p.sin_t + (long long)pos * p.pairs;
  const int hd = p.dim + p.rot;
  for (int i = threadIdx.x; i < p.H * p.pairs; i += 256) {
    const int h = i / p.pairs, j = i - h * p.pairs;
    T* x = q + h * hd + p.dim + 2 * j;
    const float u = to_f(x[0]), v = to_f(x[1]), c = ct[j], s = sn[j];
    x[0] = from_f<T>(u * c - v * s);
    x[1] = from_f<T>(v * c + u * s);
  }
  if (p.dkv_off < 0) return;
  const T* d = q + p.dkv_off;
  const int row = p.row[n];
  if (row < 0 || row >= p.cache_rows) {
    if (threadIdx.x == 0) atomicCAS(p.status, 0, OB_ERR_BAD_ARG | (n << 8));
    return;
  }
  T* dst = (T*)p.cache + (long long)row * p.ldc;
  T* dst2 = p.packed ? (T*)p.packed + (long long)n * p.ldc : nullptr;
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.rank; i += 256) {
    const float v = to_f(d[i]);
    ss += v * v;
  }
  const float rstd = 1.f / sqrtf(block_sum<256>(ss, red) / (float)p.rank + p.eps);
  for (int i = threadIdx.x; i < p.rank; i += 256) {
    const T v = from_f<T>(to_f(d[i]) * rstd * to_f(((const T*)p.norm_w)[i]));
    dst[i] = v;
    if (dst2) dst2[i] = v;
  }
  const T* r = d + p.rank;
  for (int i = threadIdx.x; i < p.rot; i += 256) {
    T v = r[i];
    if ((i >> 1) < p.pairs) {
      const int j = i >> 1;
      const float u = to_f(r[2 * j]), w = to_f(r[2 * j + 1]);
      v = from_f<T>((i & 1) ? w * ct[j] + u * sn[j] : u * ct[j] - w * sn[j]);
    }
    dst[p.rank + i] = v;
    if (dst2) dst2[p.rank + i] = v;
  }
}

// ------------------------------------------------------------------------------------------------ absorb / expand
// q_lat[n, h, r] = sum_d q[n, h, d] W_uk[h*dim + d, r]; CTA = (128 latent columns, head, 8 queries):
// a lane owns 4 columns, the four warps split the sum over d.  VEC: rank % 4 == 0.
template <typename T, typename O, bool VEC>
__global__ void __launch_bounds__(128) latent_absorb_kernel(const T* __restrict__ q, long long ldq, int head_stride,
                                                            const T* __restrict__ uk, O* __restrict__ out, int N, int H,
                                                            int dim, int rank) {
  extern __shared__ __align__(16) float sq[];   // [dim][8]
  __shared__ float part[4][8][128];
  const int h = blockIdx.y, n0 = blockIdx.z * 8, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int r = blockIdx.x * 128 + lane * 4, nn = min(8, N - n0);
  for (int i = threadIdx.x; i < 8 * dim; i += 128) {
    const int t = i / dim, d = i - t * dim;
    sq[d * 8 + t] = t < nn ? to_f(q[(long long)(n0 + t) * ldq + (long long)h * head_stride + d]) : 0.f;
  }
  __syncthreads();
  const T* w = uk + (long long)h * dim * rank + r;
  float acc[8][4] = {};
  if (r < rank) {
#pragma unroll 8
    for (int d = warp; d < dim; d += 4) {
      const T* wd = w + (long long)d * rank;
      float x[4];
      if (VEC) {
        *reinterpret_cast<float4*>(x) = load4(wd);
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c) x[c] = r + c < rank ? to_f(wd[c]) : 0.f;
      }
      const float4 a = load4(sq + d * 8), b = load4(sq + d * 8 + 4);
      const float qq[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
      for (int t = 0; t < 8; ++t)
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[t][c] = fmaf(x[c], qq[t], acc[t][c]);
    }
  }
#pragma unroll
  for (int t = 0; t < 8; ++t) store4(&part[warp][t][lane * 4], make_float4(acc[t][0], acc[t][1], acc[t][2], acc[t][3]));
  __syncthreads();
  const int rc = blockIdx.x * 128 + threadIdx.x;
  if (rc >= rank) return;
  for (int t = 0; t < nn; ++t)
    out[((long long)(n0 + t) * H + h) * rank + rc] =
        from_f<O>((part[0][t][threadIdx.x] + part[1][t][threadIdx.x]) + (part[2][t][threadIdx.x] + part[3][t][threadIdx.x]));
}

// o[n, h, v] = sum_r o_lat[n, h, r] W_uv[h*vdim + v, r]; CTA = (32 value rows, head, 8 queries), four rows
// per warp.  VEC: rank % 4 == 0.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) latent_expand_kernel(const float* __restrict__ ol, const T* __restrict__ uv,
                                                            T* __restrict__ out, int N, int H, int vdim, int rank) {
  extern __shared__ __align__(16) float so[];   // [8][rank padded to 4]
  const int h = blockIdx.y, n0 = blockIdx.z * 8, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nn = min(8, N - n0), ld = (rank + 3) & ~3;
  for (int i = threadIdx.x; i < 8 * ld; i += 256) {
    const int t = i / ld, r = i - t * ld;
    so[i] = t < nn && r < rank ? ol[((long long)(n0 + t) * H + h) * rank + r] : 0.f;
  }
  __syncthreads();
  const int v0 = blockIdx.x * 32 + warp * 4;
  if (v0 >= vdim) return;
  float acc[4][8] = {};
#pragma unroll 2
  for (int r = lane * 4; r < rank; r += 128) {
    float x[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const T* w = uv + ((long long)h * vdim + min(v0 + j, vdim - 1)) * rank + r;
      if (VEC) {
        *reinterpret_cast<float4*>(x[j]) = load4(w);
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c) x[j][c] = r + c < rank ? to_f(w[c]) : 0.f;
      }
    }
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      const float4 o = load4(so + t * ld + r);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        acc[j][t] = fmaf(x[j][3], o.w, fmaf(x[j][2], o.z, fmaf(x[j][1], o.y, fmaf(x[j][0], o.x, acc[j][t]))));
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int t = 0; t < 8; ++t) {
      const float s = warp_sum(acc[j][t]);
      if (lane == 0 && t < nn && v0 + j < vdim) out[((long long)(n0 + t) * H + h) * vdim + v0 + j] = from_f<T>(s);
    }
}

// ------------------------------------------------------------------------------------------------ any-size attention
struct LatentAttnArgs {
  const void* q_lat;       // fp32 [N, H, rank]
  const void* q_rot;       // T, q_rot + n*ldq + h*head_stride: rot values
  const void* cache;       // T [rows, ldc]
  const int* seq;          // [N]
  const int* len;          // [N] visible tokens of the query's sequence, 0: no query
  const int* table;        // [B, max_blocks]
  float* out;              // [N, H, rank]
  long long ldq, ldc;
  int head_stride, H, rank, rot, max_blocks, page_size;
  float scale;
};

constexpr int kAnyKeys = 64;

template <typename T>
__global__ void __launch_bounds__(128) latent_attn_any_kernel(const LatentAttnArgs p) {
  extern __shared__ float sm[];     // q[rank + rot], o[rank], s[kAnyKeys]; then rows[kAnyKeys]
  const int n = blockIdx.y, h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int F = p.rank + p.rot;
  float *q = sm, *o = sm + F, *sc = o + p.rank;
  int* rows = (int*)(sc + kAnyKeys);
  const int len = p.len[n];
  float* out = p.out + ((long long)n * p.H + h) * p.rank;
  for (int i = tid; i < p.rank; i += 128) {
    q[i] = ((const float*)p.q_lat)[((long long)n * p.H + h) * p.rank + i];
    o[i] = 0.f;
    if (len <= 0) out[i] = 0.f;
  }
  if (len <= 0) return;
  const T* qr = (const T*)p.q_rot + (long long)n * p.ldq + (long long)h * p.head_stride;
  for (int i = tid; i < p.rot; i += 128) q[p.rank + i] = to_f(qr[i]);
  const int* bt = p.table + (long long)p.seq[n] * p.max_blocks;
  const T* cache = (const T*)p.cache;
  float m = -INFINITY, l = 0.f;
  for (int k0 = 0; k0 < len; k0 += kAnyKeys) {
    const int nk = min(kAnyKeys, len - k0);
    __syncthreads();
    if (tid < nk) {
      const int k = k0 + tid;
      rows[tid] = bt[k / p.page_size] * p.page_size + k % p.page_size;
    }
    __syncthreads();
    for (int k = warp; k < nk; k += 4) {
      const T* r = cache + (long long)rows[k] * p.ldc;
      float d = 0.f;
      for (int i = lane; i < F; i += 32) d = fmaf(q[i], to_f(r[i]), d);
      d = warp_sum(d);
      if (lane == 0) sc[k] = d * p.scale;
    }
    __syncthreads();
    float mx = m;
    for (int k = 0; k < nk; ++k) mx = fmaxf(mx, sc[k]);
    const float a = expf(m - mx);       // 0 on the first tile
    l *= a;
    m = mx;
    for (int k = 0; k < nk; ++k) l += expf(sc[k] - m);
    __syncthreads();
    if (tid < nk) sc[tid] = expf(sc[tid] - m);
    __syncthreads();
    for (int i = tid; i < p.rank; i += 128) {
      float acc = o[i] * a;
      for (int k = 0; k < nk; ++k) acc = fmaf(sc[k], to_f(cache[(long long)rows[k] * p.ldc + i]), acc);
      o[i] = acc;
    }
  }
  for (int i = tid; i < p.rank; i += 128) out[i] = o[i] / l;
}

// ------------------------------------------------------------------------------------------------ bf16 decode
__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src));
}

struct LatentDecodeArgs {
  const bf16* q_lat;       // [B, H, rank]
  const bf16* q_rot;       // q_rot + b*ldq + h*head_stride
  const bf16* cache;       // [rows, ldc]
  const int* len;          // [B]
  const int* table;        // [B, max_blocks]
  float* part_o;           // [B, splits, H, rank]
  float* part_ml;          // [B, splits, H, 2] (running maximum in log2 units, sum)
  long long ldq, ldc;
  int head_stride, H, rank, rot, max_blocks, page_size, splits;
  float scale_log2;
};

constexpr int kDecKeys = 64;      // keys per tile

// CTA = (key split, block of 16*MT heads, sequence), 8 warps.  Shared memory: Q [16*MT][LD],
// two key tiles [64][LD], P [16*MT][72] (bf16), LD = rank_pad + rot_pad + 8 (rank padded to a multiple
// of 64, rot to one of 16; the padding holds zeros).  Scores: a warp owns one 16-head tile and 8 * MT
// keys.  Output: warp w owns rank_pad / 8 = 8 * NT latent columns for all heads of the block, in registers.
template <int MT, int NT>
__global__ void __launch_bounds__(256) latent_decode_kernel(const LatentDecodeArgs p) {
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int HB = 16 * MT;
  constexpr int RP = 64 * NT;
  constexpr int LDP = kDecKeys + 8;
  constexpr int KG = 8 / MT;                  // key groups of a tile (warps per head tile)
  const int rotp = (p.rot + 15) & ~15;
  const int LD = RP + rotp + 8;
  bf16* sQ = (bf16*)smem;
  bf16* sK = sQ + HB * LD;                    // two tiles
  bf16* sP = sK + 2 * kDecKeys * LD;
  float* s_max = (float*)(sP + HB * LDP);     // [KG][HB]
  float* s_sum = s_max + KG * HB;             // [KG][HB]
  const int b = blockIdx.z, h0 = blockIdx.y * HB, sp = blockIdx.x;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int len = p.len[b];
  // whole tiles are handed out to the splits
  const int tiles = (len + kDecKeys - 1) / kDecKeys;
  const int per = (tiles + p.splits - 1) / p.splits;
  const int t_lo = min(sp * per, tiles), t_hi = min(t_lo + per, tiles);
  float* po = p.part_o + ((long long)b * p.splits + sp) * p.H * p.rank;
  float* pml = p.part_ml + ((long long)b * p.splits + sp) * p.H * 2;
  if (t_lo >= t_hi) {
    for (int i = tid; i < HB && h0 + i < p.H; i += 256) {
      pml[(h0 + i) * 2] = -INFINITY;
      pml[(h0 + i) * 2 + 1] = 0.f;
    }
    return;
  }
  // zero the padding columns once (both tiles and Q), then fill
  const int pad_lo = p.rank, pad_hi = RP, rpad_lo = RP + p.rot, rpad_hi = LD;
  for (int r = warp; r < HB + 2 * kDecKeys; r += 8) {
    bf16* x = sQ + (long long)r * LD;          // Q rows and key rows are contiguous
    for (int c = pad_lo + lane; c < pad_hi; c += 32) x[c] = __float2bfloat16(0.f);
    for (int c = rpad_lo + lane; c < rpad_hi; c += 32) x[c] = __float2bfloat16(0.f);
  }
  const int* bt = p.table + (long long)b * p.max_blocks;
  const int cv = p.rank >> 3, rv = p.rot >> 3;      // 16-byte vectors per row
  // lane l (mod 8) knows the cache row of key warp + 8 l of a tile; looked up one tile ahead
  auto find_rows = [&](int t) {
    const int k = min(t * kDecKeys + warp + 8 * (lane & 7), len - 1);   // past the end: the last row again (masked below)
    return bt[k / p.page_size] * p.page_size + k % p.page_size;
  };
  int rows = find_rows(t_lo);
  auto load_tile = [&](int t) {
    bf16* dst = sK + (t & 1) * kDecKeys * LD;
    const int now = rows;
    rows = find_rows(min(t + 1, t_hi - 1));
#pragma unroll
    for (int i = 0; i < kDecKeys / 8; ++i) {
      const bf16* src = p.cache + (long long)__shfl_sync(0xffffffffu, now, i) * p.ldc;
      const uint32_t d = smem_u32(dst + (warp + 8 * i) * LD);
      for (int v = lane; v < cv + rv; v += 32)
        cp16(d + (v < cv ? v * 16 : (RP + (v - cv) * 8) * 2), src + v * 8);
    }
    asm volatile("cp.async.commit_group;");
  };
  load_tile(t_lo);
  for (int i = tid; i < HB * (cv + rv); i += 256) {
    const int r = i / (cv + rv), v = i - r * (cv + rv), h = h0 + r;
    uint4 u = make_uint4(0, 0, 0, 0);
    if (h < p.H)
      u = v < cv ? *reinterpret_cast<const uint4*>(p.q_lat + ((long long)b * p.H + h) * p.rank + v * 8)
                 : *reinterpret_cast<const uint4*>(p.q_rot + (long long)b * p.ldq + (long long)h * p.head_stride + (v - cv) * 8);
    *reinterpret_cast<uint4*>(sQ + r * LD + (v < cv ? v * 8 : RP + (v - cv) * 8)) = u;
  }
  float o[MT][NT][4];
  float m[MT][2], l[2] = {0.f, 0.f};
  const int mt = warp % MT, kgrp = warp / MT;  // this warp's head tile and key group in the score phase
#pragma unroll
  for (int i = 0; i < MT; ++i) {
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) o[i][j][c] = 0.f;
    m[i][0] = m[i][1] = -INFINITY;
  }
  const int ksteps = (RP + rotp) >> 4;
  const int g = lane >> 2, tq = lane & 3;
  for (int t = t_lo; t < t_hi; ++t) {
    if (t + 1 < t_hi) {
      load_tile(t + 1);
      asm volatile("cp.async.wait_group 1;");
    } else {
      asm volatile("cp.async.wait_group 0;");
    }
    __syncthreads();
    const bf16* kt = sK + (t & 1) * kDecKeys * LD;
    // scores [16 heads][8 * MT keys]: two k-steps per round into separate accumulators
    float s2[2][MT][4];
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int c = 0; c < 4; ++c) s2[e][i][c] = 0.f;
    const uint32_t qb = smem_u32(sQ + (mt * 16 + (lane & 15)) * LD + (lane >> 4) * 8);
    // one ldmatrix.x4 brings 8 keys x 32 channels
    const uint32_t kb = smem_u32(kt + (kgrp * 8 * MT + (lane & 7)) * LD + (lane >> 3) * 8);
    int k = 0;
#pragma unroll 2
    for (; k + 1 < ksteps; k += 2) {
      uint32_t a0[4], a1[4], bb[MT][4];
      ldsm4(a0, qb + k * 32);
      ldsm4(a1, qb + k * 32 + 32);
#pragma unroll
      for (int i = 0; i < MT; ++i) ldsm4(bb[i], kb + (i * 8 * LD + k * 16) * 2);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        mma16816(s2[0][i], a0, bb[i][0], bb[i][1]);
        mma16816(s2[1][i], a1, bb[i][2], bb[i][3]);
      }
    }
    if (k < ksteps) {   // odd count: the upper half of the x4 load would pass the row's end, so it repeats the lower
      uint32_t a0[4], bb[4];
      ldsm4(a0, qb + k * 32);
      const uint32_t kb1 = smem_u32(kt + (kgrp * 8 * MT + (lane & 7)) * LD + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        ldsm4(bb, kb1 + (i * 8 * LD + k * 16) * 2);
        mma16816(s2[0][i], a0, bb[0], bb[1]);
      }
    }
    // mask, maximum over this warp's keys, then over the key groups
    float mine[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int key = t * kDecKeys + (kgrp * MT + i) * 8 + tq * 2;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const float x = s2[0][i][c] + s2[1][i][c];
        s2[0][i][c] = key + (c & 1) < len ? x * p.scale_log2 : -INFINITY;
        mine[c >> 1] = fmaxf(mine[c >> 1], s2[0][i][c]);
      }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mine[r] = fmaxf(mine[r], __shfl_xor_sync(0xffffffffu, mine[r], 1));
      mine[r] = fmaxf(mine[r], __shfl_xor_sync(0xffffffffu, mine[r], 2));
      if (tq == 0) s_max[kgrp * HB + mt * 16 + r * 8 + g] = mine[r];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int hr = i * 16 + r * 8 + g;
        float mx = m[i][r];
#pragma unroll
        for (int w = 0; w < KG; ++w) mx = fmaxf(mx, s_max[w * HB + hr]);   // a tile has at least one visible key
        const float a = fast_exp2(m[i][r] - mx);
        m[i][r] = mx;
        if (a != 1.f) {
#pragma unroll
          for (int j = 0; j < NT; ++j) {
            o[i][j][2 * r] *= a;
            o[i][j][2 * r + 1] *= a;
          }
        }
        if (i == mt) {
          l[r] *= a;
#pragma unroll
          for (int x = 0; x < MT; ++x) {
            const float p0 = fast_exp2(s2[0][x][2 * r] - mx), p1 = fast_exp2(s2[0][x][2 * r + 1] - mx);
            l[r] += p0 + p1;      // this lane's keys only; summed at the end
            *reinterpret_cast<uint32_t*>(sP + hr * LDP + (kgrp * MT + x) * 8 + tq * 2) = pack_bf16(p0, p1);
          }
        }
      }
    __syncthreads();
    // o += P V, V = latent columns of the key tile
    const uint32_t pb = smem_u32(sP + (lane & 15) * LDP + (lane >> 4) * 8);
#pragma unroll
    for (int kk = 0; kk < kDecKeys / 16; ++kk) {
      uint32_t a[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ldsm4(a[i], pb + (i * 16 * LDP + kk * 16) * 2);
      const uint32_t vb = smem_u32(kt + (kk * 16 + (lane & 15)) * LD + warp * NT * 8);
#pragma unroll
      for (int j = 0; j + 1 < NT; j += 2) {
        uint32_t v[4];
        ldsm4t(v, vb + (j * 8 + (lane >> 4) * 8) * 2);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma16816(o[i][j], a[i], v[0], v[1]);
          mma16816(o[i][j + 1], a[i], v[2], v[3]);
        }
      }
      if (NT & 1) {
        uint32_t v[4];
        ldsm4t(v, vb + (NT - 1) * 16);        // both halves read the same 8 columns
#pragma unroll
        for (int i = 0; i < MT; ++i) mma16816(o[i][NT - 1], a[i], v[0], v[1]);
      }
    }
    __syncthreads();      // the tile and P are free for the next round
  }
  // row sums: over the four lanes of a row, then over the key groups
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float x = l[r];
    x += __shfl_xor_sync(0xffffffffu, x, 1);
    x += __shfl_xor_sync(0xffffffffu, x, 2);
    if (tq == 0) s_sum[kgrp * HB + mt * 16 + r * 8 + g] = x;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int hr = i * 16 + r * 8 + g, h = h0 + hr;
      if (h >= p.H) continue;
      if (warp == 0 && tq == 0) {
        float t = 0.f;
        for (int w = 0; w < KG; ++w) t += s_sum[w * HB + hr];
        pml[h * 2] = m[i][r];
        pml[h * 2 + 1] = t;
      }
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int c = (warp * NT + j) * 8 + tq * 2;
        if (c < p.rank) *reinterpret_cast<float2*>(po + (long long)h * p.rank + c) = make_float2(o[i][j][2 * r], o[i][j][2 * r + 1]);
      }
    }
}

// out[b, h, :] = sum over at most 64 splits; CTA = (head, sequence, 128 columns)
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                             float* __restrict__ out, int H, int rank, int splits) {
  __shared__ float wgt[64];
  const int h = blockIdx.x, b = blockIdx.y;
  const float2* ml = (const float2*)part_ml + (long long)b * splits * H + h;
  const float* po = part_o + (long long)b * splits * H * rank + (long long)h * rank;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    float2 x[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) x[i] = lane + 32 * i < splits ? ml[(long long)(lane + 32 * i) * H] : make_float2(-INFINITY, 0.f);
    const float m = warp_max(fmaxf(x[0].x, x[1].x));
    float e[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) e[i] = x[i].x == -INFINITY ? 0.f : fast_exp2(x[i].x - m);
    const float l = warp_sum(e[0] * x[0].y + e[1] * x[1].y);
    const float inv = l > 0.f ? 1.f / l : 0.f;
    wgt[lane] = e[0] * inv;
    wgt[lane + 32] = e[1] * inv;
  }
  __syncthreads();
  const int c = blockIdx.z * 128 + threadIdx.x;
  if (c >= rank) return;
  float o = 0.f;
  for (int s0 = 0; s0 < splits; s0 += 16) {
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) x[i] = po[(long long)min(s0 + i, splits - 1) * H * rank + c];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      const float w = s0 + i < splits ? wgt[s0 + i] : 0.f;
      o += w != 0.f ? x[i] * w : 0.f;      // a split without keys wrote no row
    }
  }
  out[((long long)b * H + h) * rank + c] = o;
}

template <int MT, int NT>
static int launch_decode(const LatentDecodeArgs& a, int B, cudaStream_t s) {
  const int LD = 64 * NT + ((a.rot + 15) & ~15) + 8;
  const int smem = (16 * MT + 2 * kDecKeys) * LD * 2 + 16 * MT * (kDecKeys + 8) * 2 + 2 * (8 / MT) * 16 * MT * 4;
  if (smem > 227 * 1024) return 6005;
  auto kern = latent_decode_kernel<MT, NT>;
  OB_ENSURE_DYN_SMEM(kern, 227 * 1024);
  dim3 grid(a.splits, (a.H + 16 * MT - 1) / (16 * MT), B);
  kern<<<grid, 256, smem, s>>>(a);
  OB_CHECK_LAUNCH();
  return 0;
}

template <int MT>
static int dispatch_decode(const LatentDecodeArgs& a, int B, cudaStream_t s) {
  switch ((a.rank + 63) / 64) {
    case 1: return launch_decode<MT, 1>(a, B, s);
    case 2: return launch_decode<MT, 2>(a, B, s);
    case 3: return launch_decode<MT, 3>(a, B, s);
    case 4: return launch_decode<MT, 4>(a, B, s);
    case 5: case 6: return launch_decode<MT, 6>(a, B, s);
    case 7: case 8: return launch_decode<MT, 8>(a, B, s);
  }
  return 6005;
}

template <typename T>
static int launch_prepare(const LatentPrepArgs& a, int N, cudaStream_t s) {
  latent_prepare_kernel<T><<<N, 256, 0, s>>>(a);
  OB_CHECK_LAUNCH();
  return 0;
}

}  // namespace ob

using namespace ob;

extern "C" {

int ob_latent_prepare(void* proj, long long ldp, int dkv_off, const int* pos, const int* row, const float* cos_t,
                      const float* sin_t, int table_rows, int pairs, const void* norm_w, void* cache, long long cache_rows,
                      long long ldc, void* packed, int N, int H, int dim, int rot, int rank, float eps, int fp32,
                      int* status, cudaStream_t s) {
  if (N <= 0) return 0;
  if (2 * pairs > rot) return 6005;
  LatentPrepArgs a = {proj, pos, row, cos_t, sin_t, norm_w, cache, packed, ldp, ldc, cache_rows, dkv_off, H, dim, rot,
                      rank, pairs, table_rows, eps, status};
  return fp32 ? launch_prepare<float>(a, N, s) : launch_prepare<bf16>(a, N, s);
}

// out: fp32 [N, H, rank], or bf16 when out_bf16 (bf16 inputs only)
int ob_latent_absorb(const void* q, long long ldq, int head_stride, const void* uk, void* out, int N, int H, int dim,
                     int rank, int fp32, int out_bf16, cudaStream_t s) {
  if (N <= 0) return 0;
  const int smem = 8 * dim * 4;
  if (smem > 30 * 1024 || (fp32 && out_bf16)) return 6005;
  const bool vec = rank % 4 == 0 && !((uintptr_t)uk & 15);
  for (int n0 = 0; n0 < N; n0 += 8 * 65535) {     // gridDim.z limit
    const int n = N - n0 < 8 * 65535 ? N - n0 : 8 * 65535;
    const dim3 grid((rank + 127) / 128, H, (n + 7) / 8);
    const long long qo = n0 * ldq, oo = (long long)n0 * H * rank;
#define OB_ABSORB(T, O)                                                                                              \
  do {                                                                                                               \
    if (vec) latent_absorb_kernel<T, O, true><<<grid, 128, smem, s>>>((const T*)q + qo, ldq, head_stride, (const T*)uk, (O*)out + oo, n, H, dim, rank); \
    else latent_absorb_kernel<T, O, false><<<grid, 128, smem, s>>>((const T*)q + qo, ldq, head_stride, (const T*)uk, (O*)out + oo, n, H, dim, rank);    \
  } while (0)
    if (fp32) OB_ABSORB(float, float);
    else if (out_bf16) OB_ABSORB(bf16, bf16);
    else OB_ABSORB(bf16, float);
#undef OB_ABSORB
    OB_CHECK_LAUNCH();
  }
  return 0;
}

int ob_latent_expand(const float* o_lat, const void* uv, void* out, int N, int H, int vdim, int rank, int fp32,
                     cudaStream_t s) {
  if (N <= 0) return 0;
  const int smem = 8 * ((rank + 3) & ~3) * 4;
  if (smem > 48 * 1024) return 6005;
  const bool vec = rank % 4 == 0 && !((uintptr_t)uv & 15);
  for (int n0 = 0; n0 < N; n0 += 8 * 65535) {
    const int n = N - n0 < 8 * 65535 ? N - n0 : 8 * 65535;
    const dim3 grid((vdim + 31) / 32, H, (n + 7) / 8);
    const float* ol = o_lat + (long long)n0 * H * rank;
#define OB_EXPAND(T)                                                                                                 \
  do {                                                                                                               \
    T* o = (T*)out + (long long)n0 * H * vdim;                                                                       \
    if (vec) latent_expand_kernel<T, true><<<grid, 256, smem, s>>>(ol, (const T*)uv, o, n, H, vdim, rank);           \
    else latent_expand_kernel<T, false><<<grid, 256, smem, s>>>(ol, (const T*)uv, o, n, H, vdim, rank);              \
  } while (0)
    if (fp32) OB_EXPAND(float);
    else OB_EXPAND(bf16);
#undef OB_EXPAND
    OB_CHECK_LAUNCH();
  }
  return 0;
}

int ob_latent_attn_any(const float* q_lat, const void* q_rot, long long ldq, int head_stride, const void* cache,
                       long long ldc, const int* seq, const int* len, const int* table, int max_blocks, int page_size,
                       float* out, int N, int H, int rank, int rot, float scale, int fp32, cudaStream_t s) {
  if (N <= 0) return 0;
  LatentAttnArgs a = {q_lat, q_rot, cache, seq, len, table, out, ldq, ldc, head_stride, H, rank, rot, max_blocks, page_size, scale};
  const int smem = (2 * rank + rot + 2 * kAnyKeys) * 4;
  if (smem > 48 * 1024) return 6005;
  for (int n0 = 0; n0 < N; n0 += 32768) {      // gridDim.y limit
    const int n = N - n0 < 32768 ? N - n0 : 32768;
    LatentAttnArgs c = a;
    c.q_lat = q_lat + (long long)n0 * H * rank;
    c.q_rot = fp32 ? (const void*)((const float*)q_rot + n0 * ldq) : (const void*)((const bf16*)q_rot + n0 * ldq);
    c.seq = seq + n0; c.len = len + n0; c.out = out + (long long)n0 * H * rank;
    if (fp32) latent_attn_any_kernel<float><<<dim3(H, n), 128, smem, s>>>(c);
    else latent_attn_any_kernel<bf16><<<dim3(H, n), 128, smem, s>>>(c);
    OB_CHECK_LAUNCH();
  }
  return 0;
}

// bf16 decode, one query row per sequence.  rank, rot, ldc, ldq, head_stride multiples of 8; rank <= 512.
// part_o fp32 [B*splits*H*rank], part_ml fp32 [B*splits*H*2]; out fp32 [B, H, rank].
int ob_latent_decode(const void* q_lat, const void* q_rot, long long ldq, int head_stride, const void* cache,
                     long long ldc, const int* len, const int* table, int max_blocks, int page_size, float* part_o,
                     float* part_ml, float* out, int B, int H, int rank, int rot, int splits, float scale,
                     cudaStream_t s) {
  if (B <= 0) return 0;
  if ((rank & 7) || (rot & 7) || (ldc & 7) || (ldq & 7) || (head_stride & 7) || splits < 1 || splits > 64) return 6001;
  if ((((uintptr_t)q_lat) | ((uintptr_t)q_rot) | ((uintptr_t)cache)) & 15) return 6002;
  LatentDecodeArgs a = {(const bf16*)q_lat, (const bf16*)q_rot, (const bf16*)cache, len, table, part_o, part_ml, ldq, ldc,
                        head_stride, H, rank, rot, max_blocks, page_size, splits, scale * 1.4426950408889634f};
  const int rc = H <= 16 ? dispatch_decode<1>(a, B, s) : dispatch_decode<2>(a, B, s);
  if (rc) return rc;
  latent_combine_kernel<<<dim3(H, B, (rank + 127) / 128), 128, 0, s>>>(part_o, part_ml, out, H, rank, splits);
  OB_CHECK_LAUNCH();
  return 0;
}

}  // extern "C"
