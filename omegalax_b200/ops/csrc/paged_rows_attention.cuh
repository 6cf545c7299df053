// Attention over a paged cache whose rows hold, per key/value head, [c (rank) | r (rot)] of one token:
// the value is c, and the score of a query is either (q_c . c + q_r . r) (kScoreValues, latent
// attention: the latent is key and value at once) or q_r . r alone (c the value, r the key of ordinary
// attention).  H query heads share G = H / group key/value heads; the rows of page p are
// p * page_size ..., pitch ldc elements.  A query of a sequence with ``len`` visible tokens sees the last
// ``window`` of them (0: all).  ``sink`` (null: none) is one logit per query head that enters the
// softmax denominator without a value.
//
//   paged_attn_any_kernel      any query rows, any sizes, fp32 arithmetic
//   paged_decode_kernel        bf16, one query row per sequence, mma.sync tiles, split over the keys;
//                              partials are merged by paged_combine_kernel, a single split writes the result
#pragma once
#include "host_utils.h"
#include "serve_common.cuh"

namespace ob {

// ------------------------------------------------------------------------------------------------ any-size attention
struct PagedAttnArgs {
  const float* q_lat;      // [N, H, rank] (kScoreValues)
  const void* q_rot;       // T, q_rot + n*ldq + h*head_stride: rot values
  const void* cache;       // T [rows, ldc]
  const int* seq;          // [N]
  const int* len;          // [N] visible tokens of the query's sequence, 0: no query
  const int* table;        // [B, max_blocks]
  const void* sink;        // T [H] or null
  void* out;               // O [N, H, rank]
  long long ldq, ldc;
  int head_stride, H, group, rank, rot, max_blocks, page_size, window;
  float scale;
};

constexpr int kAnyKeys = 64;

template <typename T, typename O, bool kScoreValues>
__global__ void __launch_bounds__(128) paged_attn_any_kernel(const PagedAttnArgs p) {
  extern __shared__ float sm[];     // q[rank + rot], o[rank], s[kAnyKeys]; then rows[kAnyKeys]
  const int n = blockIdx.y, h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int F = p.rank + p.rot;
  constexpr bool kBoth = kScoreValues;
  float *q = sm, *o = sm + F, *sc = o + p.rank;
  int* rows = (int*)(sc + kAnyKeys);
  const int len = p.len[n];
  O* out = (O*)p.out + ((long long)n * p.H + h) * p.rank;
  for (int i = tid; i < p.rank; i += 128) {
    if (kBoth) q[i] = p.q_lat[((long long)n * p.H + h) * p.rank + i];
    o[i] = 0.f;
    if (len <= 0) out[i] = from_f<O>(0.f);
  }
  if (len <= 0) return;
  const T* qr = (const T*)p.q_rot + (long long)n * p.ldq + (long long)h * p.head_stride;
  for (int i = tid; i < p.rot; i += 128) q[p.rank + i] = to_f(qr[i]);
  const int* bt = p.table + (long long)p.seq[n] * p.max_blocks;
  const T* cache = (const T*)p.cache + (long long)(h / p.group) * F;
  const int lo = p.window > 0 ? max(0, len - p.window) : 0;
  float m = -INFINITY, l = 0.f;
  if (p.sink) {                       // a key with this score and no value
    m = to_f(((const T*)p.sink)[h]);
    l = 1.f;
  }
  for (int k0 = lo; k0 < len; k0 += kAnyKeys) {
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
      for (int i = (kBoth ? 0 : p.rank) + lane; i < F; i += 32) d = fmaf(q[i], to_f(r[i]), d);
      d = warp_sum(d);
      if (lane == 0) sc[k] = d * p.scale;
    }
    __syncthreads();
    float mx = m;
    for (int k = 0; k < nk; ++k) mx = fmaxf(mx, sc[k]);
    const float a = expf(m - mx);       // 0 on the first tile without a sink
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
  for (int i = tid; i < p.rank; i += 128) out[i] = from_f<O>(o[i] / l);
}

// N query rows; returns 6005 when a head does not fit shared memory
template <typename T, typename O, bool kScoreValues>
static int launch_paged_any(const PagedAttnArgs& a, int N, cudaStream_t s) {
  const int smem = (2 * a.rank + a.rot + 2 * kAnyKeys) * 4;
  if (smem > 48 * 1024) return 6005;
  for (int n0 = 0; n0 < N; n0 += 32768) {      // gridDim.y limit
    const int n = N - n0 < 32768 ? N - n0 : 32768;
    PagedAttnArgs c = a;
    if (kScoreValues) c.q_lat = a.q_lat + (long long)n0 * a.H * a.rank;
    c.q_rot = (const T*)a.q_rot + n0 * a.ldq;
    c.seq = a.seq + n0;
    c.len = a.len + n0;
    c.out = (O*)a.out + (long long)n0 * a.H * a.rank;
    paged_attn_any_kernel<T, O, kScoreValues><<<dim3(a.H, n), 128, smem, s>>>(c);
    OB_CHECK_LAUNCH();
  }
  return 0;
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

struct PagedDecodeArgs {
  const bf16* q_lat;       // [B, H, rank] (kScoreValues)
  const bf16* q_rot;       // q_rot + b*ldq + h*head_stride
  const bf16* cache;       // [rows, ldc]
  const int* len;          // [B]
  const int* table;        // [B, max_blocks]
  float* part_o;           // [B, splits, H, rank]
  float* part_ml;          // [B, splits, H, 2] (running maximum in log2 units, sum)
  const bf16* sink;        // [H] or null
  void* out;               // O [B, H, rank]; written here with one split, by the merge otherwise
  long long ldq, ldc;
  int head_stride, H, group, rank, rot, max_blocks, page_size, splits, window;
  float scale_log2;
};

constexpr int kDecKeys = 64;      // keys per tile
constexpr float kLog2e = 1.4426950408889634f;

// CTA = (key split, block of 16*MT heads of one key/value head, sequence), 8 warps.  Shared memory: Q [16*MT][LD],
// two key tiles [64][LD], P [16*MT][72] (bf16), LD = rank_pad + rot_pad + 8 (rank padded to a multiple
// of 64, rot to one of 16; the padding holds zeros).  Scores: a warp owns one 16-head tile and 8 * MT
// keys.  Output: warp w owns rank_pad / 8 = 8 * NT value columns for all heads of the block, in registers.
template <int MT, int NT, bool kScoreValues, typename O>
__global__ void __launch_bounds__(256) paged_decode_kernel(const PagedDecodeArgs p) {
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
  const int hblocks = (p.group + HB - 1) / HB;
  const int b = blockIdx.z, kvh = blockIdx.y / hblocks, sp = blockIdx.x;
  const int h0 = kvh * p.group + (blockIdx.y - kvh * hblocks) * HB;      // first head of the block
  const int h_end = min(h0 + HB, (kvh + 1) * p.group);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int first = p.window > 0 ? max(0, p.len[b] - p.window) : 0;
  const int len = p.len[b] - first;           // visible keys, first ... first + len - 1
  // whole tiles are handed out to the splits
  const int tiles = (len + kDecKeys - 1) / kDecKeys;
  const int per = (tiles + p.splits - 1) / p.splits;
  const int t_lo = min(sp * per, tiles), t_hi = min(t_lo + per, tiles);
  float* po = p.part_o + ((long long)b * p.splits + sp) * p.H * p.rank;
  float* pml = p.part_ml + ((long long)b * p.splits + sp) * p.H * 2;
  O* out = (O*)p.out + (long long)b * p.H * p.rank;
  if (t_lo >= t_hi) {
    if (p.splits == 1) {
      for (int i = h0 * p.rank + tid; i < h_end * p.rank; i += 256) out[i] = from_f<O>(0.f);
    } else {
      for (int h = h0 + tid; h < h_end; h += 256) {
        pml[h * 2] = -INFINITY;
        pml[h * 2 + 1] = 0.f;
      }
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
    const int k = first + min(t * kDecKeys + warp + 8 * (lane & 7), len - 1);   // past the end: the last row again (masked below)
    return bt[k / p.page_size] * p.page_size + k % p.page_size;
  };
  int rows = find_rows(t_lo);
  const bf16* cache = p.cache + (long long)kvh * (p.rank + p.rot);
  auto load_tile = [&](int t) {
    bf16* dst = sK + (t & 1) * kDecKeys * LD;
    const int now = rows;
    rows = find_rows(min(t + 1, t_hi - 1));
#pragma unroll
    for (int i = 0; i < kDecKeys / 8; ++i) {
      const bf16* src = cache + (long long)__shfl_sync(0xffffffffu, now, i) * p.ldc;
      const uint32_t d = smem_u32(dst + (warp + 8 * i) * LD);
      for (int v = lane; v < cv + rv; v += 32)
        cp16(d + (v < cv ? v * 16 : (RP + (v - cv) * 8) * 2), src + v * 8);
    }
    asm volatile("cp.async.commit_group;");
  };
  load_tile(t_lo);
  const int qv = kScoreValues ? cv + rv : rv;       // without kScoreValues the value columns of Q are not read
  for (int i = tid; i < HB * qv; i += 256) {
    const int r = i / qv, v = i - r * qv + (kScoreValues ? 0 : cv), h = h0 + r;
    uint4 u = make_uint4(0, 0, 0, 0);
    if (h < h_end)
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
  constexpr int kFrom = kScoreValues ? 0 : RP;      // first column that takes part in the score
  const int ksteps = (RP + rotp - kFrom) >> 4;
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
    const uint32_t qb = smem_u32(sQ + (mt * 16 + (lane & 15)) * LD + kFrom + (lane >> 4) * 8);
    // one ldmatrix.x4 brings 8 keys x 32 channels
    const uint32_t kb = smem_u32(kt + (kgrp * 8 * MT + (lane & 7)) * LD + kFrom + (lane >> 3) * 8);
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
      const uint32_t kb1 = smem_u32(kt + (kgrp * 8 * MT + (lane & 7)) * LD + kFrom + ((lane >> 3) & 1) * 8);
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
    // o += P V, V = value columns of the key tile
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
      if (h >= h_end) continue;
      float t = 0.f;
      for (int w = 0; w < KG; ++w) t += s_sum[w * HB + hr];
      if (p.splits == 1) {
        if (p.sink) t += fast_exp2(__bfloat162float(p.sink[h]) * kLog2e - m[i][r]);
        const float inv = 1.f / t;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const int c = (warp * NT + j) * 8 + tq * 2;
          if (c < p.rank) store2(out + (long long)h * p.rank + c, o[i][j][2 * r] * inv, o[i][j][2 * r + 1] * inv);
        }
        continue;
      }
      if (warp == 0 && tq == 0) {
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
template <typename O>
__global__ void __launch_bounds__(128) paged_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                                            const bf16* __restrict__ sink, O* __restrict__ out, int H,
                                                            int rank, int splits) {
  __shared__ float wgt[64];
  const int h = blockIdx.x, b = blockIdx.y;
  const float2* ml = (const float2*)part_ml + (long long)b * splits * H + h;
  const float* po = part_o + (long long)b * splits * H * rank + (long long)h * rank;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    float2 x[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) x[i] = lane + 32 * i < splits ? ml[(long long)(lane + 32 * i) * H] : make_float2(-INFINITY, 0.f);
    const float sk = sink ? __bfloat162float(sink[h]) * kLog2e : -INFINITY;
    const float m = fmaxf(warp_max(fmaxf(x[0].x, x[1].x)), sk);
    float e[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) e[i] = x[i].x == -INFINITY ? 0.f : fast_exp2(x[i].x - m);
    const float l = warp_sum(e[0] * x[0].y + e[1] * x[1].y) + (sink ? fast_exp2(sk - m) : 0.f);
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
  out[((long long)b * H + h) * rank + c] = from_f<O>(o);
}

template <int MT, int NT, bool kScoreValues, typename O>
static int launch_paged_decode(const PagedDecodeArgs& a, int B, cudaStream_t s) {
  const int LD = 64 * NT + ((a.rot + 15) & ~15) + 8;
  const int smem = (16 * MT + 2 * kDecKeys) * LD * 2 + 16 * MT * (kDecKeys + 8) * 2 + 2 * (8 / MT) * 16 * MT * 4;
  if (smem > 227 * 1024) return 6005;
  auto kern = paged_decode_kernel<MT, NT, kScoreValues, O>;
  OB_ENSURE_DYN_SMEM(kern, 227 * 1024);
  dim3 grid(a.splits, (a.group + 16 * MT - 1) / (16 * MT) * (a.H / a.group), B);
  kern<<<grid, 256, smem, s>>>(a);
  OB_CHECK_LAUNCH();
  if (a.splits > 1) {
    paged_combine_kernel<O><<<dim3(a.H, B, (a.rank + 127) / 128), 128, 0, s>>>(a.part_o, a.part_ml, a.sink, (O*)a.out, a.H,
                                                                               a.rank, a.splits);
    OB_CHECK_LAUNCH();
  }
  return 0;
}

template <int MT, bool kScoreValues, typename O>
static int dispatch_paged_decode_rank(const PagedDecodeArgs& a, int B, cudaStream_t s) {
  switch ((a.rank + 63) / 64) {
    case 1: return launch_paged_decode<MT, 1, kScoreValues, O>(a, B, s);
    case 2: return launch_paged_decode<MT, 2, kScoreValues, O>(a, B, s);
    case 3: return launch_paged_decode<MT, 3, kScoreValues, O>(a, B, s);
    case 4: return launch_paged_decode<MT, 4, kScoreValues, O>(a, B, s);
    case 5: case 6: return launch_paged_decode<MT, 6, kScoreValues, O>(a, B, s);
    case 7: case 8: return launch_paged_decode<MT, 8, kScoreValues, O>(a, B, s);
  }
  return 6005;
}

// rank, rot, ldc, ldq, head_stride multiples of 8; rank <= 512; 16-byte aligned tensors
template <bool kScoreValues, typename O>
static int dispatch_paged_decode(const PagedDecodeArgs& a, int B, cudaStream_t s) {
  if ((a.rank & 7) || (a.rot & 7) || (a.ldc & 7) || (a.ldq & 7) || (a.head_stride & 7) || a.splits < 1 || a.splits > 64)
    return 6001;
  if ((((uintptr_t)a.q_lat) | ((uintptr_t)a.q_rot) | ((uintptr_t)a.cache)) & 15) return 6002;
  return a.group <= 16 ? dispatch_paged_decode_rank<1, kScoreValues, O>(a, B, s)
                       : dispatch_paged_decode_rank<2, kScoreValues, O>(a, B, s);
}

}  // namespace ob
