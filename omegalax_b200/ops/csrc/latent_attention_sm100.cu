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
// Attention over the pages is that of paged_rows_attention.cuh with one row for all heads.
#include "paged_rows_attention.cuh"

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
  PagedAttnArgs a = {q_lat, q_rot, cache, seq, len, table, nullptr, out, ldq, ldc, head_stride, H, H, rank, rot,
                     max_blocks, page_size, 0, scale};
  return fp32 ? launch_paged_any<float, float, true>(a, N, s) : launch_paged_any<bf16, float, true>(a, N, s);
}

// bf16 decode, one query row per sequence.  part_o fp32 [B*splits*H*rank], part_ml fp32 [B*splits*H*2];
// out fp32 [B, H, rank].
int ob_latent_decode(const void* q_lat, const void* q_rot, long long ldq, int head_stride, const void* cache,
                     long long ldc, const int* len, const int* table, int max_blocks, int page_size, float* part_o,
                     float* part_ml, float* out, int B, int H, int rank, int rot, int splits, float scale,
                     cudaStream_t s) {
  if (B <= 0) return 0;
  PagedDecodeArgs a = {(const bf16*)q_lat, (const bf16*)q_rot, (const bf16*)cache, len, table, part_o, part_ml, nullptr, out,
                       ldq, ldc, head_stride, H, H, rank, rot, max_blocks, page_size, splits, 0, scale * kLog2e};
  return dispatch_paged_decode<true, float>(a, B, s);
}

}  // extern "C"
