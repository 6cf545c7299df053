// Grouped-query attention with a sliding window, a sink, norms over whole projections and value mixing, over
// a paged cache, forward only.
//
//   window_prepare_kernel   RMS norm of all query heads at once and of all key heads at once, rotate-half
//                           rotation, values mixed with another layer's; [v | k] -> cache row, q, k and v
//                           rewritten in place (prompts attend to the packed rows)
//
// Attention over the pages is that of paged_rows_attention.cuh with c = value and r = key.
#include "paged_rows_attention.cuh"

namespace ob {

struct WindowPrepArgs {
  void* proj;              // T [N, ldp]: q [H, dim] | k [G, dim] | v [G, vdim]
  const int* pos;          // [N] position in the sequence, -1: no token
  const int* row;          // [N] cache row of the token
  const float* cos_t;      // [positions, pairs]
  const float* sin_t;
  const void* norm_w;      // T [(H + G) * dim]
  const void* mix;         // T [1] or null: share of v_first in v
  const void* v_first;     // T [N, ldv]
  void* cache;             // T [rows, ldc]
  long long ldp, ldv, ldc, cache_rows;
  int H, G, dim, vdim, pairs, table_rows;
  float eps;
  int* status;
};

// false when the row holds no token or its indices are out of range (reported)
__device__ __forceinline__ bool window_row_ok(const WindowPrepArgs& p, int n, int pos, int row) {
  if (pos >= 0 && pos < p.table_rows && row >= 0 && row < p.cache_rows) return true;
  if (pos != -1 && threadIdx.x == 0) atomicCAS(p.status, 0, OB_ERR_BAD_ARG | (n << 8));
  return false;
}

// Vectors of 8: a unit is a vector of the first half of a head's rotated channels with its partner in the
// second half, or a vector of the channels that are not rotated.  A thread keeps NU units in registers
// from the sums of squares to the stores.  2 * pairs % 16, dim % 8, vdim % 8 == 0, 16-byte aligned rows.
template <typename T, int NU>
__global__ void __launch_bounds__(256) window_prepare_kernel(const WindowPrepArgs p) {
  __shared__ float red[33];
  const int n = blockIdx.x;
  const int pos = p.pos[n], row = p.row[n];
  if (!window_row_ok(p, n, pos, row)) return;
  T* proj = (T*)p.proj + (long long)n * p.ldp;
  T* dst = (T*)p.cache + (long long)row * p.ldc;
  const int hu = p.pairs >> 3, U = hu + ((p.dim - 2 * p.pairs) >> 3), units = (p.H + p.G) * U, hd = p.dim + p.vdim;
  float a[NU][8], b[NU][8];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < NU; ++i) {
    const int u = threadIdx.x + i * 256;
    if (u >= units) continue;
    const int h = u / U, j = u - h * U;
    const T* x = proj + h * p.dim + (j < hu ? 8 * j : 2 * p.pairs + 8 * (j - hu));
    load8(x, a[i]);
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) s = fmaf(a[i][e], a[i][e], s);
    if (j < hu) {
      load8(x + p.pairs, b[i]);
#pragma unroll
      for (int e = 0; e < 8; ++e) s = fmaf(b[i][e], b[i][e], s);
    }
    (h < p.H ? sq : sk) += s;
  }
  // values: no dependence on the norms
  const int vv = p.vdim >> 3;
  const float lam = p.mix ? to_f(*(const T*)p.mix) : 0.f;
  for (int u = threadIdx.x; u < p.G * vv; u += 256) {
    const int g = u / vv, j = u - g * vv;
    T* x = proj + (p.H + p.G) * p.dim + 8 * u;
    float v[8];
    load8(x, v);
    if (p.mix) {
      float f[8];
      load8((const T*)p.v_first + (long long)n * p.ldv + 8 * u, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = (1.f - lam) * v[e] + lam * f[e];
      store8(x, v);
    }
    store8(dst + g * hd + 8 * j, v);
  }
  const float rq = 1.f / sqrtf(block_sum<256>(sq, red) / (float)(p.H * p.dim) + p.eps);
  const float rk = 1.f / sqrtf(block_sum<256>(sk, red) / (float)(p.G * p.dim) + p.eps);
  const float *ct = p.cos_t + (long long)pos * p.pairs, *st = p.sin_t + (long long)pos * p.pairs;
#pragma unroll
  for (int i = 0; i < NU; ++i) {
    const int u = threadIdx.x + i * 256;
    if (u >= units) continue;
    const int h = u / U, j = u - h * U;
    const int off = j < hu ? 8 * j : 2 * p.pairs + 8 * (j - hu);
    const T* w = (const T*)p.norm_w + h * p.dim + off;
    T* x = proj + h * p.dim + off;
    T* c = h < p.H ? nullptr : dst + (h - p.H) * hd + p.vdim + off;
    const float r = h < p.H ? rq : rk;
    float wa[8];
    load8(w, wa);
#pragma unroll
    for (int e = 0; e < 8; ++e) a[i][e] *= r * wa[e];
    if (j < hu) {
      float cs[8], sn[8];
      load8(w + p.pairs, wa);
      load8(ct + 8 * j, cs);
      load8(st + 8 * j, sn);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float x0 = a[i][e], x1 = b[i][e] * r * wa[e];
        a[i][e] = x0 * cs[e] - x1 * sn[e];
        b[i][e] = x1 * cs[e] + x0 * sn[e];
      }
      store8(x + p.pairs, b[i]);
      if (c) store8(c + p.pairs, b[i]);
    }
    store8(x, a[i]);
    if (c) store8(c, a[i]);
  }
}

// any sizes
template <typename T>
__global__ void __launch_bounds__(256) window_prepare_any_kernel(const WindowPrepArgs p) {
  __shared__ float red[33];
  const int n = blockIdx.x;
  const int pos = p.pos[n], row = p.row[n];
  if (!window_row_ok(p, n, pos, row)) return;
  T* proj = (T*)p.proj + (long long)n * p.ldp;
  T* dst = (T*)p.cache + (long long)row * p.ldc;
  const int nq = p.H * p.dim, nk = p.G * p.dim, hd = p.dim + p.vdim, plain = p.dim - p.pairs;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < nq + nk; i += 256) {
    const float v = to_f(proj[i]);
    (i < nq ? sq : sk) += v * v;
  }
  const float lam = p.mix ? to_f(*(const T*)p.mix) : 0.f;
  for (int i = threadIdx.x; i < p.G * p.vdim; i += 256) {
    T* x = proj + nq + nk + i;
    T v = *x;
    if (p.mix) {
      v = from_f<T>((1.f - lam) * to_f(v) + lam * to_f(((const T*)p.v_first)[(long long)n * p.ldv + i]));
      *x = v;
    }
    dst[i / p.vdim * hd + i % p.vdim] = v;
  }
  const float rq = 1.f / sqrtf(block_sum<256>(sq, red) / (float)nq + p.eps);
  const float rk = 1.f / sqrtf(block_sum<256>(sk, red) / (float)nk + p.eps);
  const float *ct = p.cos_t + (long long)pos * p.pairs, *st = p.sin_t + (long long)pos * p.pairs;
  // per head: pairs (i, i + pairs), then the channels from 2 * pairs on
  for (int i = threadIdx.x; i < (p.H + p.G) * plain; i += 256) {
    const int h = i / plain, j = i - h * plain, off = j < p.pairs ? j : j + p.pairs;
    const T* w = (const T*)p.norm_w + h * p.dim + off;
    T* x = proj + h * p.dim + off;
    T* c = h < p.H ? nullptr : dst + (h - p.H) * hd + p.vdim + off;
    const float r = h < p.H ? rq : rk;
    float u = to_f(x[0]) * r * to_f(w[0]);
    if (j < p.pairs) {
      const float v = to_f(x[p.pairs]) * r * to_f(w[p.pairs]);
      const T y = from_f<T>(v * ct[j] + u * st[j]);
      x[p.pairs] = y;
      if (c) c[p.pairs] = y;
      u = u * ct[j] - v * st[j];
    }
    const T y = from_f<T>(u);
    x[0] = y;
    if (c) c[0] = y;
  }
}

template <typename T>
static int launch_window_prepare(const WindowPrepArgs& a, int N, cudaStream_t s) {
  const int U = (a.pairs >> 3) + ((a.dim - 2 * a.pairs) >> 3), units = (a.H + a.G) * U;
  const uintptr_t bases = (uintptr_t)a.proj | (uintptr_t)a.norm_w | (uintptr_t)a.cache | (uintptr_t)a.v_first |
                          (uintptr_t)a.cos_t | (uintptr_t)a.sin_t;
  const bool vec = !((a.pairs | a.dim | a.vdim) & 7) && !((a.ldp | a.ldv | a.ldc) & 7) && !(bases & 15);
  if (vec && units <= 256) window_prepare_kernel<T, 1><<<N, 256, 0, s>>>(a);
  else if (vec && units <= 512) window_prepare_kernel<T, 2><<<N, 256, 0, s>>>(a);
  else if (vec && units <= 1024) window_prepare_kernel<T, 4><<<N, 256, 0, s>>>(a);
  else window_prepare_any_kernel<T><<<N, 256, 0, s>>>(a);
  OB_CHECK_LAUNCH();
  return 0;
}

}  // namespace ob

using namespace ob;

extern "C" {

int ob_window_prepare(void* proj, long long ldp, const int* pos, const int* row, const float* cos_t, const float* sin_t,
                      int table_rows, int pairs, const void* norm_w, const void* mix, const void* v_first, long long ldv,
                      void* cache, long long cache_rows, long long ldc, int N, int H, int G, int dim, int vdim, float eps,
                      int fp32, int* status, cudaStream_t s) {
  if (N <= 0) return 0;
  if (2 * pairs > dim || (mix && !v_first)) return 6005;
  WindowPrepArgs a = {proj, pos, row, cos_t, sin_t, norm_w, mix, v_first, cache, ldp, ldv, ldc, cache_rows, H, G, dim, vdim,
                      pairs, table_rows, eps, status};
  return fp32 ? launch_window_prepare<float>(a, N, s) : launch_window_prepare<bf16>(a, N, s);
}

// q T [N, H, dim] (pitch ldq) against the pages of each row's sequence; out T [N, H, vdim]
int ob_window_attn_any(const void* q, long long ldq, const void* cache, long long ldc, const int* seq, const int* len,
                       const int* table, int max_blocks, int page_size, const void* sink, void* out, int N, int H, int G,
                       int dim, int vdim, int window, float scale, int fp32, cudaStream_t s) {
  if (N <= 0) return 0;
  if (G <= 0 || H % G) return 6005;
  PagedAttnArgs a = {nullptr, q, cache, seq, len, table, sink, out, ldq, ldc, dim, H, H / G, vdim, dim, max_blocks, page_size,
                     window, scale};
  return fp32 ? launch_paged_any<float, float, false>(a, N, s) : launch_paged_any<bf16, bf16, false>(a, N, s);
}

// bf16 decode, one query row per sequence: q [B, H, dim] (pitch ldq) -> out bf16 [B, H, vdim].
// part_o fp32 [B*splits*H*vdim], part_ml fp32 [B*splits*H*2] with more than one split.
int ob_window_decode(const void* q, long long ldq, const void* cache, long long ldc, const int* len, const int* table,
                     int max_blocks, int page_size, const void* sink, float* part_o, float* part_ml, void* out, int B, int H,
                     int G, int dim, int vdim, int window, int splits, float scale, cudaStream_t s) {
  if (B <= 0) return 0;
  if (G <= 0 || H % G) return 6005;
  PagedDecodeArgs a = {nullptr, (const bf16*)q, (const bf16*)cache, len, table, part_o, part_ml, (const bf16*)sink, out, ldq,
                       ldc, dim, H, H / G, vdim, dim, max_blocks, page_size, splits, window, scale * kLog2e};
  return dispatch_paged_decode<false, bf16>(a, B, s);
}

}  // extern "C"
