// Row operations of decoders whose residual stream is kept in fp32: token embedding into fp32 rows,
// layer norm with bias and RMS norm from fp32 rows to the matrix-product dtype, squared-relu and gated
// activations, soft-capped logits.  Forward only.  Every kernel exists for bf16 and fp32 weights / outputs.
#include "host_utils.h"
#include "serve_common.cuh"

namespace ob {

template <typename T>
__global__ void embed_rows_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out,
                                  int V, int D, int* status) {
  const int n = blockIdx.x;
  const int id = ids[n];
  float* o = out + (long long)n * D;
  const bool vec = D % 4 == 0;      // rows of both tensors then start on vector boundaries
  if (id < 0 || id >= V) {   // a row without a token (padding of a fixed-size decode batch): zeros
    if (id != -1 && threadIdx.x == 0) atomicCAS(status, 0, OB_ERR_BAD_ARG | (n << 8));
    for (int i = threadIdx.x; i < D; i += blockDim.x) o[i] = 0.f;
    return;
  }
  const T* r = table + (long long)id * D;
  if (vec) {
#pragma unroll 4
    for (int i = threadIdx.x * 4; i < D; i += blockDim.x * 4) store4(o + i, load4(r + i));
  } else {
    for (int i = threadIdx.x; i < D; i += blockDim.x) o[i] = to_f(r[i]);
  }
}

// kMean: y = (x - mean) / sqrt(var + eps) * w + b with the variance of the deviations (two passes over
// registers); otherwise y = x / sqrt(mean(x^2) + eps) * w.  One CTA of 256 threads per row; NV float4 per
// thread cover D <= 1024 * NV, D % 4 == 0.
template <typename T, int NV, bool kMean>
__global__ void __launch_bounds__(256) norm_rows_kernel(const float* __restrict__ x, const T* __restrict__ w,
                                                        const T* __restrict__ b, T* __restrict__ y, int D, float eps) {
  __shared__ float red[33];
  const float* xr = x + (long long)blockIdx.x * D;
  T* yr = y + (long long)blockIdx.x * D;
  float4 v[NV];
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * 256) * 4;
    v[i] = c < D ? load4(xr + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
  }
  const float mean = kMean ? block_sum<256>(s, red) / (float)D : 0.f;
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * 256) * 4;
    if (c < D) {
      v[i].x -= mean; v[i].y -= mean; v[i].z -= mean; v[i].w -= mean;
      q += (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
    }
  }
  const float rstd = 1.f / sqrtf(block_sum<256>(q, red) / (float)D + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * 256) * 4;
    if (c < D) {
      const float4 ww = load4(w + c), bb = kMean ? load4(b + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      store4(yr + c, make_float4(v[i].x * rstd * ww.x + bb.x, v[i].y * rstd * ww.y + bb.y,
                                 v[i].z * rstd * ww.z + bb.z, v[i].w * rstd * ww.w + bb.w));
    }
  }
}

// any D
template <typename T, bool kMean>
__global__ void __launch_bounds__(256) norm_rows_any_kernel(const float* __restrict__ x, const T* __restrict__ w,
                                                            const T* __restrict__ b, T* __restrict__ y, int D, float eps) {
  __shared__ float red[33];
  const float* xr = x + (long long)blockIdx.x * D;
  T* yr = y + (long long)blockIdx.x * D;
  float mean = 0.f;
  if (kMean) {
    float s = 0.f;
    for (int c = threadIdx.x; c < D; c += 256) s += xr[c];
    mean = block_sum<256>(s, red) / (float)D;
  }
  float q = 0.f;
  for (int c = threadIdx.x; c < D; c += 256) {
    const float d = xr[c] - mean;
    q += d * d;
  }
  const float rstd = 1.f / sqrtf(block_sum<256>(q, red) / (float)D + eps);
  for (int c = threadIdx.x; c < D; c += 256)
    yr[c] = from_f<T>((xr[c] - mean) * rstd * to_f(w[c]) + (kMean ? to_f(b[c]) : 0.f));
}

// act(gate) * up over rows [gate F | up F]; kGelu: the tanh form 0.5 z (1 + tanh t) = z sigmoid(2 t) with
// t = sqrt(2/pi) (z + 0.044715 z^3), else silu.  bf16 rows take the fast exponential and division.
template <typename T, bool kGelu>
__device__ __forceinline__ float gate_value(float z, float up) {
  const float t = kGelu ? 1.5957691216057308f * (z + 0.044715f * z * z * z) : z;
  if (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-t)) * up;
  return z / (1.f + expf(-t)) * up;
}

// rows: a device count of the rows that matter (null: all of them).  VEC: F % 8 == 0.
template <typename T, bool kGelu, bool VEC>
__global__ void __launch_bounds__(256) gated_act_kernel(const T* __restrict__ x, T* __restrict__ y, const int* __restrict__ rows,
                                                        long long M, int F) {
  if (rows) M = min(M, (long long)*rows);
  const unsigned C = VEC ? F >> 3 : F;
  const long long n = M * C, stride = (long long)gridDim.x * 256;
  for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += stride) {
    const long long r = n < (1ll << 32) ? (unsigned)i / C : i / C;
    const unsigned c = (unsigned)(i - r * C);
    const T *a = x + r * 2 * F, *b = a + F;
    if (VEC) {
      float g[8], u[8];
      load8(a + 8 * c, g);
      load8(b + 8 * c, u);
#pragma unroll
      for (int e = 0; e < 8; ++e) g[e] = gate_value<T, kGelu>(g[e], u[e]);
      store8(y + r * F + 8 * c, g);
    } else {
      y[r * F + c] = from_f<T>(gate_value<T, kGelu>(to_f(a[c]), to_f(b[c])));
    }
  }
}

template <typename T>
__global__ void relu_sq_kernel(const T* __restrict__ x, T* __restrict__ y, long long n) {
  const long long n4 = n >> 2;
  const long long stride = (long long)gridDim.x * blockDim.x;
  const long long t0 = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  for (long long i = t0; i < n4; i += stride) {
    float4 v = load4(x + 4 * i);
    v.x = fmaxf(v.x, 0.f); v.y = fmaxf(v.y, 0.f); v.z = fmaxf(v.z, 0.f); v.w = fmaxf(v.w, 0.f);
    store4(y + 4 * i, make_float4(v.x * v.x, v.y * v.y, v.z * v.z, v.w * v.w));
  }
  for (long long i = 4 * n4 + t0; i < n; i += stride) {
    const float v = fmaxf(to_f(x[i]), 0.f);
    y[i] = from_f<T>(v * v);
  }
}

__global__ void soft_cap_kernel(float* __restrict__ x, long long n, float cap) {
  const long long stride = (long long)gridDim.x * blockDim.x;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += stride)
    x[i] = cap * tanhf(x[i] / cap);
}

template <typename T, bool kMean>
static int launch_norm(const float* x, const void* w, const void* b, void* y, int N, int D, float eps, cudaStream_t s) {
  const T *wt = (const T*)w, *bt = (const T*)b;
  T* yt = (T*)y;
  if (D % 4 || D > 8192) norm_rows_any_kernel<T, kMean><<<N, 256, 0, s>>>(x, wt, bt, yt, D, eps);
  else if (D <= 1024) norm_rows_kernel<T, 1, kMean><<<N, 256, 0, s>>>(x, wt, bt, yt, D, eps);
  else if (D <= 2048) norm_rows_kernel<T, 2, kMean><<<N, 256, 0, s>>>(x, wt, bt, yt, D, eps);
  else if (D <= 4096) norm_rows_kernel<T, 4, kMean><<<N, 256, 0, s>>>(x, wt, bt, yt, D, eps);
  else norm_rows_kernel<T, 8, kMean><<<N, 256, 0, s>>>(x, wt, bt, yt, D, eps);
  OB_CHECK_LAUNCH();
  return 0;
}

static unsigned flat_grid(long long n) {
  const long long blocks = (n + 255) / 256, cap = (long long)num_sms() * 16;
  return (unsigned)(blocks < 1 ? 1 : blocks < cap ? blocks : cap);
}

}  // namespace ob

using namespace ob;

extern "C" {

// ids [N] (-1: no token, zero row); table [V, D]; out fp32 [N, D]
int ob_embed_rows(const int* ids, const void* table, float* out, int N, int V, int D, int fp32, int* status,
                  cudaStream_t s) {
  if (N <= 0) return 0;
  if (fp32) embed_rows_kernel<float><<<N, 256, 0, s>>>(ids, (const float*)table, out, V, D, status);
  else embed_rows_kernel<bf16><<<N, 256, 0, s>>>(ids, (const bf16*)table, out, V, D, status);
  OB_CHECK_LAUNCH();
  return 0;
}

int ob_ln_rows(const float* x, const void* w, const void* b, void* y, int N, int D, float eps, int fp32,
               cudaStream_t s) {
  if (N <= 0) return 0;
  return fp32 ? launch_norm<float, true>(x, w, b, y, N, D, eps, s) : launch_norm<bf16, true>(x, w, b, y, N, D, eps, s);
}

int ob_rms_rows(const float* x, const void* w, void* y, int N, int D, float eps, int fp32, cudaStream_t s) {
  if (N <= 0) return 0;
  return fp32 ? launch_norm<float, false>(x, w, nullptr, y, N, D, eps, s)
              : launch_norm<bf16, false>(x, w, nullptr, y, N, D, eps, s);
}

// x T [M, 2F] = [gate | up] -> y T [M, F]; gelu: 1 tanh-form gelu, 0 silu; rows: device row count or null
int ob_gated_act(const void* x, void* y, const int* rows, long long M, int F, int gelu, int fp32, cudaStream_t s) {
  if (M <= 0 || F <= 0) return 0;
  const bool vec = F % 8 == 0 && !((((uintptr_t)x) | ((uintptr_t)y)) & 15);
  const unsigned grid = flat_grid(M * (vec ? F / 8 : F));
#define OB_ACT(T, G)                                                                                  \
  do {                                                                                                \
    if (vec) gated_act_kernel<T, G, true><<<grid, 256, 0, s>>>((const T*)x, (T*)y, rows, M, F);       \
    else gated_act_kernel<T, G, false><<<grid, 256, 0, s>>>((const T*)x, (T*)y, rows, M, F);          \
  } while (0)
  if (fp32) { if (gelu) OB_ACT(float, true); else OB_ACT(float, false); }
  else { if (gelu) OB_ACT(bf16, true); else OB_ACT(bf16, false); }
#undef OB_ACT
  OB_CHECK_LAUNCH();
  return 0;
}

int ob_relu_sq(const void* x, void* y, long long n, int fp32, cudaStream_t s) {
  if (n <= 0) return 0;
  if (fp32) relu_sq_kernel<float><<<flat_grid(n / 4), 256, 0, s>>>((const float*)x, (float*)y, n);
  else relu_sq_kernel<bf16><<<flat_grid(n / 4), 256, 0, s>>>((const bf16*)x, (bf16*)y, n);
  OB_CHECK_LAUNCH();
  return 0;
}

int ob_soft_cap(float* x, long long n, float cap, cudaStream_t s) {
  if (n <= 0) return 0;
  soft_cap_kernel<<<flat_grid(n), 256, 0, s>>>(x, n, cap);
  OB_CHECK_LAUNCH();
  return 0;
}

}  // extern "C"
