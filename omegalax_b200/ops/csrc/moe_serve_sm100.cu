// Routed experts of serving decoders, forward only: the router's weight scales an expert's input and the
// outputs of a token's experts are summed into its fp32 residual row.
//
// Prompts sort (token, slot) pairs by expert (moe_route_sm100.cu), gather the scaled rows, run the
// grouped tcgen05 GEMM (or, for fp32 and sizes it cannot address, expert_rows_any_kernel) and sum.
// Few pairs (decoding) skip the sort: a CTA of the *_few kernels owns 16 output features of one expert,
// finds the pairs routed to it and streams the expert's weights past them on mma.sync tiles, weights as
// the 16-row operand and up to 16 pairs as columns, so that every weight is read once.
#include "host_utils.h"
#include "serve_common.cuh"

namespace ob {

constexpr int kFewPairs = 2048;      // most (token, slot) pairs of the *_few kernels

// ------------------------------------------------------------------------------------------------ row movement
// xs[dest[p]] = w[p] * h[p / k]
template <typename T, bool VEC>
__global__ void __launch_bounds__(128) moe_gather_kernel(const T* __restrict__ h, const float* __restrict__ w,
                                                         const int* __restrict__ dest, T* __restrict__ xs, int k, int D,
                                                         int max_rows) {
  const long long pr = blockIdx.x;
  const int d = dest[pr];
  if (d < 0 || d >= max_rows) return;
  const T* src = h + pr / k * D;
  T* dst = xs + (long long)d * D;
  const float a = w[pr];
  if (VEC) {
    for (int i = threadIdx.x * 8; i < D; i += 1024) {
      float v[8];
      load8(src + i, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= a;
      store8(dst + i, v);
    }
  } else {
    for (int i = threadIdx.x; i < D; i += 128) dst[i] = from_f<T>(to_f(src[i]) * a);
  }
}

// x[m] += sum over the k slots of y[dest[m * k + j]] (dest null: row m * k + j)
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) moe_sum_kernel(const T* __restrict__ y, const int* __restrict__ dest,
                                                      float* __restrict__ x, int k, int D, int max_rows) {
  const long long m = blockIdx.y;
  const int i = (blockIdx.x * 256 + threadIdx.x) * (VEC ? 4 : 1);
  if (i >= D) return;
  float* o = x + m * D + i;
  float4 acc = VEC ? load4(o) : make_float4(o[0], 0.f, 0.f, 0.f);
  for (int j = 0; j < k; ++j) {
    const long long r = dest ? dest[m * k + j] : m * k + j;
    if (r < 0 || r >= max_rows) continue;
    const T* s = y + r * D + i;
    if (VEC) {
      const float4 v = load4(s);
      acc.x += v.x; acc.y += v.y; acc.z += v.z; acc.w += v.w;
    } else {
      acc.x += to_f(s[0]);
    }
  }
  if (VEC) store4(o, acc);
  else o[0] = acc.x;
}

// ------------------------------------------------------------------------------------------------ any-size grouped product
// C[r, :N] = A[r, :K] W[e]^T for the rows r of [offsets[e], offsets[e + 1]); 64 x 64 tiles, fp32 arithmetic.
// CTA = (column block, expert, every gridDim.z-th row block).
template <typename T, typename O>
__global__ void __launch_bounds__(256) expert_rows_any_kernel(const T* __restrict__ A, const T* __restrict__ W,
                                                              O* __restrict__ C, const int* __restrict__ offsets, int N,
                                                              int K, int max_rows) {
  __shared__ __align__(16) float sa[16][68], sb[16][68];
  const int e = blockIdx.y, n0 = blockIdx.x * 64;
  const int lo = offsets[e], hi = min(offsets[e + 1], max_rows);
  const T* w = W + (long long)e * N * K;
  const int tr = threadIdx.x >> 4, tc = threadIdx.x & 15;
  for (int m0 = lo + blockIdx.z * 64; m0 < hi; m0 += gridDim.z * 64) {
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += 16) {
      __syncthreads();
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = tr + 16 * i, k = k0 + tc;
        sa[tc][r] = m0 + r < hi && k < K ? to_f(A[(long long)(m0 + r) * K + k]) : 0.f;
        sb[tc][r] = n0 + r < N && k < K ? to_f(w[(long long)(n0 + r) * K + k]) : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int kk = 0; kk < 16; ++kk) {
        const float4 a = load4(&sa[kk][tr * 4]), b = load4(&sb[kk][tc * 4]);
        const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = m0 + tr * 4 + i, n = n0 + tc * 4 + j;
        if (r < hi && n < N) C[(long long)r * N + n] = from_f<O>(acc[i][j]);
      }
  }
}

// ------------------------------------------------------------------------------------------------ few pairs
__device__ __forceinline__ void mma_bf16(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// The pairs routed to expert e, in any order (results do not depend on it).
__device__ __forceinline__ int find_pairs(const int* __restrict__ idx, int P, int e, int* list, int* count) {
  if (threadIdx.x == 0) *count = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < P; i += 128)
    if (idx[i] == e) list[atomicAdd(count, 1)] = i;
  __syncthreads();
  return *count;
}

// acc[t][c] += 16 rows of NW weight matrices (w[t], pitch K) times up to 16 columns, over this warp's quarter of
// K.  Column g of block c is the row x[c] of its lane group.  The four lanes of a group hold 8 consecutive
// channels each; both operands use that order, so a pair of MMAs consumes a 32-channel chunk with one
// 16-byte load per operand row.  K % 8 == 0.
template <int NW>
__device__ __forceinline__ void few_rows(const bf16* const* w, const bf16* const* x, bool two, int K, int warp, int tq,
                                         float (&acc)[NW][2][4]) {
  constexpr int U = 4;                     // chunks in flight
  const uint4 zero = make_uint4(0, 0, 0, 0);
  for (int k0 = warp * 32 * U; k0 < K; k0 += 4 * 32 * U) {
    uint4 a[U][NW][2], b[U][2];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = k0 + u * 32 + tq * 8;
      const bool in = k < K;
#pragma unroll
      for (int t = 0; t < NW; ++t) {
        a[u][t][0] = in ? __ldg(reinterpret_cast<const uint4*>(w[2 * t] + k)) : zero;
        a[u][t][1] = in ? __ldg(reinterpret_cast<const uint4*>(w[2 * t + 1] + k)) : zero;
      }
#pragma unroll
      for (int c = 0; c < 2; ++c) b[u][c] = in && x[c] && (c == 0 || two) ? *reinterpret_cast<const uint4*>(x[c] + k) : zero;
    }
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        if (c == 1 && !two) break;
#pragma unroll
        for (int t = 0; t < NW; ++t) {
          mma_bf16(acc[t][c], a[u][t][0].x, a[u][t][1].x, a[u][t][0].y, a[u][t][1].y, b[u][c].x, b[u][c].y);
          mma_bf16(acc[t][c], a[u][t][0].z, a[u][t][1].z, a[u][t][0].w, a[u][t][1].w, b[u][c].z, b[u][c].w);
        }
      }
  }
}

// act[p, f] = silu(s W_gate h) * (s W_up h), s = weight of pair p, for the pairs of expert blockIdx.y and the
// features f of block blockIdx.x; W [E][gate F rows | up F rows][K].  The products are linear in the input,
// so its scale is applied to them.
__global__ void __launch_bounds__(128) expert_up_few_kernel(const bf16* __restrict__ h, const bf16* __restrict__ W,
                                                            const int* __restrict__ idx, const float* __restrict__ weight,
                                                            bf16* __restrict__ act, int P, int k, int F, int K) {
  __shared__ int list[kFewPairs], count;
  __shared__ __align__(16) float red[4][2][2][128];
  const int e = blockIdx.y, f0 = blockIdx.x * 16;
  const int n = find_pairs(idx, P, e, list, &count);
  if (n == 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const bf16* we = W + (long long)e * 2 * F * K;
  const int r0 = min(f0 + g, F - 1), r1 = min(f0 + g + 8, F - 1);
  const bf16* w[4] = {we + (long long)r0 * K, we + (long long)r1 * K, we + (long long)(F + r0) * K, we + (long long)(F + r1) * K};
  for (int p0 = 0; p0 < n; p0 += 16) {
    const bf16* x[2];
#pragma unroll
    for (int c = 0; c < 2; ++c) x[c] = p0 + c * 8 + g < n ? h + (long long)(list[p0 + c * 8 + g] / k) * K : nullptr;
    float acc[2][2][4] = {};
    few_rows<2>(w, x, n - p0 > 8, K, warp, tq, acc);
    __syncthreads();           // the sums of the round before are read
#pragma unroll
    for (int t = 0; t < 2; ++t)
#pragma unroll
      for (int c = 0; c < 2; ++c) store4(&red[warp][t][c][lane * 4], make_float4(acc[t][c][0], acc[t][c][1], acc[t][c][2], acc[t][c][3]));
    __syncthreads();
    // element i of a 16 x 8 block: lane i / 4's value i % 4 = (row g + 8 (v >> 1), column 2 tq + (v & 1))
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      const int i = threadIdx.x, ln = i >> 2, v = i & 3;
      const int f = f0 + (ln >> 2) + 8 * (v >> 1), q = p0 + c * 8 + (ln & 3) * 2 + (v & 1);
      if (f >= F || q >= n) continue;
      const int pr = list[q];
      const float s = weight[pr];
      const float gt = ((red[0][0][c][i] + red[1][0][c][i]) + (red[2][0][c][i] + red[3][0][c][i])) * s;
      const float up = ((red[0][1][c][i] + red[1][1][c][i]) + (red[2][1][c][i] + red[3][1][c][i])) * s;
      act[(long long)pr * F + f] = __float2bfloat16(silu_f(gt) * up);
    }
  }
}

// y[p, d] = W_down[d, :] act[p, :] for the pairs of expert blockIdx.y; W [E][D][F]
__global__ void __launch_bounds__(128) expert_down_few_kernel(const bf16* __restrict__ act, const bf16* __restrict__ W,
                                                              const int* __restrict__ idx, float* __restrict__ y, int P, int D,
                                                              int F) {
  __shared__ int list[kFewPairs], count;
  __shared__ __align__(16) float red[4][2][128];
  const int e = blockIdx.y, d0 = blockIdx.x * 16;
  const int n = find_pairs(idx, P, e, list, &count);
  if (n == 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
  const bf16* we = W + (long long)e * D * F;
  const bf16* w[2] = {we + (long long)min(d0 + g, D - 1) * F, we + (long long)min(d0 + g + 8, D - 1) * F};
  for (int p0 = 0; p0 < n; p0 += 16) {
    const bf16* x[2];
#pragma unroll
    for (int c = 0; c < 2; ++c) x[c] = p0 + c * 8 + g < n ? act + (long long)list[p0 + c * 8 + g] * F : nullptr;
    float acc[1][2][4] = {};
    few_rows<1>(w, x, n - p0 > 8, F, warp, tq, acc);
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 2; ++c) store4(&red[warp][c][lane * 4], make_float4(acc[0][c][0], acc[0][c][1], acc[0][c][2], acc[0][c][3]));
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      const int i = threadIdx.x, ln = i >> 2, v = i & 3;
      const int d = d0 + (ln >> 2) + 8 * (v >> 1), q = p0 + c * 8 + (ln & 3) * 2 + (v & 1);
      if (d >= D || q >= n) continue;
      y[(long long)list[q] * D + d] = (red[0][c][i] + red[1][c][i]) + (red[2][c][i] + red[3][c][i]);
    }
  }
}

}  // namespace ob

using namespace ob;

extern "C" {

// h T [M, D], w fp32 [P], dest [P] (P = M * k) -> xs T [max_rows, D]
int ob_moe_gather(const void* h, const float* w, const int* dest, void* xs, long long P, int k, int D, int max_rows, int fp32,
                  cudaStream_t s) {
  if (P <= 0) return 0;
  if (k <= 0) return 6005;
  const bool vec = D % 8 == 0 && !((((uintptr_t)h) | ((uintptr_t)xs)) & 15);
#define OB_GATHER(T, V) moe_gather_kernel<T, V><<<(unsigned)P, 128, 0, s>>>((const T*)h, w, dest, (T*)xs, k, D, max_rows)
  if (fp32) { if (vec) OB_GATHER(float, true); else OB_GATHER(float, false); }
  else { if (vec) OB_GATHER(bf16, true); else OB_GATHER(bf16, false); }
#undef OB_GATHER
  OB_CHECK_LAUNCH();
  return 0;
}

// x fp32 [M, D] += the k rows of y (bf16 or fp32) of every token
int ob_moe_sum(const void* y, const int* dest, float* x, int M, int k, int D, int max_rows, int y_fp32, cudaStream_t s) {
  const bool vec = D % 4 == 0 && !((((uintptr_t)y) | ((uintptr_t)x)) & 15);
  for (int m0 = 0; m0 < M; m0 += 65535) {      // gridDim.y limit
    const int n = M - m0 < 65535 ? M - m0 : 65535;
    const dim3 grid((D + (vec ? 1023 : 255)) / (vec ? 1024 : 256), n);
    const int* d = dest ? dest + (long long)m0 * k : nullptr;
    const long long skip = dest ? 0 : (long long)m0 * k;
    float* xo = x + (long long)m0 * D;
    const int rows = max_rows - (int)skip;
#define OB_SUM(T, V) moe_sum_kernel<T, V><<<grid, 256, 0, s>>>((const T*)y + skip * D, d, xo, k, D, rows)
    if (y_fp32) { if (vec) OB_SUM(float, true); else OB_SUM(float, false); }
    else { if (vec) OB_SUM(bf16, true); else OB_SUM(bf16, false); }
#undef OB_SUM
    OB_CHECK_LAUNCH();
  }
  return 0;
}

// C T [max_rows, N] = rows of A T [max_rows, K], grouped by offsets [E + 1], times W T [E, N, K]
int ob_expert_rows_any(const void* A, const void* W, void* C, const int* offsets, int E, int N, int K, int max_rows, int fp32,
                       cudaStream_t s) {
  if (max_rows <= 0) return 0;
  if (E <= 0 || E > 65535) return 6001;
  const int blocks = (max_rows + 64 * E - 1) / (64 * E);      // row blocks of an average expert
  const dim3 grid((N + 63) / 64, E, blocks < 1 ? 1 : blocks > 64 ? 64 : blocks);
  if (fp32) expert_rows_any_kernel<float, float><<<grid, 256, 0, s>>>((const float*)A, (const float*)W, (float*)C, offsets, N, K, max_rows);
  else expert_rows_any_kernel<bf16, bf16><<<grid, 256, 0, s>>>((const bf16*)A, (const bf16*)W, (bf16*)C, offsets, N, K, max_rows);
  OB_CHECK_LAUNCH();
  return 0;
}

// Experts of P = M * k pairs, P <= 2048, bf16: h [M, D], idx / weight [P], gate_up [E, 2F, D], down [E, D, F];
// scratch act bf16 [P, F]; y fp32 [P, D].  D, F multiples of 8.
int ob_experts_few(const void* h, const int* idx, const float* weight, const void* gate_up, const void* down, void* act,
                   float* y, int P, int k, int E, int D, int F, cudaStream_t s) {
  if (P <= 0) return 0;
  if (P > kFewPairs || k <= 0 || E <= 0 || E > 65535) return 6005;
  if ((D & 7) || (F & 7)) return 6001;
  if ((((uintptr_t)h) | ((uintptr_t)gate_up) | ((uintptr_t)down) | ((uintptr_t)act)) & 15) return 6002;
  expert_up_few_kernel<<<dim3((F + 15) / 16, E), 128, 0, s>>>((const bf16*)h, (const bf16*)gate_up, idx, weight, (bf16*)act, P, k, F, D);
  OB_CHECK_LAUNCH();
  expert_down_few_kernel<<<dim3((D + 15) / 16, E), 128, 0, s>>>((const bf16*)act, (const bf16*)down, idx, y, P, D, F);
  OB_CHECK_LAUNCH();
  return 0;
}

}  // extern "C"
