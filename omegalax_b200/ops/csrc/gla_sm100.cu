// Gated linear attention with a decay per key channel, forward only, fp32 recurrence:
//
//   S_t = diag(alpha_t) S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t        (per head, S is [K, V])
//
// The recurrence is walked token by token with the state in registers.  In fp32 on CUDA cores the
// chunked form costs as many multiply-adds as the recurrence (the intra-chunk products replace the
// per-token ones), and the walk needs no quotients of decay products, so it is exact for any decay.
//
//   gla_decay_kernel   alpha = sigmoid(z + bias)^(1/tau) in place
//   gla_scan_kernel    packed sequences: CTA = (32 value columns, head, sequence); a thread owns KT key
//                      rows x 4 value columns of S (packed fp32 pairs); 16 lanes share a value quad and
//                      add their partial o
//   gla_step_kernel    one token per sequence: decay, state update, read-out, per-head RMS norm and
//                      silu gate in one launch; one pass over the state in memory
//   gla_norm_gate_kernel  per-head RMS norm of o, weight, times silu(g)
//
// q, k, v, g are column ranges of one projection row [q | k | v | g | ...] of pitch ldp.
#include "host_utils.h"
#include "serve_common.cuh"

namespace ob {

// grid (column quads, rows); a thread keeps its bias quad over the rows it walks.  VEC: C % 4 == 0.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) gla_decay_kernel(float* __restrict__ z, const T* __restrict__ bias, long long N, int C,
                                                        float inv_tau) {
  const int c = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (c >= C) return;
  float b[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) b[i] = c + i < C ? to_f(bias[c + i]) : 0.f;
#pragma unroll 2
  for (long long n = blockIdx.y; n < N; n += gridDim.y) {
    float* p = z + n * C + c;
    if (VEC) {
      float4 v = load4(p);
      v.x = expf(log_sigmoid(v.x + b[0]) * inv_tau);
      v.y = expf(log_sigmoid(v.y + b[1]) * inv_tau);
      v.z = expf(log_sigmoid(v.z + b[2]) * inv_tau);
      v.w = expf(log_sigmoid(v.w + b[3]) * inv_tau);
      store4(p, v);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (c + i < C) p[i] = expf(log_sigmoid(p[i] + b[i]) * inv_tau);
    }
  }
}

struct GlaScanArgs {
  const void* proj;        // T [N, ldp]
  const float* alpha;      // [N, H*K]
  float* o;                // [N, H, V]
  float* state;            // [slots, H, K, V]
  const int* cu;           // [B+1] packed rows of the sequences
  const int* history;      // [B] tokens before this call: 0 starts from a zero state
  long long ldp;
  int H, K, V;
  float q_scale;
};

// two fp32 values in one 64-bit register pair (packed fp32 arithmetic)
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t pair2(float lo, float hi) {
  return (uint64_t)__float_as_uint(lo) | ((uint64_t)__float_as_uint(hi) << 32);
}
__device__ __forceinline__ float lo2(uint64_t v) { return __uint_as_float((uint32_t)v); }
__device__ __forceinline__ float hi2(uint64_t v) { return __uint_as_float((uint32_t)(v >> 32)); }

// four consecutive elements as they lie in memory, kept unconverted while they are in flight
template <typename T>
struct Raw4;
template <>
struct Raw4<bf16> {
  uint2 u;
  __device__ __forceinline__ void load(const bf16* p) { u = *reinterpret_cast<const uint2*>(p); }
  __device__ __forceinline__ void set(int i, bf16 v) {
    const uint32_t b = (uint32_t)__bfloat16_as_ushort(v) << (16 * (i & 1));
    if (i < 2) u.x |= b; else u.y |= b;
  }
  __device__ __forceinline__ void zero() { u = make_uint2(0, 0); }
  __device__ __forceinline__ float4 get() const {
    const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
};
template <>
struct Raw4<float> {
  float4 u;
  __device__ __forceinline__ void load(const float* p) { u = *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ void set(int i, float v) { (&u.x)[i] = v; }
  __device__ __forceinline__ void zero() { u = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ float4 get() const { return u; }
};

// VEC: K, V, the pitch and every base are multiples of four elements.
// A thread's state pairs rows (k, k+1) of one value column.  Tokens are staged TC at a time (registers
// -> the other shared buffer while the current one is walked) and walked four at a time, so that the
// 16 partial sums of four tokens x four columns leave through one transposing reduction over 16 lanes.
template <typename T, int KT, bool VEC>
__global__ void __launch_bounds__(128) gla_scan_kernel(const GlaScanArgs p) {
  constexpr int KP = KT * 16;                 // padded key width
  constexpr int NJ = KT / 4;
  constexpr int TC = KT > 8 ? 8 : 16;         // tokens per stage
  constexpr int QN = TC * KP / 512;           // key quads per thread and stage
  constexpr int kA = 0, kK = TC * KP, kQ = 2 * TC * KP, kV = 3 * TC * KP, kBuf = 3 * TC * KP + TC * 64;
  extern __shared__ __align__(16) float sm[]; // 2 x { a[TC][KP], k[TC][KP], q[TC][KP], v[TC][32] doubled }
  const int b = blockIdx.z, h = blockIdx.y, v_base = blockIdx.x * 32;
  const int row0 = p.cu[b], len = p.cu[b + 1] - row0;
  if (len <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, kg = lane & 15;
  const int vq = ((tid >> 5) * 2 + (lane >> 4)) * 4;      // first of this thread's 4 columns in the slice
  const int K = p.K, V = p.V, HK = p.H * p.K;
  const T* proj = (const T*)p.proj + (long long)row0 * p.ldp;
  const float* alpha = p.alpha + (long long)row0 * HK + (long long)h * K;
  const int q_off = h * K, k_off = HK + h * K, v_off = 2 * HK + h * V;
  float* st = p.state + ((long long)b * p.H + h) * (long long)K * V;

  uint64_t S[KT / 2][4];
  const bool fresh = p.history[b] == 0;
#pragma unroll
  for (int r = 0; r < KT / 2; ++r) {
    const int k = (r >> 1) * 64 + kg * 4 + (r & 1) * 2;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int v = v_base + vq + c;
      const bool in = !fresh && v < V;
      S[r][c] = pair2(in && k < K ? st[(long long)k * V + v] : 0.f, in && k + 1 < K ? st[(long long)(k + 1) * V + v] : 0.f);
    }
  }

  float4 ra[QN];
  Raw4<T> rk[QN], rq[QN], rv;
  const int vt = tid >> 3, vk = (tid & 7) * 4;            // value quad of this thread: token vt, columns vk ..
  // Loads are unconditional at clamped places, so that all of a stage are in flight at once; what lies
  // past the end is replaced when the stage is written: decay 1 and zero key leave the state unchanged.
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < QN; ++i) {
      const int e = (tid + i * 128) * 4, t = min(t0 + e / KP, len - 1), k = e % KP;
      const float* ap = alpha + (long long)t * HK;
      const T* r = proj + (long long)t * p.ldp;
      if (VEC) {
        const int kc = min(k, K - 4);
        ra[i] = *reinterpret_cast<const float4*>(ap + kc);
        rk[i].load(r + k_off + kc);
        rq[i].load(r + q_off + kc);
      } else {
        rk[i].zero();
        rq[i].zero();
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int kc = min(k + c, K - 1);
          (&ra[i].x)[c] = ap[kc];
          rk[i].set(c, r[k_off + kc]);
          rq[i].set(c, r[q_off + kc]);
        }
      }
    }
    const T* r = proj + (long long)min(t0 + min(vt, TC - 1), len - 1) * p.ldp + v_off;
    if (VEC) {
      rv.load(r + min(v_base + vk, V - 4));
    } else {
      rv.zero();
#pragma unroll
      for (int c = 0; c < 4; ++c) rv.set(c, r[min(v_base + vk + c, V - 1)]);
    }
  };
  auto put = [&](float* buf, int t0) {
#pragma unroll
    for (int i = 0; i < QN; ++i) {
      const int e = (tid + i * 128) * 4, k = e % KP;
      const bool in = t0 + e / KP < len;
      const float4 kk = rk[i].get(), qq = rq[i].get();
      float4 a = ra[i], x = kk, y = make_float4(qq.x * p.q_scale, qq.y * p.q_scale, qq.z * p.q_scale, qq.w * p.q_scale);
#pragma unroll
      for (int c = 0; c < 4; ++c)
        if (!in || k + c >= K) {
          (&a.x)[c] = 1.f;
          (&x.x)[c] = 0.f;
          (&y.x)[c] = 0.f;
        }
      store4(buf + kA + e, a);
      store4(buf + kK + e, x);
      store4(buf + kQ + e, y);
    }
    if (vt < TC) {      // value columns past the end are computed and never stored
      const float4 v = rv.get();
      float* d = buf + kV + vt * 64 + vk * 2;
      store4(d, make_float4(v.x, v.x, v.y, v.y));
      store4(d + 4, make_float4(v.z, v.z, v.w, v.w));
    }
  };

  // this lane's place in the reduced 4 x 4 block: token (bits 8, 4), column (bits 2, 1)
  const bool b8 = kg & 8, b4 = kg & 4, b2 = kg & 2, b1 = kg & 1;
  const int my_t = (b8 ? 2 : 0) + (b4 ? 1 : 0), my_v = v_base + vq + (b2 ? 2 : 0) + (b1 ? 1 : 0);
  const long long o_stride = (long long)p.H * V;
  float* o = p.o + ((long long)row0 * p.H + h) * V + my_v + my_t * o_stride;
  const bool writer = my_v < V;

  fetch(0);
  put(sm, 0);
  __syncthreads();
  int cur = 0;
  for (int t0 = 0; t0 < len; t0 += TC) {
    const bool more = t0 + TC < len;
    if (more) fetch(t0 + TC);
    const float* buf = sm + cur * kBuf;
#pragma unroll 1
    for (int tb = 0; tb < TC; tb += 4) {
      float y[4][4];
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        const ulonglong2 v01 = *reinterpret_cast<const ulonglong2*>(buf + kV + (tb + t) * 64 + vq * 2);
        const ulonglong2 v23 = *reinterpret_cast<const ulonglong2*>(buf + kV + (tb + t) * 64 + vq * 2 + 4);
        const uint64_t vv[4] = {v01.x, v01.y, v23.x, v23.y};
        uint64_t acc[4] = {0, 0, 0, 0};
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const float* c = buf + (tb + t) * KP + j * 64 + kg * 4;
          const ulonglong2 a2 = *reinterpret_cast<const ulonglong2*>(c + kA), k2 = *reinterpret_cast<const ulonglong2*>(c + kK),
                           q2 = *reinterpret_cast<const ulonglong2*>(c + kQ);
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            S[2 * j][x] = fma2(a2.x, S[2 * j][x], mul2(k2.x, vv[x]));
            acc[x] = fma2(q2.x, S[2 * j][x], acc[x]);
            S[2 * j + 1][x] = fma2(a2.y, S[2 * j + 1][x], mul2(k2.y, vv[x]));
            acc[x] = fma2(q2.y, S[2 * j + 1][x], acc[x]);
          }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) y[t][x] = lo2(acc[x]) + hi2(acc[x]);
      }
      float y2[2][4], y3[4], y4[2];
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int x = 0; x < 4; ++x)
          y2[t][x] = (b8 ? y[t + 2][x] : y[t][x]) + __shfl_xor_sync(0xffffffffu, b8 ? y[t][x] : y[t + 2][x], 8);
#pragma unroll
      for (int x = 0; x < 4; ++x) y3[x] = (b4 ? y2[1][x] : y2[0][x]) + __shfl_xor_sync(0xffffffffu, b4 ? y2[0][x] : y2[1][x], 4);
#pragma unroll
      for (int x = 0; x < 2; ++x) y4[x] = (b2 ? y3[x + 2] : y3[x]) + __shfl_xor_sync(0xffffffffu, b2 ? y3[x] : y3[x + 2], 2);
      const float r = (b1 ? y4[1] : y4[0]) + __shfl_xor_sync(0xffffffffu, b1 ? y4[0] : y4[1], 1);
      if (writer && t0 + tb + my_t < len) o[(long long)(t0 + tb) * o_stride] = r;
    }
    if (more) {
      cur ^= 1;
      put(sm + cur * kBuf, t0 + TC);     // the other buffer: its readers finished before the last barrier
      __syncthreads();
    }
  }
#pragma unroll
  for (int r = 0; r < KT / 2; ++r) {
    const int k = (r >> 1) * 64 + kg * 4 + (r & 1) * 2;
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int v = v_base + vq + c;
      if (v < V && k < K) st[(long long)k * V + v] = lo2(S[r][c]);
      if (v < V && k + 1 < K) st[(long long)(k + 1) * V + v] = hi2(S[r][c]);
    }
  }
}

// one warp per (row, head)
template <typename T>
__global__ void gla_norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ g, long long ldg,
                                     const T* __restrict__ w, T* __restrict__ out, long long rows, int H, int V, float eps,
                                     bool vec) {
  const int lane = threadIdx.x & 31;
  const long long wid = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  if (wid >= rows * H) return;
  const long long n = wid / H;
  const int h = (int)(wid - n * H);
  const float* orow = o + wid * V;
  const T* grow = g + n * ldg + (long long)h * V;
  T* dst = out + wid * V;
  float ss = 0.f;
  if (vec) {     // V = 128: one vector per lane
    const float4 x = load4(orow + lane * 4), gg = load4(grow + lane * 4), ww = load4(w + lane * 4);
    ss = (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)V + eps);
    store4(dst + lane * 4, make_float4(x.x * r * ww.x * silu_f(gg.x), x.y * r * ww.y * silu_f(gg.y),
                                       x.z * r * ww.z * silu_f(gg.z), x.w * r * ww.w * silu_f(gg.w)));
    return;
  }
  for (int v = lane; v < V; v += 32) ss += orow[v] * orow[v];
  const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)V + eps);
  for (int v = lane; v < V; v += 32) dst[v] = from_f<T>(orow[v] * rstd * to_f(w[v]) * silu_f(to_f(grow[v])));
}

struct GlaStepArgs {
  const void* proj;        // T [B, ldp]
  const float* z;          // [B, H*K] decay logits without bias
  const void* bias;        // T [H*K]
  const void* norm_w;      // T [V]
  void* out;               // T [B, H*V]
  float* state;            // [slots, H, K, V], slot = row
  const int* active;       // [B] tokens visible after this step; 0: row without a token
  long long ldp;
  int H, K, V;
  float q_scale, inv_tau, eps;
};

// CTA = (head, sequence), 256 threads as R rows x (V / VW) column groups; VW = 4 needs V % 4 == 0.
template <typename T, int VW>
__global__ void __launch_bounds__(256) gla_step_kernel(const GlaStepArgs p) {
  extern __shared__ float sm[];     // a[K], k[K], q[K], v[V], part[R*V]
  __shared__ float red[33];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int K = p.K, V = p.V, HK = p.H * K;
  T* out = (T*)p.out + ((long long)b * p.H + h) * V;
  const int seen = p.active[b];
  if (seen <= 0) {
    for (int v = tid; v < V; v += 256) out[v] = from_f<T>(0.f);
    return;
  }
  const bool fresh = seen == 1;
  const T* row = (const T*)p.proj + (long long)b * p.ldp;
  float *sa = sm, *sk = sm + K, *sq = sm + 2 * K, *sv = sm + 3 * K, *part = sv + V;
  for (int k = tid; k < K; k += 256) {
    const int c = h * K + k;
    sa[k] = expf(log_sigmoid(p.z[(long long)b * HK + c] + to_f(((const T*)p.bias)[c])) * p.inv_tau);
    sk[k] = to_f(row[HK + c]);
    sq[k] = to_f(row[c]) * p.q_scale;
  }
  for (int v = tid; v < V; v += 256) sv[v] = to_f(row[2 * HK + h * V + v]);
  __syncthreads();
  const int ncol = V / VW, R = max(256 / ncol, 1);
  float* st = p.state + ((long long)b * p.H + h) * (long long)K * V;
  for (int c0 = 0; c0 < ncol; c0 += 256) {               // one trip unless V / VW > 256
    const int r = tid / ncol, c = c0 + (ncol > 256 ? tid : tid - r * ncol);
    if ((ncol > 256 || r < R) && c < ncol) {
      float acc[VW], vv[VW];
#pragma unroll
      for (int i = 0; i < VW; ++i) { acc[i] = 0.f; vv[i] = sv[c * VW + i]; }
      const int r0 = ncol > 256 ? 0 : r;
      for (int kb = r0; kb < K; kb += 8 * R) {
        float x[8][VW];
#pragma unroll
        for (int u = 0; u < 8; ++u) {      // eight state rows in flight before any arithmetic
          const float* s = st + (long long)min(kb + u * R, K - 1) * V + c * VW;
          if (VW == 4) *reinterpret_cast<float4*>(x[u]) = *reinterpret_cast<const float4*>(s);
          else x[u][0] = s[0];
        }
        if (fresh) {
#pragma unroll
          for (int u = 0; u < 8; ++u)
#pragma unroll
            for (int i = 0; i < VW; ++i) x[u][i] = 0.f;
        }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const int k = kb + u * R;
          if (k >= K) break;
          float* s = st + (long long)k * V + c * VW;
          const float a = sa[k], kk = sk[k], qq = sq[k];
#pragma unroll
          for (int i = 0; i < VW; ++i) {
            x[u][i] = fmaf(a, x[u][i], kk * vv[i]);
            acc[i] = fmaf(qq, x[u][i], acc[i]);
          }
          if (VW == 4) *reinterpret_cast<float4*>(s) = *reinterpret_cast<float4*>(x[u]);
          else s[0] = x[u][0];
        }
      }
#pragma unroll
      for (int i = 0; i < VW; ++i) part[(ncol > 256 ? 0 : r) * V + c * VW + i] = acc[i];
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int v = tid; v < V; v += 256) {
    float o = part[v];
    for (int r = 1; r < R; ++r) o += part[r * V + v];
    part[v] = o;              // only this thread touches column v
    ss += o * o;
  }
  const float rstd = 1.f / sqrtf(block_sum<256>(ss, red) / (float)V + p.eps);
  const T* g = row + 2 * HK + p.H * V + h * V;
  for (int v = tid; v < V; v += 256)
    out[v] = from_f<T>(part[v] * rstd * to_f(((const T*)p.norm_w)[v]) * silu_f(to_f(g[v])));
}

template <typename T, int KT, bool VEC>
static int run_scan(const GlaScanArgs& a, int B, cudaStream_t s) {
  constexpr int TC = KT > 8 ? 8 : 16, smem = 2 * (3 * TC * KT * 16 + TC * 64) * 4;
  auto kern = gla_scan_kernel<T, KT, VEC>;
  OB_ENSURE_DYN_SMEM(kern, smem);
  kern<<<dim3((a.V + 31) / 32, a.H, B), 128, smem, s>>>(a);
  OB_CHECK_LAUNCH();
  return 0;
}

template <typename T>
static int launch_scan(const GlaScanArgs& a, int B, cudaStream_t s) {
  const bool vec = !((a.K | a.V | (int)(a.ldp & 3)) & 3) && !(((uintptr_t)a.proj | (uintptr_t)a.alpha) & 15);
#define OB_SCAN(KT) return vec ? run_scan<T, KT, true>(a, B, s) : run_scan<T, KT, false>(a, B, s)
  if (a.K <= 64) OB_SCAN(4);
  if (a.K <= 128) OB_SCAN(8);
  if (a.K <= 256) OB_SCAN(16);
#undef OB_SCAN
  return 6005;
}

template <typename T>
static int launch_step(const GlaStepArgs& a, int B, cudaStream_t s) {
  dim3 grid(a.H, B);
  const int vw = a.V % 4 == 0 ? 4 : 1;
  const int ncol = a.V / vw, R = 256 / ncol > 1 ? 256 / ncol : 1;
  const int smem = (3 * a.K + a.V + R * a.V) * 4;
  if (smem > 48 * 1024) return 6005;
  if (vw == 4) gla_step_kernel<T, 4><<<grid, 256, smem, s>>>(a);
  else gla_step_kernel<T, 1><<<grid, 256, smem, s>>>(a);
  OB_CHECK_LAUNCH();
  return 0;
}

}  // namespace ob

using namespace ob;

extern "C" {

int ob_gla_decay(float* z, const void* bias, long long N, int C, float inv_tau, int fp32, cudaStream_t s) {
  if (N <= 0) return 0;
  const int gx = (C + 1023) / 1024;
  const long long cap = (long long)num_sms() * 16 / gx + 1;
  const dim3 grid(gx, (unsigned)(N < cap ? N : cap));
  const bool vec = C % 4 == 0 && !((uintptr_t)z & 15);
  if (fp32) {
    if (vec) gla_decay_kernel<float, true><<<grid, 256, 0, s>>>(z, (const float*)bias, N, C, inv_tau);
    else gla_decay_kernel<float, false><<<grid, 256, 0, s>>>(z, (const float*)bias, N, C, inv_tau);
  } else {
    if (vec) gla_decay_kernel<bf16, true><<<grid, 256, 0, s>>>(z, (const bf16*)bias, N, C, inv_tau);
    else gla_decay_kernel<bf16, false><<<grid, 256, 0, s>>>(z, (const bf16*)bias, N, C, inv_tau);
  }
  OB_CHECK_LAUNCH();
  return 0;
}

int ob_gla_scan(const void* proj, long long ldp, const float* alpha, float* o, float* state, const int* cu,
                const int* history, int B, int H, int K, int V, float q_scale, int fp32, cudaStream_t s) {
  if (B <= 0) return 0;
  GlaScanArgs a = {proj, alpha, o, state, cu, history, ldp, H, K, V, q_scale};
  return fp32 ? launch_scan<float>(a, B, s) : launch_scan<bf16>(a, B, s);
}

int ob_gla_norm_gate(const float* o, const void* g, long long ldg, const void* w, void* out, long long rows, int H,
                     int V, float eps, int fp32, cudaStream_t s) {
  if (rows <= 0) return 0;
  const unsigned grid = (unsigned)((rows * H * 32 + 255) / 256);
  const bool vec = V == 128 && ldg % 4 == 0 && !(((uintptr_t)g | (uintptr_t)o | (uintptr_t)w) & 15);
  if (fp32)
    gla_norm_gate_kernel<float><<<grid, 256, 0, s>>>(o, (const float*)g, ldg, (const float*)w, (float*)out, rows, H, V, eps, vec);
  else
    gla_norm_gate_kernel<bf16><<<grid, 256, 0, s>>>(o, (const bf16*)g, ldg, (const bf16*)w, (bf16*)out, rows, H, V, eps, vec);
  OB_CHECK_LAUNCH();
  return 0;
}

int ob_gla_step(const void* proj, long long ldp, const float* z, const void* bias, const void* norm_w, void* out,
                float* state, const int* active, int B, int H, int K, int V, float q_scale, float inv_tau, float eps,
                int fp32, cudaStream_t s) {
  if (B <= 0) return 0;
  GlaStepArgs a = {proj, z, bias, norm_w, out, state, active, ldp, H, K, V, q_scale, inv_tau, eps};
  return fp32 ? launch_step<float>(a, B, s) : launch_step<bf16>(a, B, s);
}

}  // extern "C"
