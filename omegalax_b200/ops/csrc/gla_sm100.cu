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
//                      rows x 4 value columns of S; 16 lanes share a value quad and add their partial o
//   gla_step_kernel    one token per sequence: decay, state update, read-out, per-head RMS norm and
//                      silu gate in one launch; one pass over the state in memory
//   gla_norm_gate_kernel  per-head RMS norm of o, weight, times silu(g)
//
// q, k, v, g are column ranges of one projection row [q | k | v | g | ...] of pitch ldp.
#include "host_utils.h"
#include "serve_common.cuh"

namespace ob {

template <typename T>
__global__ void gla_decay_kernel(float* __restrict__ z, const T* __restrict__ bias, long long n, int C, float inv_tau) {
  const long long stride = (long long)gridDim.x * blockDim.x;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += stride)
    z[i] = expf(log_sigmoid(z[i] + to_f(bias[i % C])) * inv_tau);
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

constexpr int kScanTok = 8;     // tokens staged at a time

template <typename T, int KT>
__global__ void __launch_bounds__(128) gla_scan_kernel(const GlaScanArgs p) {
  constexpr int KP = KT * 16;                 // padded key width
  constexpr int NJ = KT / 4;
  extern __shared__ float sm[];               // 2 x { a[8][KP], k[8][KP], q[8][KP], v[8][32] }
  constexpr int kBuf = kScanTok * (3 * KP + 32);
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

  float S[KT][4];
  const bool fresh = p.history[b] == 0;
#pragma unroll
  for (int j = 0; j < NJ; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = j * 64 + kg * 4 + i;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int v = v_base + vq + c;
        S[j * 4 + i][c] = (!fresh && k < K && v < V) ? st[(long long)k * V + v] : 0.f;
      }
    }

  float ra[KT], rk[KT], rq[KT], rv[2];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < KT; ++i) {
      const int e = tid + i * 128, t = t0 + e / KP, k = e % KP;
      const bool in = t < len && k < K;
      const long long r = (long long)t * p.ldp;
      ra[i] = in ? alpha[(long long)t * HK + k] : 0.f;
      rk[i] = in ? to_f(proj[r + k_off + k]) : 0.f;
      rq[i] = in ? to_f(proj[r + q_off + k]) * p.q_scale : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int e = tid + i * 128, t = t0 + (e >> 5), v = v_base + (e & 31);
      rv[i] = (t < len && v < V) ? to_f(proj[(long long)t * p.ldp + v_off + v]) : 0.f;
    }
  };
  auto put = [&](float* buf) {
#pragma unroll
    for (int i = 0; i < KT; ++i) {
      const int e = tid + i * 128;
      buf[e] = ra[i];
      buf[kScanTok * KP + e] = rk[i];
      buf[2 * kScanTok * KP + e] = rq[i];
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) buf[3 * kScanTok * KP + tid + i * 128] = rv[i];
  };

  const bool hi8 = kg & 8, hi4 = kg & 4;
  const int my_v = v_base + vq + (hi8 ? 2 : 0) + (hi4 ? 1 : 0);
  const bool writer = (kg & 3) == 0 && my_v < V;
  float* o = p.o + ((long long)row0 * p.H + h) * V + my_v;
  const long long o_stride = (long long)p.H * V;

  fetch(0);
  put(sm);
  __syncthreads();
  int cur = 0;
  for (int t0 = 0; t0 < len; t0 += kScanTok) {
    const bool more = t0 + kScanTok < len;
    if (more) fetch(t0 + kScanTok);
    const float* buf = sm + cur * kBuf;
    const int nt = min(kScanTok, len - t0);
#pragma unroll 2
    for (int t = 0; t < nt; ++t) {
      const float4 vv = load4(buf + 3 * kScanTok * KP + t * 32 + vq);
      float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int c = t * KP + j * 64 + kg * 4;
        const float4 a4 = load4(buf + c), k4 = load4(buf + kScanTok * KP + c), q4 = load4(buf + 2 * kScanTok * KP + c);
        const float aa[4] = {a4.x, a4.y, a4.z, a4.w}, kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          float* s = S[j * 4 + i];
          s[0] = fmaf(aa[i], s[0], kk[i] * vv.x); o0 = fmaf(qq[i], s[0], o0);
          s[1] = fmaf(aa[i], s[1], kk[i] * vv.y); o1 = fmaf(qq[i], s[1], o1);
          s[2] = fmaf(aa[i], s[2], kk[i] * vv.z); o2 = fmaf(qq[i], s[2], o2);
          s[3] = fmaf(aa[i], s[3], kk[i] * vv.w); o3 = fmaf(qq[i], s[3], o3);
        }
      }
      // sum of four values over 16 lanes: halve the set twice, then two plain exchanges
      float x0 = hi8 ? o2 : o0, x1 = hi8 ? o3 : o1;
      x0 += __shfl_xor_sync(0xffffffffu, hi8 ? o0 : o2, 8);
      x1 += __shfl_xor_sync(0xffffffffu, hi8 ? o1 : o3, 8);
      float y = hi4 ? x1 : x0;
      y += __shfl_xor_sync(0xffffffffu, hi4 ? x0 : x1, 4);
      y += __shfl_xor_sync(0xffffffffu, y, 2);
      y += __shfl_xor_sync(0xffffffffu, y, 1);
      if (writer) o[(long long)(t0 + t) * o_stride] = y;
    }
    if (more) {
      cur ^= 1;
      put(sm + cur * kBuf);     // the other buffer: its readers finished before the last barrier
      __syncthreads();
    }
  }
#pragma unroll
  for (int j = 0; j < NJ; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = j * 64 + kg * 4 + i;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int v = v_base + vq + c;
        if (k < K && v < V) st[(long long)k * V + v] = S[j * 4 + i][c];
      }
    }
}

// one warp per (row, head)
template <typename T>
__global__ void gla_norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ g, long long ldg,
                                     const T* __restrict__ w, T* __restrict__ out, long long rows, int H, int V, float eps) {
  const int lane = threadIdx.x & 31;
  const long long wid = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  if (wid >= rows * H) return;
  const long long n = wid / H;
  const int h = (int)(wid - n * H);
  const float* orow = o + wid * V;
  const T* grow = g + n * ldg + (long long)h * V;
  T* dst = out + wid * V;
  float ss = 0.f;
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
#pragma unroll 8
      for (int k = r0; k < K; k += R) {
        float* s = st + (long long)k * V + c * VW;
        const float a = sa[k], kk = sk[k], qq = sq[k];
        float x[VW];
        if (fresh) {
#pragma unroll
          for (int i = 0; i < VW; ++i) x[i] = 0.f;
        } else if (VW == 4) {
          *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(s);
        } else {
          x[0] = s[0];
        }
#pragma unroll
        for (int i = 0; i < VW; ++i) {
          x[i] = fmaf(a, x[i], kk * vv[i]);
          acc[i] = fmaf(qq, x[i], acc[i]);
        }
        if (VW == 4) *reinterpret_cast<float4*>(s) = *reinterpret_cast<float4*>(x);
        else s[0] = x[0];
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

template <typename T>
static int launch_scan(const GlaScanArgs& a, int B, cudaStream_t s) {
  dim3 grid((a.V + 31) / 32, a.H, B);
#define OB_SCAN(KT)                                                                    \
  do {                                                                                 \
    auto kern = gla_scan_kernel<T, KT>;                                                \
    constexpr int smem = 2 * kScanTok * (3 * KT * 16 + 32) * 4;                        \
    OB_ENSURE_DYN_SMEM(kern, smem);                                                    \
    kern<<<grid, 128, smem, s>>>(a);                                                   \
  } while (0)
  if (a.K <= 64) OB_SCAN(4);
  else if (a.K <= 128) OB_SCAN(8);
  else if (a.K <= 256) OB_SCAN(16);
  else return 6005;
#undef OB_SCAN
  OB_CHECK_LAUNCH();
  return 0;
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
  const long long n = N * C, blocks = (n + 255) / 256, cap = (long long)num_sms() * 16;
  const unsigned grid = (unsigned)(blocks < cap ? blocks : cap);
  if (fp32) gla_decay_kernel<float><<<grid, 256, 0, s>>>(z, (const float*)bias, n, C, inv_tau);
  else gla_decay_kernel<bf16><<<grid, 256, 0, s>>>(z, (const bf16*)bias, n, C, inv_tau);
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
  if (fp32)
    gla_norm_gate_kernel<float><<<grid, 256, 0, s>>>(o, (const float*)g, ldg, (const float*)w, (float*)out, rows, H, V, eps);
  else
    gla_norm_gate_kernel<bf16><<<grid, 256, 0, s>>>(o, (const bf16*)g, ldg, (const bf16*)w, (bf16*)out, rows, H, V, eps);
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
