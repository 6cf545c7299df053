// K3 forward: GQA flash attention with 64-, 128- and 256-wide heads (kernel: attention_fwd_sm100.cuh).
#include "attention_fwd_sm100.cuh"

namespace ob {

template <int HD>
static int launch_attn_fwd(const void* q, const void* k, const void* v, AttnFwdArgs a,
                           long long q_row_stride, long long k_row_stride, long long v_row_stride,
                           int B, int max_seqlen, cudaStream_t stream) {
  CUtensorMap tmQ, tmK, tmV;
  int e = make_tmap_3d(&tmQ, q, HD, a.H, a.total_rows, (uint64_t)HD * 2, (uint64_t)q_row_stride * 2,
                       64, 1, 128);
  if (e) return 2000 + e;
  e = make_tmap_3d(&tmK, k, HD, a.G, a.total_rows, (uint64_t)HD * 2, (uint64_t)k_row_stride * 2, 64,
                   1, 128);
  if (e) return 3000 + e;
  e = make_tmap_3d(&tmV, v, HD, a.G, a.total_rows, (uint64_t)HD * 2, (uint64_t)v_row_stride * 2, 64,
                   1, 128);
  if (e) return 3500 + e;
  a.nb1 = HD / 64;
  a.vdim = HD;
  return run_attn_fwd<HD / 64, HD / 64, 2, 2>(tmQ, tmK, tmV, tmQ, tmK, a, B, max_seqlen, stream);
}

// attention_fwd256_sm100.cu
int launch_attn_fwd256(const void* q, const void* k, const void* v, void* out, float* lse, const int* cu_seqlens, int B,
                       int max_seqlen, long long total_rows, int H, int G, long long q_row_stride,
                       long long k_row_stride, long long v_row_stride, long long o_row_stride, float scale, int causal,
                       int* status, cudaStream_t stream);

}  // namespace ob

using namespace ob;

extern "C" {

// q/out: [total_rows, H, HD]; k, v: [total_rows, G, HD]; row strides in elements.
// cu_seqlens: device int32 [B+1].  lse: [H, total_rows] fp32 (may be null).
int ob_attn_fwd(const void* q, const void* k, const void* v, void* out, float* lse,
                const int* cu_seqlens, int B, int max_seqlen, long long total_rows, int H, int G,
                int HD, long long q_row_stride, long long k_row_stride, long long v_row_stride,
                long long o_row_stride, float scale, int causal, int* status,
                cudaStream_t stream) {
  if (B <= 0 || total_rows <= 0) return 0;
  if ((q_row_stride & 7) || (k_row_stride & 7) || (v_row_stride & 7) || (o_row_stride & 7))
    return 6001;
  if ((((uintptr_t)q) | ((uintptr_t)k) | ((uintptr_t)v) | ((uintptr_t)out)) & 15) return 6002;
  AttnFwdArgs a = {};
  a.cu_seqlens = cu_seqlens;
  a.out = (bf16*)out;
  a.o_row_stride = o_row_stride;
  a.lse = lse;
  a.total_rows = total_rows;
  a.H = H; a.G = G; a.causal = causal;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.status = status;
  if (HD == 128)
    return launch_attn_fwd<128>(q, k, v, a, q_row_stride, k_row_stride, v_row_stride, B, max_seqlen,
                                stream);
  if (HD == 64)
    return launch_attn_fwd<64>(q, k, v, a, q_row_stride, k_row_stride, v_row_stride, B, max_seqlen,
                               stream);
  if (HD == 256)
    return launch_attn_fwd256(q, k, v, out, lse, cu_seqlens, B, max_seqlen, total_rows, H, G, q_row_stride,
                              k_row_stride, v_row_stride, o_row_stride, scale, causal, status, stream);
  return 6005;
}

}  // extern "C"
