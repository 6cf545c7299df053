// Flash attention whose heads are made of two parts, for the prompts of latent attention
// (kernel: attention_fwd_sm100.cuh).
#include "attention_fwd_sm100.cuh"

using namespace ob;

extern "C" {

// Causal attention whose heads have a first part of d1 channels (own key per head) and a second part
// of d2 channels (one key for all heads), and vdim value channels; forward only.
//   q  [rows, H, d1 + d2] (pitch q_row_stride)       out [rows, H, vdim]
//   k1 [rows, H, d1] (pitch k_row_stride)            v   [rows, H, vdim] (pitch v_row_stride)
//   k2 [rows, d2] (pitch k2_row_stride)
// Every width and pitch is a multiple of 8 elements.  Returns 6005 for widths without an instantiation
// (ceil(d1/64) + ceil(d2/64) > 4, or vdim > 128).
int ob_attn_fwd_two_part(const void* q, const void* k1, const void* k2, const void* v, void* out, const int* cu_seqlens,
                         int B, int max_seqlen, long long total_rows, int H, int d1, int d2, int vdim,
                         long long q_row_stride, long long k_row_stride, long long k2_row_stride, long long v_row_stride,
                         float scale, int* status, cudaStream_t stream) {
  if (B <= 0 || total_rows <= 0) return 0;
  if ((q_row_stride & 7) || (k_row_stride & 7) || (k2_row_stride & 7) || (v_row_stride & 7) || (d1 & 7) || (d2 & 7) || (vdim & 7))
    return 6001;
  if ((((uintptr_t)q) | ((uintptr_t)k1) | ((uintptr_t)k2) | ((uintptr_t)v) | ((uintptr_t)out)) & 15) return 6002;
  AttnFwdArgs a = {};
  a.cu_seqlens = cu_seqlens;
  a.out = (bf16*)out;
  a.o_row_stride = (long long)H * vdim;
  a.total_rows = total_rows;
  a.H = H; a.G = H; a.causal = 1;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.nb1 = (d1 + 63) / 64;
  a.vdim = vdim;
  a.status = status;
  const int qb = a.nb1 + (d2 + 63) / 64, vb = (vdim + 63) / 64;
  if (qb > 4 || vb > 2) return 6005;
  const uint64_t head_bytes = (uint64_t)(d1 + d2) * 2;
  CUtensorMap tmQ, tmK, tmV, tmQ2, tmK2;
  int e = make_tmap_3d(&tmQ, q, d1, H, total_rows, head_bytes, (uint64_t)q_row_stride * 2, 64, 1, 128);
  if (!e) e = make_tmap_3d(&tmQ2, (const bf16*)q + d1, d2, H, total_rows, head_bytes, (uint64_t)q_row_stride * 2, 64, 1, 128);
  if (e) return 2000 + e;
  e = make_tmap_3d(&tmK, k1, d1, H, total_rows, (uint64_t)d1 * 2, (uint64_t)k_row_stride * 2, 64, 1, 128);
  if (!e) e = make_tmap_3d(&tmK2, k2, d2, 1, total_rows, (uint64_t)k2_row_stride * 2, (uint64_t)k2_row_stride * 2, 64, 1, 128);
  if (e) return 3000 + e;
  e = make_tmap_3d(&tmV, v, vdim, H, total_rows, (uint64_t)vdim * 2, (uint64_t)v_row_stride * 2, 64, 1, 128);
  if (e) return 3500 + e;
#define OB_TP(Q, V, KS, VS) return run_attn_fwd<Q, V, KS, VS>(tmQ, tmK, tmV, tmQ2, tmK2, a, B, max_seqlen, stream)
  if (vb == 1) {
    if (qb == 2) OB_TP(2, 1, 2, 2);
    if (qb == 3) OB_TP(3, 1, 2, 2);
    if (qb == 4) OB_TP(4, 1, 1, 2);
  } else {
    if (qb == 2) OB_TP(2, 2, 2, 2);
    if (qb == 3) OB_TP(3, 2, 2, 1);
    if (qb == 4) OB_TP(4, 2, 1, 1);
  }
#undef OB_TP
  return 6005;
}

}  // extern "C"
