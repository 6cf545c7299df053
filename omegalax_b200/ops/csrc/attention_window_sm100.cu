// Flash attention over packed prompts with a sliding window and a sink, grouped key/value heads and separate
// query/key and value widths (kernel: attention_fwd_sm100.cuh).
#include "attention_fwd_sm100.cuh"

using namespace ob;

extern "C" {

// Causal; forward only.  A query sees the last ``window`` tokens of its sequence up to itself (0: all).
//   q [rows, H, dim] (pitch q_row_stride)     k [rows, G, dim] (pitch k_row_stride)
//   v [rows, G, vdim] (pitch v_row_stride)    out [rows, H, vdim]    sink bf16 [H] or null
// Every width and pitch is a multiple of 8 elements.  Returns 6005 for widths without an instantiation
// (dim > 256 or vdim > 128).
int ob_attn_fwd_window(const void* q, const void* k, const void* v, void* out, const int* cu_seqlens, int B,
                       int max_seqlen, long long total_rows, int H, int G, int dim, int vdim, long long q_row_stride,
                       long long k_row_stride, long long v_row_stride, float scale, int window, const void* sink,
                       int* status, cudaStream_t stream) {
  if (B <= 0 || total_rows <= 0) return 0;
  if ((q_row_stride & 7) || (k_row_stride & 7) || (v_row_stride & 7) || (dim & 7) || (vdim & 7)) return 6001;
  if ((((uintptr_t)q) | ((uintptr_t)k) | ((uintptr_t)v) | ((uintptr_t)out)) & 15) return 6002;
  if (G <= 0 || H % G || window < 0) return 6005;
  AttnFwdArgs a = {};
  a.cu_seqlens = cu_seqlens;
  a.out = (bf16*)out;
  a.o_row_stride = (long long)H * vdim;
  a.total_rows = total_rows;
  a.H = H; a.G = G; a.causal = 1;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.nb1 = (dim + 63) / 64;
  a.vdim = vdim;
  a.window = window;
  a.sink = (const bf16*)sink;
  a.status = status;
  const int qb = a.nb1, vb = (vdim + 63) / 64;
  if (qb < 1 || qb > 4 || vb < 1 || vb > 2) return 6005;
  CUtensorMap tmQ, tmK, tmV;
  int e = make_tmap_3d(&tmQ, q, dim, H, total_rows, (uint64_t)dim * 2, (uint64_t)q_row_stride * 2, 64, 1, 128);
  if (e) return 2000 + e;
  e = make_tmap_3d(&tmK, k, dim, G, total_rows, (uint64_t)dim * 2, (uint64_t)k_row_stride * 2, 64, 1, 128);
  if (e) return 3000 + e;
  e = make_tmap_3d(&tmV, v, vdim, G, total_rows, (uint64_t)vdim * 2, (uint64_t)v_row_stride * 2, 64, 1, 128);
  if (e) return 3500 + e;
#define OB_WIN(Q, V, KS, VS) return run_attn_fwd<Q, V, KS, VS, true>(tmQ, tmK, tmV, tmQ, tmK, a, B, max_seqlen, stream)
  if (vb == 1) {
    if (qb == 1) OB_WIN(1, 1, 2, 2);
    if (qb == 2) OB_WIN(2, 1, 2, 2);
    if (qb == 3) OB_WIN(3, 1, 2, 2);
    if (qb == 4) OB_WIN(4, 1, 1, 2);
  } else {
    if (qb == 1) OB_WIN(1, 2, 2, 2);
    if (qb == 2) OB_WIN(2, 2, 2, 2);
    if (qb == 3) OB_WIN(3, 2, 2, 1);
    if (qb == 4) OB_WIN(4, 2, 1, 1);
  }
#undef OB_WIN
  return 6005;
}

}  // extern "C"
