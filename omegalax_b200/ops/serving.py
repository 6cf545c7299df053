"""Forward-only ops of decoders with an fp32 residual stream: norm rows, squared-relu and gated
activations, gated linear attention, latent attention over a paged latent cache, windowed grouped-query
attention over paged keys and values, routed experts, soft-capped logits.

Tensors are CUDA bf16 or fp32 (``T`` below: one type per call); the fp32 form of every kernel is
exact single precision and its matrix products are cuBLAS SGEMMs.  There is no CPU implementation.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from . import kernels as K
from . import lib

bf16, f32 = torch.bfloat16, torch.float32


def _fp32(t: torch.Tensor) -> int:
    if not t.is_cuda:
        raise RuntimeError("this op runs on CUDA tensors only")
    if t.dtype == f32:
        return 1
    if t.dtype == bf16:
        return 0
    raise TypeError(f"bf16 or fp32 expected, got {t.dtype}")


def _same(*ts) -> int:
    kind = _fp32(ts[0])
    for t in ts[1:]:
        if t is not None and (t.dtype != ts[0].dtype or not t.is_cuda):
            raise TypeError(f"operands differ in dtype or device: {[(x.dtype, x.device) for x in ts if x is not None]}")
    return kind


def _contig(*ts) -> None:
    for t in ts:
        if t is not None and not t.is_contiguous():
            raise ValueError("contiguous tensor expected")


# ----------------------------------------------------------------------------------------------- products
def project(x, w, *, out_dtype=None, into=None):
    """x [M, K] @ w [N, K]^T in ``out_dtype`` (default: that of x), or added into the fp32 rows
    ``into``.  bf16 products run on the tcgen05 GEMM; sizes it cannot address are zero-padded."""
    if _same(x, w):
        if into is not None:
            return into.addmm_(x, w.t())
        return x @ w.t()
    N, Kd = w.shape
    if Kd % 8:
        x, w = F.pad(x, (0, 8 - Kd % 8)), F.pad(w, (0, 8 - Kd % 8))
    if into is not None:
        if N % 8 == 0:
            return K.gemm(x, w, out=into, accumulate=True)
        return into.add_(project(x, w, out_dtype=f32))
    if N % 8:
        w = F.pad(w, (0, 0, 0, 8 - N % 8))
    y = K.gemm(x, w, out_dtype=out_dtype or bf16)
    return y[:, :N] if N % 8 else y


# ----------------------------------------------------------------------------------------------- row ops
def embed_rows(ids32, table):
    """fp32 rows of ``table``; id -1 gives a zero row, any other id outside the table an error status."""
    n, (V, D) = ids32.numel(), table.shape
    _contig(ids32, table)
    out = torch.empty(n, D, dtype=f32, device=table.device)
    K._call("ob_embed_rows", ids32.data_ptr(), table.data_ptr(), out.data_ptr(), n, V, D, _fp32(table),
            lib.status_tensor(table.device).data_ptr(), lib.stream_ptr())
    return out


def layernorm_rows(x, w, b, eps: float):
    """fp32 rows -> layer norm with weight and bias in the dtype of the weights."""
    kind = _same(w, b)
    if x.dtype != f32:
        raise TypeError("layernorm_rows reads fp32 rows")
    _contig(x, w, b)
    y = torch.empty(x.shape, dtype=w.dtype, device=x.device)
    K._call("ob_ln_rows", x.data_ptr(), w.data_ptr(), b.data_ptr(), y.data_ptr(), x.shape[0], x.shape[1], float(eps), kind,
            lib.stream_ptr())
    return y


def rms_rows(x, w, eps: float):
    """fp32 rows -> RMS norm times w, in the dtype of w."""
    kind = _fp32(w)
    if x.dtype != f32:
        raise TypeError("rms_rows reads fp32 rows")
    _contig(x, w)
    y = torch.empty(x.shape, dtype=w.dtype, device=x.device)
    K._call("ob_rms_rows", x.data_ptr(), w.data_ptr(), y.data_ptr(), x.shape[0], x.shape[1], float(eps), kind, lib.stream_ptr())
    return y


GATES = {"silu": 0, "gelu_tanh": 1}


def gated_act(gu, act: str, rows=None):
    """gu [M, 2F] = [gate | up] -> act(gate) * up [M, F].  ``rows`` (int32 [1] on the device): only that
    many rows hold anything."""
    _contig(gu)
    M, F2 = gu.shape
    y = torch.empty(M, F2 // 2, dtype=gu.dtype, device=gu.device)
    K._call("ob_gated_act", gu.data_ptr(), y.data_ptr(), lib.ptr(rows), M, F2 // 2, GATES[act], _fp32(gu), lib.stream_ptr())
    return y


def relu_squared(x):
    _contig(x)
    y = torch.empty_like(x)
    K._call("ob_relu_sq", x.data_ptr(), y.data_ptr(), x.numel(), _fp32(x), lib.stream_ptr())
    return y


def soft_cap_(x, cap: float):
    """cap * tanh(x / cap) in place on fp32."""
    if x.dtype != f32 or not x.is_cuda:
        raise TypeError("soft_cap_ works on CUDA fp32")
    _contig(x)
    K._call("ob_soft_cap", x.data_ptr(), x.numel(), float(cap), lib.stream_ptr())
    return x


# ----------------------------------------------------------------------------------------------- gated linear attention
def gla_decay_(z, bias, tau: float):
    """fp32 decay logits [N, C] -> sigmoid(z + bias)^(1/tau), in place."""
    _contig(z, bias)
    if z.dtype != f32 or bias.numel() != z.shape[1]:
        raise ValueError("decay logits are fp32 [N, C] with a bias of C")
    K._call("ob_gla_decay", z.data_ptr(), bias.data_ptr(), z.shape[0], z.shape[1], 1.0 / float(tau), _fp32(bias),
            lib.stream_ptr())
    return z


def gla_scan(proj, alpha, state, cu, history, H: int, Kd: int, V: int, q_scale: float):
    """Walk packed sequences: ``proj`` rows [q | k | v | ...] (T, any pitch), ``alpha`` fp32 [N, H*K],
    ``state`` fp32 [>=B, H, K, V] read where ``history`` > 0 and rewritten.  Returns fp32 [N, H, V]."""
    _contig(alpha, state, cu, history)
    if Kd > 256:
        raise ValueError("key heads wider than 256 channels are not supported")
    N, B = alpha.shape[0], history.numel()
    if proj.stride(1) != 1 or proj.shape[0] < N or state.shape[0] < B or tuple(state.shape[1:]) != (H, Kd, V):
        raise ValueError("projection or state does not fit the sequences")
    o = torch.empty(N, H, V, dtype=f32, device=proj.device)
    K._call("ob_gla_scan", proj.data_ptr(), proj.stride(0), alpha.data_ptr(), o.data_ptr(), state.data_ptr(), cu.data_ptr(),
            history.data_ptr(), B, H, Kd, V, float(q_scale), _fp32(proj), lib.stream_ptr())
    return o


def gla_norm_gate(o, gate, w, eps: float):
    """Per-head RMS norm of o fp32 [N, H, V], times w, times silu(gate [N, H*V], any pitch) -> T [N, H*V]."""
    kind = _same(gate, w)
    _contig(o, w)
    N, H, V = o.shape
    out = torch.empty(N, H * V, dtype=gate.dtype, device=o.device)
    K._call("ob_gla_norm_gate", o.data_ptr(), gate.data_ptr(), gate.stride(0), w.data_ptr(), out.data_ptr(), N, H, V,
            float(eps), kind, lib.stream_ptr())
    return out


def gla_step(proj, z, bias, norm_w, state, seen, H: int, Kd: int, V: int, q_scale: float, tau: float, eps: float):
    """One token per row: ``proj`` T [B, >= 2HK + 2HV] = [q | k | v | g], ``z`` fp32 [B, H*K] without its
    bias; ``seen`` int32 [B] counts the row's tokens including this one (0: idle row, state untouched)."""
    kind = _same(proj, bias, norm_w)
    _contig(z, bias, norm_w, state, seen)
    B = seen.numel()
    if state.shape[0] < B or tuple(state.shape[1:]) != (H, Kd, V) or proj.shape[1] < 2 * H * (Kd + V):
        raise ValueError("projection or state does not fit the batch")
    out = torch.empty(B, H * V, dtype=proj.dtype, device=proj.device)
    K._call("ob_gla_step", proj.data_ptr(), proj.stride(0), z.data_ptr(), bias.data_ptr(), norm_w.data_ptr(), out.data_ptr(),
            state.data_ptr(), seen.data_ptr(), B, H, Kd, V, float(q_scale), 1.0 / float(tau), float(eps), kind,
            lib.stream_ptr())
    return out


# ----------------------------------------------------------------------------------------------- latent attention
def latent_prepare(proj, pos, row, cos, sin, H: int, dim: int, rot: int, rank: int, *, dkv_off: int = -1, norm_w=None,
                   cache=None, eps: float = 0.0, packed=None):
    """Rotate the second part of every query head of ``proj`` in place; with ``dkv_off`` >= 0 also norm
    the latent at that column, rotate the shared key part and store both in ``cache`` [rows, pitch] at
    ``row`` (and in ``packed`` [N, pitch]).  ``pos`` -1 marks a row without a token."""
    kind = _fp32(proj)
    _contig(pos, row, cos, sin, norm_w, cache, packed)
    ldc = cache.shape[1] if cache is not None else 0
    if dkv_off >= 0 and (ldc < rank + rot or norm_w.numel() != rank or proj.shape[1] < dkv_off + rank + rot
                         or (packed is not None and packed.shape[1] != ldc)):
        raise ValueError("latent cache rows do not fit")
    K._call("ob_latent_prepare", proj.data_ptr(), proj.stride(0), dkv_off, pos.data_ptr(), row.data_ptr(), cos.data_ptr(),
            sin.data_ptr(), cos.shape[0], cos.shape[1], lib.ptr(norm_w), lib.ptr(cache),
            cache.shape[0] if cache is not None else 0, ldc, lib.ptr(packed), pos.numel(), H, dim, rot, rank, float(eps), kind,
            lib.status_tensor(proj.device).data_ptr(), lib.stream_ptr())


def two_part_fits(dtype, dim: int, rot: int, vdim: int, rank: int) -> bool:
    """Sizes the tcgen05 prompt kernel covers (expanded keys + shared rotated part)."""
    return (dtype == bf16 and not (dim | rot | vdim | rank) & 7 and -(-dim // 64) + -(-rot // 64) <= 4 and vdim <= 128)


def attn_two_part(q, k1, k2, v, cu, max_len: int, H: int, d1: int, d2: int, vdim: int, scale: float):
    """Causal attention over packed rows: q [N, H*(d1+d2)], k1 [N, H*d1], k2 [N, d2] shared by the heads,
    v [N, H*vdim] (row-strided views allowed) -> [N, H*vdim]."""
    N = q.shape[0]
    out = torch.empty(N, H * vdim, dtype=bf16, device=q.device)
    K._call("ob_attn_fwd_two_part", q.data_ptr(), k1.data_ptr(), k2.data_ptr(), v.data_ptr(), out.data_ptr(), cu.data_ptr(),
            cu.numel() - 1, int(max_len), N, H, d1, d2, vdim, q.stride(0), k1.stride(0), k2.stride(0), v.stride(0),
            float(scale), lib.status_tensor(q.device).data_ptr(), lib.stream_ptr())
    return out


def latent_absorb(q, head_stride: int, uk, H: int, dim: int, rank: int, out_dtype):
    """W_uk^T applied to the first ``dim`` channels of every query head: [N, H, rank]."""
    kind = _same(q, uk)
    _contig(uk)
    out = torch.empty(q.shape[0], H, rank, dtype=out_dtype, device=q.device)
    K._call("ob_latent_absorb", q.data_ptr(), q.stride(0), head_stride, uk.data_ptr(), out.data_ptr(), q.shape[0], H, dim, rank,
            kind, int(out_dtype == bf16), lib.stream_ptr())
    return out


def latent_expand(o_lat, uv, vdim: int):
    """o_lat fp32 [N, H, rank] -> W_uv o_lat, T [N, H*vdim]."""
    _contig(o_lat, uv)
    N, H, rank = o_lat.shape
    out = torch.empty(N, H * vdim, dtype=uv.dtype, device=uv.device)
    K._call("ob_latent_expand", o_lat.data_ptr(), uv.data_ptr(), out.data_ptr(), N, H, vdim, rank, _fp32(uv), lib.stream_ptr())
    return out


def latent_attn_any(q_lat, q, head_stride: int, dim: int, rot: int, cache, seq, seen, block_table, page_size: int, scale: float):
    """Attention of any query rows against their sequences' cached latents: ``seen`` int32 [N] keys are
    visible to a query of sequence ``seq``.  q_lat fp32 [N, H, rank] -> fp32 [N, H, rank]."""
    kind = _same(q, cache)
    _contig(q_lat, cache, seq, seen, block_table)
    N, H, rank = q_lat.shape
    out = torch.empty_like(q_lat)
    K._call("ob_latent_attn_any", q_lat.data_ptr(), q.data_ptr() + dim * q.element_size(), q.stride(0), head_stride,
            cache.data_ptr(), cache.shape[1], seq.data_ptr(), seen.data_ptr(), block_table.data_ptr(), block_table.shape[1],
            page_size, out.data_ptr(), N, H, rank, rot, float(scale), kind, lib.stream_ptr())
    return out


def latent_decode_fits(dtype, dim: int, rot: int, rank: int) -> bool:
    """Sizes the bf16 tensor-core decode kernel covers."""
    return dtype == bf16 and not (dim | rot | rank) & 7 and rank <= 512 and rot <= 64


def latent_decode_splits(B: int, H: int, capacity: int) -> int:
    """Key splits per sequence: one wave of CTAs over the SMs, at least one 64-key tile of capacity each."""
    blocks = B * -(-H // (16 if H <= 16 else 32))
    return max(1, min(148 // blocks, capacity // 64, 64))


def latent_decode(q_lat, q, head_stride: int, dim: int, rot: int, cache, seen, block_table, page_size: int, scale: float,
                  splits: int | None = None):
    """One query row per sequence, bf16: q_lat [B, H, rank] -> fp32 [B, H, rank]."""
    _contig(q_lat, cache, seen, block_table)
    B, H, rank = q_lat.shape
    if splits is None:
        splits = latent_decode_splits(B, H, block_table.shape[1] * page_size)
    dev = q_lat.device
    part_o = torch.empty(B * splits * H * rank, dtype=f32, device=dev)
    part_ml = torch.empty(B * splits * H * 2, dtype=f32, device=dev)
    out = torch.empty(B, H, rank, dtype=f32, device=dev)
    K._call("ob_latent_decode", q_lat.data_ptr(), q.data_ptr() + dim * q.element_size(), q.stride(0), head_stride,
            cache.data_ptr(), cache.shape[1], seen.data_ptr(), block_table.data_ptr(), block_table.shape[1], page_size,
            part_o.data_ptr(), part_ml.data_ptr(), out.data_ptr(), B, H, rank, rot, splits, float(scale), lib.stream_ptr())
    return out


# ----------------------------------------------------------------------------------------------- windowed attention
def window_prepare(proj, pos, row, cos, sin, H: int, G: int, dim: int, vdim: int, norm_w, cache, eps: float, *, mix=None,
                   v_first=None):
    """``proj`` rows [q H*dim | k G*dim | v G*vdim]: norm all of q and all of k, rotate halves by position,
    mix v with ``v_first`` [N, G*vdim] by the scalar ``mix``; in place, and [v | k] per head into ``cache``
    [rows, pitch] at ``row``.  ``pos`` -1 marks a row without a token."""
    kind = _same(proj, norm_w, cache, mix, v_first)
    _contig(pos, row, cos, sin, norm_w, cache)
    if (cache.shape[1] < G * (dim + vdim) or norm_w.numel() != (H + G) * dim or proj.shape[1] < (H + G) * dim + G * vdim
            or proj.stride(1) != 1 or (mix is not None and (v_first is None or v_first.shape[0] < pos.numel()
                                                            or v_first.shape[1] < G * vdim or v_first.stride(1) != 1))):
        raise ValueError("projection, norm weights or cache rows do not fit")
    K._call("ob_window_prepare", proj.data_ptr(), proj.stride(0), pos.data_ptr(), row.data_ptr(), cos.data_ptr(), sin.data_ptr(),
            cos.shape[0], cos.shape[1], norm_w.data_ptr(), lib.ptr(mix), lib.ptr(v_first),
            v_first.stride(0) if v_first is not None else 0, cache.data_ptr(), cache.shape[0], cache.shape[1], pos.numel(), H, G,
            dim, vdim, float(eps), kind, lib.status_tensor(proj.device).data_ptr(), lib.stream_ptr())


def window_prompt_fits(dtype, dim: int, vdim: int) -> bool:
    """Sizes the tcgen05 prompt kernel covers."""
    return dtype == bf16 and not (dim | vdim) & 7 and dim <= 256 and vdim <= 128


def attn_window(q, k, v, cu, max_len: int, H: int, G: int, dim: int, vdim: int, scale: float, window: int, sink=None):
    """Causal attention over packed rows that all start at position 0: q [N, H*dim], k [N, G*dim],
    v [N, G*vdim] (row-strided views allowed) -> [N, H*vdim].  A query sees the last ``window`` tokens
    (0: all); ``sink`` [H] adds a logit without a value to every denominator."""
    _same(q, k, v, sink)
    _contig(sink)
    N = q.shape[0]
    out = torch.empty(N, H * vdim, dtype=bf16, device=q.device)
    K._call("ob_attn_fwd_window", q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), cu.data_ptr(), cu.numel() - 1,
            int(max_len), N, H, G, dim, vdim, q.stride(0), k.stride(0), v.stride(0), float(scale), int(window), lib.ptr(sink),
            lib.status_tensor(q.device).data_ptr(), lib.stream_ptr())
    return out


def window_attn_any(q, cache, seq, seen, block_table, page_size: int, H: int, G: int, dim: int, vdim: int, scale: float,
                    window: int, sink=None):
    """Attention of any query rows against their sequences' cached rows: ``seen`` int32 [N] tokens of
    sequence ``seq`` end at the query's own.  q [N, H*dim] -> [N, H*vdim]."""
    kind = _same(q, cache, sink)
    _contig(cache, seq, seen, block_table, sink)
    out = torch.empty(q.shape[0], H * vdim, dtype=q.dtype, device=q.device)
    K._call("ob_window_attn_any", q.data_ptr(), q.stride(0), cache.data_ptr(), cache.shape[1], seq.data_ptr(), seen.data_ptr(),
            block_table.data_ptr(), block_table.shape[1], page_size, lib.ptr(sink), out.data_ptr(), q.shape[0], H, G, dim, vdim,
            int(window), float(scale), kind, lib.stream_ptr())
    return out


def window_decode_fits(dtype, dim: int, vdim: int) -> bool:
    """Sizes the bf16 tensor-core decode kernel covers."""
    return dtype == bf16 and not (dim | vdim) & 7 and vdim <= 512 and dim + vdim <= 640


def window_decode_splits(B: int, H: int, G: int, keys: int) -> int:
    """Key splits per sequence and key/value head: about two CTAs per SM, at least two 64-key tiles each
    (a tile costs a CTA 2 us, merging the splits 4)."""
    R = H // G
    blocks = B * G * -(-R // (16 if R <= 16 else 32))
    return max(1, min(296 // blocks, keys // 128, 64))


def window_decode(q, cache, seen, block_table, page_size: int, H: int, G: int, dim: int, vdim: int, scale: float, window: int,
                  sink=None, splits: int | None = None):
    """One query row per sequence, bf16: q [B, H*dim] -> [B, H*vdim]."""
    _same(q, cache, sink)
    _contig(cache, seen, block_table, sink)
    B = q.shape[0]
    if splits is None:
        keys = block_table.shape[1] * page_size
        splits = window_decode_splits(B, H, G, min(keys, window) if window else keys)
    part_o = part_ml = None
    if splits > 1:
        part_o = torch.empty(B * splits * H * vdim, dtype=f32, device=q.device)
        part_ml = torch.empty(B * splits * H * 2, dtype=f32, device=q.device)
    out = torch.empty(B, H * vdim, dtype=bf16, device=q.device)
    K._call("ob_window_decode", q.data_ptr(), q.stride(0), cache.data_ptr(), cache.shape[1], seen.data_ptr(),
            block_table.data_ptr(), block_table.shape[1], page_size, lib.ptr(sink), lib.ptr(part_o), lib.ptr(part_ml),
            out.data_ptr(), B, H, G, dim, vdim, int(window), splits, float(scale), lib.stream_ptr())
    return out


# ----------------------------------------------------------------------------------------------- routed experts
FEW_PAIRS = 2048      # (token, slot) pairs the kernels without a sort hold


def route_sigmoid(logits, top: int):
    """fp32 logits [M, E] -> (weights fp32 [M, top] = sigmoids of the largest logits, expert ids int32)."""
    if logits.dtype != f32 or logits.stride(1) != 1:
        raise TypeError("route_sigmoid reads fp32 rows")
    M, E = logits.shape
    w = torch.empty(M, top, dtype=f32, device=logits.device)
    idx = torch.empty(M, top, dtype=torch.int32, device=logits.device)
    K._call("ob_router_sigmoid_topk", logits.data_ptr(), logits.stride(0), w.data_ptr(), idx.data_ptr(), M, E, top, lib.stream_ptr())
    return w, idx


def experts_few_fits(dtype, pairs: int, E: int, D: int, F: int) -> bool:
    """Sizes and counts of the bf16 kernels that stream each expert's weights past the pairs routed to it."""
    return dtype == bf16 and pairs <= min(FEW_PAIRS, 16 * E) and not (D | F) & 7


def experts_into(h, w, idx, gate_up, down, act: str, into, *, few: bool | None = None):
    """into [M, D] fp32 += sum over the slots of expert(w * h): h T [M, D], w fp32 / idx int32 [M, k],
    gate_up T [E, 2F, D] with rows [gate | up], down T [E, D, F].  ``few`` overrides the choice of path."""
    kind = _same(h, gate_up, down)
    _contig(h, w, idx, gate_up, down, into)
    (M, k), (E, D, F) = idx.shape, down.shape
    P, dev = M * k, h.device
    if gate_up.shape != (E, 2 * F, D) or h.shape != (M, D) or into.shape != (M, D) or into.dtype != f32:
        raise ValueError("experts, rows or indices do not fit")
    if P == 0:
        return into
    lib.check_index("expert ids", idx, E)
    fits = act == "silu" and experts_few_fits(h.dtype, P, E, D, F)
    if fits if few is None else few:
        mid = torch.empty(P, F, dtype=bf16, device=dev)
        y = torch.empty(P, D, dtype=f32, device=dev)
        K._call("ob_experts_few", h.data_ptr(), idx.data_ptr(), w.data_ptr(), gate_up.data_ptr(), down.data_ptr(), mid.data_ptr(),
                y.data_ptr(), P, k, E, D, F, lib.stream_ptr())
        K._call("ob_moe_sum", y.data_ptr(), None, into.data_ptr(), M, k, D, P, 1, lib.stream_ptr())
        return into
    tiled = not kind and not (D | F) & 7
    # segments padded to whole tiles; CTA-pair tiles once the experts fill them
    pad = 1 if not tiled else 256 if P >= 256 * E else 128
    offsets, dest = K.moe_plan(idx, E, pad)
    rows = -(-(P + E * (pad - 1)) // pad) * pad
    xs = torch.empty(rows, D, dtype=h.dtype, device=dev)         # rows between segments stay unwritten and unread
    K._call("ob_moe_gather", h.data_ptr(), w.data_ptr(), dest.data_ptr(), xs.data_ptr(), P, k, D, rows, kind, lib.stream_ptr())
    if tiled:
        gu = K.gemm_grouped(xs, gate_up, offsets, pair=pad == 256)
        y = K.gemm_grouped(gated_act(gu, act, offsets[E:]), down, offsets, pair=pad == 256)
    else:
        def grouped(a, b):
            out = torch.empty(rows, b.shape[1], dtype=a.dtype, device=dev)
            K._call("ob_expert_rows_any", a.data_ptr(), b.data_ptr(), out.data_ptr(), offsets.data_ptr(), E, b.shape[1], b.shape[2],
                    rows, kind, lib.stream_ptr())
            return out

        y = grouped(gated_act(grouped(xs, gate_up), act, offsets[E:]), down)
    K._call("ob_moe_sum", y.data_ptr(), dest.data_ptr(), into.data_ptr(), M, k, D, rows, kind, lib.stream_ptr())
    return into
