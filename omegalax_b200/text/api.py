"""Public API for text-only causal language models (Qwen3, Qwen3.5 text, and the serving decoders Letitar
and Difedra).

    model, cfg = init_model("qwen3-smoke", 0, tp_size=1, fsdp_size=1, dp_size=1)
    hidden, aux = forward(model, token_ids, pad_id, cfg)       # hidden is *before* lm_head
    cache = make_cache(cfg, batch, prompt_len, steps)
    logits, cache, aux = decode(model, cache, token_ids, pad_id, cfg)

    model, cfg = load_model(folder, device="cuda")             # class by config.json
    new_tokens = generate(model, cfg, prompts, max_new_tokens)

Mirrors omegalax/text/api.py:42-146.
"""
from __future__ import annotations

import dataclasses

import torch

from ..models import sharding_runtime as _rt
from ..models import stream_registry
from ..models.paged_sequences import PagedSequences
from ..models.qwen3 import registry as qwen3_registry
from ..models.qwen3.cache import Cache, init_cache
from ..models.qwen3.model import Qwen3
from ..models.qwen3.paged_cache import PagedKVCache
from ..models.qwen3.utils import count_right_pads
from ..models.hf_io import load_hf_config_from_source
from ..models.shard_config import shard_config_for_mesh
from ..models.stream_decoder import StreamDecoder, StreamDecoderConfig
from ..parallel.mesh import Mesh, ensure_mesh

ModelConfig = qwen3_registry.Qwen3Config
registry = qwen3_registry
list_qwen3_dense_model_ids = qwen3_registry.list_qwen3_dense_model_ids
list_qwen3_moe_model_ids = qwen3_registry.list_qwen3_moe_model_ids


def _q35():
    from ..models import qwen3_5

    return qwen3_5


def _is_q35_text(cfg) -> bool:
    return type(cfg).__name__ == "Qwen3_5TextConfig"


def resolve_config(model_or_id):
    """Model id (Qwen3 preset / repo, Qwen3.5 id -> its text config, or any directory / repo
    with a config.json) or an already-built config, which is passed through."""
    if not isinstance(model_or_id, str):
        return model_or_id
    if qwen3_registry.is_supported_model_id(model_or_id):
        return qwen3_registry.build_config(model_or_id)
    q35 = _q35()
    if q35.config.is_supported_qwen3_5_model_id(model_or_id):
        return q35.config.make_config(model_or_id).text_config
    family = stream_registry.family_of_preset(model_or_id)
    if family is None:
        hf_cfg = load_hf_config_from_source(model_or_id)
        family = stream_registry.family_for(hf_cfg)
    if family is not None:
        return family.make_config(model_or_id)
    mt = hf_cfg.get("model_type")
    if mt in {"qwen3", "qwen3_moe"}:
        return qwen3_registry.make_config_from_hf(hf_cfg)
    if mt in {"qwen3_5", "qwen3_5_moe"}:
        return q35.config.make_config_from_hf(hf_cfg).text_config
    raise ValueError(
        f"Unsupported text model/config source '{model_or_id}'. Supported Qwen3 ids: "
        f"{sorted(set(list_qwen3_dense_model_ids() + list_qwen3_moe_model_ids()))}; supported Qwen3.5 ids: "
        f"{q35.config.list_supported_qwen3_5_model_ids()}; serving decoder ids: {stream_registry.list_model_ids()}.")


def align_config_to_mesh(cfg, mesh: Mesh):
    """Drop size-one mesh axes from the config's activation layouts."""
    return dataclasses.replace(cfg, shd_cfg=shard_config_for_mesh(cfg.shd_cfg, mesh.shape))


def batch_partition_spec(cfg):
    return _rt.batch_partition_spec(cfg.shd_cfg)


def shard_batch(token_ids_BT, cfg, mesh: Mesh | None = None, device=None):
    return _rt.shard_batch(token_ids_BT, cfg.shd_cfg, mesh, device)


def shard_batch_dict(batch: dict, cfg, mesh: Mesh | None = None, device=None) -> dict:
    return _rt.shard_batch_dict(batch, cfg.shd_cfg, mesh, device)


def model_class_for(cfg):
    if isinstance(cfg, ModelConfig):
        return Qwen3
    if isinstance(cfg, StreamDecoderConfig):
        return stream_registry.family_of(cfg).model_cls
    if _is_q35_text(cfg):
        return _q35().model.Qwen3_5ForCausalLM
    raise ValueError(f"Unsupported text config type: {type(cfg)}")


def is_inference_only(cfg) -> bool:
    """The family's kernels have no backward pass."""
    return isinstance(cfg, StreamDecoderConfig)


def init_model(model_or_id, rng: int = 0, *, tp_size: int | None = None, fsdp_size: int | None = None,
               dp_size: int | None = None, device=None, dtype=None, meta: bool = False):
    """Random-initialise a text model; returns (model, cfg).  ``rng`` is an integer seed.
    With ``meta=True`` the parameters are not allocated (the training engine materialises
    only this rank's shard)."""
    cfg = resolve_config(model_or_id)
    mesh = ensure_mesh(tp_size=tp_size, fsdp_size=fsdp_size, dp_size=dp_size)
    cfg = align_config_to_mesh(cfg, mesh)
    if device is None:
        device = "cuda" if torch.cuda.is_available() else "cpu"
    if dtype is None:
        dtype = cfg.dtype if torch.device(device).type == "cuda" else torch.float32
    model = _rt.init_model_sharded(model_class_for(cfg), cfg, int(rng), mesh, meta=meta, device=device, dtype=dtype)
    return model, cfg


def forward(model, token_ids_BT, pad_id: int, cfg):
    """Hidden states before lm_head [B,T,D] and the auxiliary (router) loss."""
    segment_ids = (token_ids_BT != pad_id).to(torch.int32)
    return model(token_ids_BT, segment_ids, None, 0)


def load_model(source, *, device=None, dtype=torch.bfloat16):
    """Model and config from a folder with config.json and safetensors; the class follows config.json."""
    cfg = resolve_config(str(source))
    device = device or ("cuda" if torch.cuda.is_available() else "cpu")
    if isinstance(cfg, StreamDecoderConfig):
        return stream_registry.family_of(cfg).load_model(source, device=device, dtype=dtype), cfg
    if isinstance(cfg, ModelConfig):
        from ..models.qwen3.loader import create_qwen3_from_safetensors

        return create_qwen3_from_safetensors(source, device=device, dtype=dtype), cfg
    raise ValueError(f"no text loader for {type(cfg).__name__}")


def decode(model, cache: Cache, token_ids_BT, pad_id: int, cfg, select=None):
    """One prefill / decode call: logits [B,V] at the last non-pad column, the cache, aux.  With a paged
    cache, ``select`` (bool [B,T]) asks for the logits of the marked tokens instead, in order."""
    if not isinstance(model, (Qwen3, StreamDecoder)):
        raise NotImplementedError("decode is only implemented for Qwen3 and the serving decoders (Letitar, Difedra).")
    segment_ids = (token_ids_BT != pad_id).to(torch.int32)
    if isinstance(cache, PagedSequences):
        hidden = model.decode_paged(token_ids_BT, segment_ids, cache, select)
        with torch.no_grad():
            return model.logits(hidden), cache, torch.zeros((), device=hidden.device)
    if select is not None:
        raise NotImplementedError("logits of chosen tokens need a paged cache")
    nrp = count_right_pads(token_ids_BT, pad_id)
    with torch.no_grad():
        hidden, aux = model(token_ids_BT, segment_ids, cache, nrp)
        col = token_ids_BT.shape[-1] - nrp - 1
        logits = model.lm_head(hidden[:, col])
        if getattr(model, "vocab_parallel", False):   # this rank's slice of the vocabulary -> all of it
            from ..parallel import tp as tp_lib

            tp = tp_lib.current()
            parts = [torch.empty_like(logits) for _ in range(tp.size)]
            torch.distributed.all_gather(parts, logits.contiguous(), group=tp.group)
            logits = torch.cat(parts, dim=-1)
    return logits, cache, aux


def make_cache(cfg, batch_size: int, token_len: int, generate_steps: int, dtype=torch.bfloat16, device=None,
               paged: bool | None = None, page_size: int = 64, tp_size: int = 1, num_pages: int | None = None):
    """KV cache for ``decode``.  On CUDA with bf16 (head_dim 128) the paged cache + decode kernels
    are used by default; otherwise the contiguous power-of-two cache of the reference.  With
    ``tp_size`` > 1 the (contiguous) cache holds this tensor-parallel rank's kv heads.  Serving decoders
    use a ``HybridCache`` in ``dtype``; ``num_pages`` bounds the pages of a paged cache when the
    sequences together hold fewer tokens than batch_size full ones."""
    if isinstance(cfg, StreamDecoderConfig):
        if tp_size > 1:
            raise NotImplementedError("the serving decoders have no tensor-parallel layout")
        return StreamDecoder.make_cache_for(cfg, batch_size, token_len + generate_steps, page_size=page_size, num_pages=num_pages,
                                      dtype=dtype, device=device)
    if not isinstance(cfg, ModelConfig):
        raise NotImplementedError("Cache is only available for Qwen3 text models and the serving decoders.")
    if tp_size > 1:
        import dataclasses

        if cfg.num_kv_heads % tp_size:
            raise ValueError(f"kv heads ({cfg.num_kv_heads}) do not divide over tp_size={tp_size}")
        return init_cache(dataclasses.replace(cfg, num_kv_heads=cfg.num_kv_heads // tp_size), batch_size, token_len,
                          generate_steps, dtype, device)
    if paged is None:
        paged = (device is not None and torch.device(device).type == "cuda" and dtype == torch.bfloat16
                 and cfg.head_dim == 128 and (cfg.num_heads // cfg.num_kv_heads) in (1, 2, 4, 8))
    if paged:
        return PagedKVCache(cfg, batch_size, token_len + generate_steps, page_size=page_size, dtype=dtype, device=device,
                            num_pages=num_pages)
    return init_cache(cfg, batch_size, token_len, generate_steps, dtype, device)


NO_TOKEN = -1      # padding id of batches whose rows may hold any vocabulary id


def batch_rows(rows, batch_size: int):
    """[batch_size, longest] int32 batch with ``rows[b]`` (a list, possibly empty) left-aligned in row b."""
    out = torch.full((batch_size, max(1, max((len(r) for r in rows), default=1))), NO_TOKEN, dtype=torch.int32)
    for b, r in enumerate(rows):
        if len(r):
            out[b, :len(r)] = torch.as_tensor(r, dtype=torch.int32)
    return out


@torch.no_grad()
def generate(model, cfg, prompts, max_new_tokens: int, *, eos_id: int | None = None):
    """Greedy continuation of a batch of prompts (lists of ids, any lengths): one prompt call, then one
    call per token through ``decode`` and a paged cache.  A finished sequence gives its pages back
    while the others go on.  Returns one list of new ids per prompt."""
    B = len(prompts)
    if B == 0 or any(len(p) == 0 for p in prompts):
        raise ValueError("every prompt needs at least one token")
    w = next(model.parameters())
    cache = make_cache(cfg, B, max(len(p) for p in prompts), max_new_tokens, dtype=w.dtype, device=w.device)
    if not isinstance(cache, PagedSequences):
        raise NotImplementedError("generate needs a model with a paged cache (CUDA)")
    out: list[list[int]] = [[] for _ in range(B)]
    rows = [list(p) for p in prompts]
    live = set(range(B)) if max_new_tokens > 0 else set()
    while live:
        ids = batch_rows(rows, B)
        if isinstance(model, Qwen3):
            ids = ids.to(w.device)
        logits, cache, _ = decode(model, cache, ids, NO_TOKEN, cfg)
        best = logits.argmax(-1).tolist()
        rows = [[] for _ in range(B)]
        for b in sorted(live):
            out[b].append(best[b])
            if len(out[b]) == max_new_tokens or best[b] == eos_id:
                live.discard(b)
                cache.free_sequence(b)
            else:
                rows[b] = [best[b]]
    return out
