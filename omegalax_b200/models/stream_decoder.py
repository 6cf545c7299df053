"""What the serving decoders share: token rows in an fp32 residual stream, a list of layers that each add a
mixer's and a feed-forward's output into it, a final norm and logits, run against a ``HybridCache``.
Inference only, on CUDA, in bf16 or fp32.

A design subclasses ``StreamDecoder`` (its norm, its layers, its logits) and describes itself to the
registry with a ``Family``.
"""
from __future__ import annotations

import dataclasses
from pathlib import Path
from typing import Any, Callable, Mapping

import torch
from torch import nn

from ..ops import serving as S
from .decode_graph import DecodeGraph
from .hf_io import load_hf_config_from_source, safetensors_shapes, save_hf_config
from .mixers import TokenBatch
from .paged_sequences import HybridCache
from .params_utils import Rule, StateAssembler, native_state, rows, save_safetensors, stream_safetensors
from .rope_scaling import RotaryTable
from .shard_config import ShardConfig


@dataclasses.dataclass(frozen=True, kw_only=True)
class StreamDecoderConfig:
    vocab_size: int
    width: int
    norm_eps: float
    layers: tuple                # each with a ``mixer`` config that has cache_spec(), and an ``mlp`` config or None
    shd_cfg: ShardConfig = dataclasses.field(default_factory=ShardConfig.default)
    dtype: Any = torch.bfloat16

    @property
    def num_layers(self) -> int:
        return len(self.layers)


class TokenTable(nn.Module):
    def __init__(self, num: int, dim: int, device=None, dtype=None):
        super().__init__()
        self.weight = nn.Parameter(torch.empty(num, dim, device=device, dtype=dtype))
        if self.weight.device.type != "meta":
            nn.init.normal_(self.weight)

    def forward(self, ids32):
        return S.embed_rows(ids32, self.weight)


class DecoderLayer(nn.Module):
    """x += mixer(norm1(x)), then x += mlp(norm2(x)) where the layer has a feed-forward."""

    def __init__(self, norm1, mixer, norm2=None, mlp=None):
        super().__init__()
        self.norm1, self.mixer, self.norm2, self.mlp = norm1, mixer, norm2, mlp

    def forward(self, x, batch: TokenBatch, store):
        self.mixer(self.norm1(x), batch, store, x)
        if self.mlp is not None:
            self.mlp(self.norm2(x), x)


class StreamDecoder(nn.Module):
    """Subclasses give ``norm`` (a module class taking width and eps) and ``make_layer``; logits are those of
    the embedding table unless they say otherwise."""
    norm: type

    def __init__(self, cfg: StreamDecoderConfig, device=None, dtype=None):
        super().__init__()
        kw = dict(device=device, dtype=dtype or torch.float32)
        self.cfg = cfg
        tables: dict = {}
        rotary = lambda rot: tables.setdefault(rot, RotaryTable(rot))  # noqa: E731  one table per rotation
        self.embedder = TokenTable(cfg.vocab_size, cfg.width, **kw)
        self.layers = nn.ModuleList(self.make_layer(cfg, lc, i, rotary, **kw) for i, lc in enumerate(cfg.layers))
        self.final_norm = self.norm(cfg.width, cfg.norm_eps, **kw)

    @staticmethod
    def make_layer(cfg, lc, index: int, rotary, device=None, dtype=None) -> DecoderLayer:
        raise NotImplementedError

    @staticmethod
    def make_cache_for(cfg: StreamDecoderConfig, batch_size: int, max_tokens_per_seq: int, *, page_size: int = 64, num_pages=None,
                       dtype=torch.bfloat16, device=None) -> HybridCache:
        return HybridCache([layer.mixer.cache_spec() for layer in cfg.layers], batch_size, max_tokens_per_seq,
                           page_size=page_size, dtype=dtype, device=device, num_pages=num_pages)

    @torch.no_grad()
    def run_layers(self, batch: TokenBatch, cache: HybridCache, after_layer=None):
        """fp32 residual rows [N, width] of the batch's tokens after the last layer."""
        x = self.embedder(batch.ids)
        for i, layer in enumerate(self.layers):
            layer(x, batch, cache.stores[i])
            if after_layer is not None:
                after_layer(i, x)
        return x

    @torch.no_grad()
    def decode_paged(self, token_ids, segment_ids, cache: HybridCache, select=None):
        """Run the new tokens of a [B, T] batch (padding anywhere) against the cache and store what the
        layers keep.  Returns normed hidden rows: of every sequence's last new token [B, D] (zeros for
        sequences without one), or, with the bool mask ``select`` [B, T], of the marked tokens in order."""
        ids, real = token_ids.cpu(), segment_ids.cpu() != 0
        tokens = [ids[b][real[b]].to(torch.int32) for b in range(cache.B)]
        new = [int(t.numel()) for t in tokens]
        cache.reserve(new)
        if max(new, default=0) == 0:
            rows = 0 if select is not None else cache.B
            return torch.zeros(rows, self.cfg.width, dtype=self.embedder.weight.dtype, device=cache.device)
        batch = TokenBatch.build(cache, tokens)
        x = DecodeGraph.step(self, cache, batch) if batch.single else self.run_layers(batch, cache)
        cache.advance(new)
        if select is None:
            if batch.single:
                h = self.final_norm(x)
                return h if min(new) > 0 else h * torch.tensor(new, device=h.device, dtype=h.dtype)[:, None]
            out = torch.zeros(cache.B, x.shape[1], dtype=self.embedder.weight.dtype, device=x.device)
            has = [b for b in range(cache.B) if new[b]]
            end = torch.tensor(new).cumsum(0) - 1
            out[has] = self.final_norm(x[end[has].to(x.device)])
            return out
        sel = select.cpu() & real
        if batch.single:
            rows = torch.nonzero(sel.any(-1)).reshape(-1)
        else:
            rows = torch.nonzero(sel[real]).reshape(-1)
        return self.final_norm(x[rows.to(x.device)])

    def logits(self, hidden):
        """fp32 logits of normed hidden rows."""
        y = S.project(hidden.reshape(-1, hidden.shape[-1]), self.embedder.weight, out_dtype=torch.float32)
        return y.reshape(*hidden.shape[:-1], self.cfg.vocab_size)

    @torch.no_grad()
    def forward(self, token_ids, segment_ids, cache=None, num_right_pads: int = 0):
        """Normed hidden states [B, T, D] (zeros at padding) and the auxiliary loss (none)."""
        B, T = token_ids.shape
        if cache is None:
            w = self.embedder.weight
            cache = self.make_cache_for(self.cfg, B, T, dtype=w.dtype, device=w.device)
        real = segment_ids != 0
        rows = self.decode_paged(token_ids, segment_ids, cache, select=real)
        out = torch.zeros(B, T, self.cfg.width, dtype=rows.dtype, device=rows.device)
        out[real.to(rows.device)] = rows
        return out, torch.zeros((), dtype=torch.float32, device=rows.device)


# ----------------------------------------------------------------------------------------------- checkpoints
def whole(key: str, target: str) -> Rule:
    """A checkpoint tensor that is one parameter."""
    return Rule(key.replace(".", r"\."), lambda m: target)


def part(key: str, target: str, index: tuple) -> Rule:
    """A checkpoint tensor that is a slice of a parameter."""
    return Rule(key.replace(".", r"\."), lambda m: target, lambda m: index)


def stacked(prefix: str, target: str, parts, first: tuple = ()) -> list[Rule]:
    """Rules for checkpoint tensors prefix + name, n rows each, that are consecutive row ranges of one
    parameter (of its entry ``first``)."""
    out, at = [], 0
    for name, n in parts:
        out.append(part(prefix + name, target, first + rows(at, at + n)))
        at += n
    return out


@dataclasses.dataclass(frozen=True)
class Family:
    """One design: how config.json names it, its configuration, model, weights and presets."""
    architecture: str                                        # config.json "architecture"
    config_cls: type
    config_from_hf: Callable[[Mapping, Mapping], Any]        # (config.json dict, tensor shapes) -> config
    config_to_hf: Callable[[Any], dict]
    key_rules: Callable[[Any], list[Rule]]                   # checkpoint tensors -> parameters
    model_cls: type
    presets: Mapping[str, Callable[[], Any]]
    kernels: str                                             # group of kernels a decode program needs (ops.build)

    def owns(self, hf_cfg: Mapping) -> bool:
        return hf_cfg.get("architecture") == self.architecture

    def make_config(self, source: str):
        """Preset name or a directory with config.json (and, for sizes only tensors know, model.safetensors)."""
        if source in self.presets:
            return self.presets[source]()
        return self.config_from_hf(load_hf_config_from_source(source), safetensors_shapes(source))

    def load_model(self, file_dir, *, device="cpu", dtype=torch.bfloat16):
        """Every checkpoint key must map and every parameter be filled, otherwise a RuntimeError lists them."""
        cfg = self.make_config(str(file_dir))
        model = self.model_cls(cfg, device=device, dtype=dtype)
        asm = StateAssembler(native_state(model), self.key_rules(cfg))
        for key, tensor in stream_safetensors(file_dir):
            asm.assign(key, tensor)
        asm.finish()
        return model

    def to_tensors(self, model, cfg) -> dict[str, torch.Tensor]:
        """Checkpoint tensors of a model: the loading rules walked backwards."""
        state, out = native_state(model), {}
        for rule in self.key_rules(cfg):
            key = rule.pattern.replace("\\.", ".")
            m = rule.regex.fullmatch(key)
            t, idx = state[rule.target(m)].detach(), rule.index(m)
            out[key] = (t if idx is None else t[idx]).to(torch.bfloat16).contiguous()
        return out

    def export(self, model, cfg, out_dir) -> Path:
        save_safetensors(self.to_tensors(model, cfg), out_dir)
        save_hf_config(self.config_to_hf(cfg), out_dir)
        return Path(out_dir)
