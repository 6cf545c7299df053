"""Letitar on the host: configuration, rotary frequencies, checkpoint mapping, cache bookkeeping."""
import dataclasses
import json

import pytest
import torch

from omegalax_b200 import export, registry
from omegalax_b200.models.letitar.config import config_to_hf, make_config_from_hf
from omegalax_b200.models.letitar.registry import FAMILY
from omegalax_b200.models.mixers import GatedLinearAttentionConfig, LatentAttentionConfig, TokenBatch
from omegalax_b200.models.paged_sequences import HybridCache, LatentPages, RecurrentState, SharedWith
from omegalax_b200.models.rope_scaling import RotaryConfig, RotaryTable, YarnScaling
from omegalax_b200.text import api

from . import letitar_models as M
from . import letitar_oracle as O


def test_config_is_read_in_full_and_written_back():
    for d in (M.EVEN, M.ODD):
        cfg = make_config_from_hf(d)
        assert json.loads(json.dumps(config_to_hf(cfg))) == json.loads(json.dumps(d))
    assert cfg.layers[2].mlp is None and cfg.layers[2].mixer.kv_from == 0 and cfg.layers[0].mixer.rot.scaling is None
    assert cfg.layers[1].mixer.tau == 3.0 and cfg.norm_eps == 1e-3 and cfg.logit_softcap == 3.0


@pytest.mark.parametrize("change", [{"kv_rank": 38}, {"rot_dim": 8}, {"kv_from": 1}, {"kv_from": 2}, {"rot": {"dims": 6, "base": 7.0}}])
def test_a_layer_can_only_read_a_matching_earlier_latent(change):
    d = json.loads(json.dumps(M.ODD))
    d["layers"][2]["mixer"].update(change)
    with pytest.raises(ValueError):
        make_config_from_hf(d)


def test_unknown_parts_are_refused():
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 0, "mlp", "kind"), "moe"), (("architecture",), "Other")):
        d = json.loads(json.dumps(M.EVEN))
        at = d
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            make_config_from_hf(d)


@pytest.mark.parametrize("dims,base,scaling", [(24, 500.0, (2.0, 64, 8.0, 1.0)), (64, 10000.0, (40.0, 4096, 32.0, 1.0)), (8, 3000.0, (16.0, 32, 4.0, 0.5)),
                                               (2, 100.0, (4.0, 100, 2.0, 1.0)), (16, 77.0, None), (6, 50.0, (1.0, 16, 2.0, 2.0))])
def test_rotary_frequencies(dims, base, scaling):
    names = ("factor", "original", "fast", "slow")
    rot = RotaryConfig(dims, base, None if scaling is None else YarnScaling(*scaling))
    freq, amp = rot.frequencies()
    want, want_amp = O.yarn_frequencies(dims, base, None if scaling is None else dict(zip(names, scaling)))
    torch.testing.assert_close(freq, torch.tensor(want, dtype=torch.float64), rtol=1e-12, atol=0)
    assert amp == pytest.approx(want_amp, rel=1e-14)
    cos, sin = RotaryTable(rot).get(3000, torch.device("cpu"))
    ang = torch.arange(3000, dtype=torch.float64)[:, None] * torch.tensor(want, dtype=torch.float64)
    assert (cos[:3000] - torch.cos(ang) * want_amp).abs().max() < 2e-7 and (sin[:3000] - torch.sin(ang) * want_amp).abs().max() < 2e-7


def test_registry_and_presets():
    assert registry.infer_arch("letitar-smoke") is registry.Arch.TEXT
    cfg = api.resolve_config("letitar-smoke")
    assert api.model_class_for(cfg).__name__ == "Letitar"
    kinds = {type(layer.mixer) for layer in cfg.layers}
    assert kinds == {GatedLinearAttentionConfig, LatentAttentionConfig}
    big = FAMILY.make_config("letitar-8layer-4096")
    assert big.width == 4096 and big.layers[-1].mixer.kv_from == 4
    with pytest.raises(NotImplementedError):
        api.make_cache(cfg, 1, 8, 8, tp_size=2)
    from omegalax_b200.trainers import text as trainer

    with pytest.raises(NotImplementedError, match="inference only"):
        trainer.init_model("letitar-smoke", 0, tp_size=1, fsdp_size=1, dp_size=1)


@pytest.mark.parametrize("cfg_dict,rank", [(M.EVEN, 8), (M.ODD, 5)])
def test_checkpoint_round_trip(tmp_path, cfg_dict, rank):
    w = M.weights(cfg_dict, 0, decay_rank=rank)
    folder = M.write(tmp_path / "a", cfg_dict, w)
    assert registry.infer_arch(str(folder)) is registry.Arch.TEXT
    model, cfg = api.load_model(folder, device="cpu")
    assert {layer.mixer.decay_rank for layer in cfg.layers if isinstance(layer.mixer, GatedLinearAttentionConfig)} == {rank}
    qk = cfg.layers[1 if cfg_dict is M.ODD else 0].mixer
    export.export_model_to_hf(model, cfg, tmp_path / "b")
    from safetensors.torch import load_file

    back = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(back) == set(w) and all(torch.equal(back[k], w[k]) for k in w)
    again, cfg2 = api.load_model(tmp_path / "b", device="cpu", dtype=torch.float32)
    assert cfg2 == cfg and qk.decay_rank == rank
    for (n, p), (n2, p2) in zip(model.named_parameters(), again.named_parameters()):
        assert n == n2 and torch.equal(p.float(), p2)


def test_incomplete_or_foreign_checkpoints_are_refused(tmp_path):
    w = M.weights(M.EVEN, 0)
    missing = {k: v for k, v in w.items() if k != "l1.mix.dkv.norm"}
    with pytest.raises(RuntimeError, match="latent_norm"):
        api.load_model(M.write(tmp_path / "a", M.EVEN, missing), device="cpu")
    with pytest.raises(RuntimeError, match="l2.mix.dkv"):      # a layer that reads another one's latent has none of its own
        api.load_model(M.write(tmp_path / "b", M.EVEN, {**w, "l2.mix.dkv": w["l1.mix.dkv"]}), device="cpu")


def test_hybrid_cache_stores_and_pages():
    specs = [RecurrentState(2, 8, 4), LatentPages(20, 6), SharedWith(1)]
    c = HybridCache(specs, 3, 40, page_size=8, device="cpu", num_pages=7)
    assert c.stores[0].shape == (3, 2, 8, 4) and c.stores[0].dtype == torch.float32
    assert c.stores[1].shape == (56, 32) and c.stores[2] is c.stores[1]
    c.reserve([9, 0, 16])
    c.advance([9, 0, 16])
    rows = c.flat_rows_host(2, 6, 4)
    assert rows.tolist() == c.flat_rows(torch.full((4,), 2), torch.arange(6, 10)).tolist() == [c.flat_row_host(2, s) for s in range(6, 10)]
    held = set(c.block_table_host[0][:2].tolist()) | set(c.block_table_host[2][:2].tolist())
    assert len(held) == 4 and len(c.allocator.free) == 3
    c.free_sequence(0)
    assert len(c.allocator.free) == 5 and c.seq_lens_host == [0, 0, 16]
    c.reserve([0, 40, 0])
    with pytest.raises(RuntimeError, match="out of pages"):
        c.reserve([1, 0, 0])
    with pytest.raises(RuntimeError, match="capacity"):
        c.reserve([0, 0, 25])
    for bad in ([SharedWith(0)], [RecurrentState(1, 1, 1), SharedWith(0)], [None]):
        with pytest.raises((ValueError, TypeError)):
            HybridCache(bad, 1, 8, device="cpu")


def test_token_batches():
    c = HybridCache([LatentPages(8, 8)], 3, 64, page_size=4, device="cpu")
    t = lambda *v: torch.tensor(v, dtype=torch.int32)  # noqa: E731
    c.reserve([2, 0, 5])
    b = TokenBatch.build(c, [t(7, 8), t(), t(1, 2, 3, 4, 5)])
    assert (b.single, b.fresh, b.max_new) == (False, True, 5)
    assert b.ids.tolist() == [7, 8, 1, 2, 3, 4, 5] and b.pos.tolist() == [0, 1, 0, 1, 2, 3, 4]
    assert b.cu.tolist() == [0, 2, 2, 7] and b.seq.tolist() == [0, 0, 2, 2, 2, 2, 2] and b.history.tolist() == [0, 0, 0]
    assert b.row.tolist() == c.flat_rows_host(0, 0, 2).tolist() + c.flat_rows_host(2, 0, 5).tolist()
    c.advance([2, 0, 5])
    c.reserve([1, 0, 1])
    b = TokenBatch.build(c, [t(9), t(), t(6)])
    assert b.single and b.ids.tolist() == [9, -1, 6] and b.pos.tolist() == [2, -1, 5] and b.seen.tolist() == [3, 0, 6]
    assert b.row.tolist() == [c.flat_row_host(0, 2), -1, c.flat_row_host(2, 5)]
    b = TokenBatch.build(c, [t(9), t(), t(6, 6)])
    assert not b.single and not b.fresh and b.pos.tolist() == [2, 5, 6]


def test_trace_runner_protocol(monkeypatch):
    """Rows, wanted places and freed requests, with the model's step replaced by a recorder."""
    from omegalax_b200.text import trace

    cfg = FAMILY.make_config("letitar-smoke")
    calls = []

    class Fake(torch.nn.Module):
        def __init__(self):
            super().__init__()
            self.p = torch.nn.Parameter(torch.zeros(1))

    def decode(model, cache, ids, pad, cfg, select=None):
        calls.append(ids.tolist())
        new = [(r >= 0).sum().item() for r in ids]
        cache.reserve(new)
        cache.advance(new)
        return ids[select].float()[:, None], cache, None

    monkeypatch.setattr(api, "decode", decode)
    r = trace.TraceRunner(Fake(), cfg, 300)
    out = r.step([{"id": "x", "tokens": [5, 6, 7], "want": [2, 0, 2]}, {"id": "y", "tokens": [8], "want": [0]}], [])
    assert out.reshape(-1).tolist() == [7.0, 5.0, 7.0, 8.0] and calls[-1] == [[5, 6, 7], [8, -1, -1]]
    assert r.step([{"id": "y", "tokens": [9], "want": []}], ["x"]) is None and calls[-1] == [[-1], [9]]
    assert r.cache.seq_lens_host == [0, 2]
    with pytest.raises(ValueError):
        r.step([{"id": "z", "tokens": [1], "want": []}], [])
    assert r.step([{"id": "y", "tokens": [3], "want": [0]}], ["y"]).tolist() == [[3.0]]
    cache = r.cache
    r.step([{"id": "a", "tokens": [1], "want": []}, {"id": "b", "tokens": [2, 2], "want": []}], ["a", "b"])
    assert r.cache is cache and len(cache.allocator.free) == cache.num_pages
    r.step([{"id": "c", "tokens": [1] * 300, "want": []}], [])
    assert r.cache.B == 1 and r.cache.seq_lens_host == [300]
    assert dataclasses.is_dataclass(cfg)
