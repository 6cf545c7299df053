"""Difedra on the host: configuration, rotary frequencies, checkpoint mapping, cache bookkeeping."""
import dataclasses
import json
import math

import pytest
import torch

from omegalax_b200 import export, registry
from omegalax_b200.models.difedra.config import config_to_hf, make_config_from_hf
from omegalax_b200.models.mixers import GatedMLPConfig, MixtureOfExpertsConfig
from omegalax_b200.models.paged_sequences import HybridCache, KeyValuePages, LatentPages, RecurrentState
from omegalax_b200.models.rope_scaling import RotaryConfig, RotaryTable, WavelengthScaling
from omegalax_b200.models.stream_registry import FAMILIES, family_of
from omegalax_b200.ops import build
from omegalax_b200.text import api

from . import difedra_models as M
from . import difedra_oracle as O


def copy_of(d):
    return json.loads(json.dumps(d))


def test_config_is_read_in_full_and_written_back():
    for d in (M.EVEN, M.ODD):
        cfg = make_config_from_hf(d)
        assert copy_of(config_to_hf(cfg)) == copy_of(d)
    assert [layer.mixer.v_from for layer in cfg.layers] == [None, 1, 1, 1] and cfg.norm_eps == 1e-3
    assert cfg.layers[0].mlp == GatedMLPConfig(51, "gelu_tanh") and cfg.layers[2].mlp is None
    assert cfg.layers[3].mlp == MixtureOfExpertsConfig(4, 2, GatedMLPConfig(21, "silu"))
    assert cfg.layers[1].mixer.rot == RotaryConfig(6, 700.0, WavelengthScaling(1.0, 16.0, 1.0, 4.0))


@pytest.mark.parametrize("layer,change", [(0, {"heads": 4, "kv_heads": 3}), (0, {"rot": {"dims": 16, "base": 7.0}}), (0, {"rot": {"dims": 3, "base": 7.0}}),
                                          (3, {"vdim": 8}), (3, {"kv_heads": 3, "heads": 3, "vdim": 3}), (1, {"mask": {"size": 0}})])
def test_layers_that_cannot_be_are_refused(layer, change):
    d = copy_of(M.ODD)
    d["layers"][layer]["mixer"].update(change)
    with pytest.raises(ValueError, match=f"layer {layer}"):
        make_config_from_hf(d)


def test_unknown_parts_are_refused():
    for path, value in ((("layers", 0, "type"), "conv"), (("layers", 0, "mlp", "kind"), "sparse"), (("architecture",), "Other"),
                        (("layers", 0, "mlp", "router", "top"), 8)):
        d = copy_of(M.EVEN)
        at = d
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            make_config_from_hf(d)


@pytest.mark.parametrize("dims,base,scaling", [(24, 500.0, (2.0, 1.0, 4.0, 64)), (128, 500000.0, (8.0, 1.0, 4.0, 8192)), (8, 3000.0, (16.0, 0.5, 2.0, 32)),
                                               (2, 100.0, (4.0, 1.0, 4.0, 100)), (16, 77.0, None), (6, 50.0, (1.0, 1.0, 4.0, 16)), (22, 9.0, (5.0, 1.0, 1.0, 40))])
def test_rotary_frequencies(dims, base, scaling):
    names = ("factor", "low", "high", "original")
    d = {"dims": dims, "base": base}
    rot = RotaryConfig(dims, base)
    if scaling is not None:
        d["scaling"] = dict(zip(names, scaling))
        rot = RotaryConfig(dims, base, WavelengthScaling(**d["scaling"]))
    freq, amp = rot.frequencies()
    want = torch.tensor(O.rotary_frequencies(d), dtype=torch.float64)
    torch.testing.assert_close(freq, want, rtol=1e-12, atol=0)
    assert amp == 1.0
    cos, sin = RotaryTable(rot).get(3000, torch.device("cpu"))
    ang = torch.arange(3000, dtype=torch.float64)[:, None] * want
    assert (cos[:3000] - torch.cos(ang)).abs().max() < 2e-7 and (sin[:3000] - torch.sin(ang)).abs().max() < 2e-7


def test_wavelengths_on_the_borders():
    """A pair with exactly ``high`` turns is kept, one with exactly ``low`` is divided."""
    original = 2 * math.pi * 16
    rot = RotaryConfig(4, 16.0, WavelengthScaling(10.0, original, 4.0, 16.0))     # frequencies 1 and 1/4: 16 and 4 turns
    freq, _ = rot.frequencies()
    torch.testing.assert_close(freq, torch.tensor([1.0, 0.025], dtype=torch.float64), rtol=1e-9, atol=0)


def test_registry_and_presets():
    assert registry.infer_arch("difedra-smoke") is registry.Arch.TEXT
    cfg = api.resolve_config("difedra-smoke")
    assert api.model_class_for(cfg).__name__ == "Difedra" and api.is_inference_only(cfg)
    kinds = {type(layer.mlp) for layer in cfg.layers}
    assert kinds == {GatedMLPConfig, MixtureOfExpertsConfig}
    assert api.resolve_config("difedra-8layer-2048").layers[-1].mlp.experts == 128
    with pytest.raises(NotImplementedError):
        api.make_cache(cfg, 1, 8, 8, tp_size=2)
    from omegalax_b200.trainers import text as trainer

    with pytest.raises(NotImplementedError, match="inference only"):
        trainer.init_model("difedra-smoke", 0, tp_size=1, fsdp_size=1, dp_size=1)
    assert len({f.architecture for f in FAMILIES}) == len(FAMILIES)
    for f in FAMILIES:
        for make in f.presets.values():
            assert family_of(make()) is f and f.config_from_hf(f.config_to_hf(make()), {}) == make()
        assert all(p.exists() for p in build.sources(f.kernels))


@pytest.mark.parametrize("cfg_dict", [M.EVEN, M.ODD])
def test_checkpoint_round_trip(tmp_path, cfg_dict):
    w = M.weights(cfg_dict, 0)
    folder = M.write(tmp_path / "a", cfg_dict, w)
    assert registry.infer_arch(str(folder)) is registry.Arch.TEXT
    model, cfg = api.load_model(folder, device="cpu")
    export.export_model_to_hf(model, cfg, tmp_path / "b")
    from safetensors.torch import load_file

    back = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(back) == set(w) and all(torch.equal(back[k], w[k]) for k in w)
    assert export.model_config_to_hf_dict(cfg) == copy_of(cfg_dict)
    again, cfg2 = api.load_model(tmp_path / "b", device="cpu", dtype=torch.float32)
    assert cfg2 == cfg
    for (n, p), (n2, p2) in zip(model.named_parameters(), again.named_parameters()):
        assert n == n2 and torch.equal(p.float(), p2)


def test_incomplete_or_foreign_checkpoints_are_refused(tmp_path):
    w = M.weights(M.EVEN, 0)
    for i, (gone, name) in enumerate([("l0.mlp.e4.up", "experts_gate_up"), ("l1.mix.sink", "sink"), ("l3.mix.k.norm", "qk_norm")]):
        with pytest.raises(RuntimeError, match=name):
            api.load_model(M.write(tmp_path / str(i), M.EVEN, {k: v for k, v in w.items() if k != gone}), device="cpu")
    with pytest.raises(RuntimeError, match="l1.mix.vmix"):       # a layer that mixes no values
        api.load_model(M.write(tmp_path / "x", M.EVEN, {**w, "l1.mix.vmix": w["l0.mix.vmix"]}), device="cpu")


def test_pages_that_left_every_window_go_back():
    c = HybridCache([KeyValuePages(2, 6, 5, 9), KeyValuePages(1, 8, 8, 4)], 2, 80, page_size=4, device="cpu", num_pages=12)
    assert c.horizon == 9 and c.stores[0].shape == (48, 24) and c.stores[1].shape == (48, 16)
    c.reserve([14, 3])
    assert len(c.allocator.free) == 12 - 4 - 1
    c.advance([14, 3])                     # the next token, at 14, sees 6 ... 14: the page of 0 ... 3 is free
    assert len(c.allocator.free) == 8 and c.block_table_host[0, :4].tolist()[0] == -1 and (c.block_table_host[0, 1:4] >= 0).all()
    kept = c.block_table_host[0, 1:4].clone()
    for pos in range(14, 60):
        c.reserve([1, 0])
        c.advance([1, 0])
        first = max(0, pos + 1 - 8)        # first token the next one sees
        held = [j for j in range(c.max_blocks) if c.block_table_host[0, j] >= 0]
        assert held == list(range(first // 4, pos // 4 + 1)) and len(held) <= 4
        pages = c.block_table_host[c.block_table_host >= 0].tolist()
        assert sorted(pages + c.allocator.free) == list(range(12))
        assert c.flat_row_host(0, first) >= 0
    assert kept.tolist() and c.seq_lens_host == [60, 3]
    c.free_sequence(0)
    c.free_sequence(1)
    assert sorted(c.allocator.free) == list(range(12)) and c.blocks_dropped == [0, 0]
    c.reserve([4, 0])
    c.advance([4, 0])
    assert c.flat_rows_host(0, 0, 4).min() >= 0


@pytest.mark.parametrize("other", [LatentPages(8, 8), KeyValuePages(1, 4, 4), RecurrentState(1, 4, 4)])
def test_pages_stay_while_a_layer_reads_them_all(other):
    c = HybridCache([KeyValuePages(1, 4, 4, 3), other], 1, 40, page_size=4, device="cpu")
    c.reserve([33])
    c.advance([33])
    assert (c.horizon == 3) == isinstance(other, RecurrentState)
    assert int((c.block_table_host[0] >= 0).sum()) == (2 if c.horizon else 9)      # tokens 31 ... 33 or all


def test_config_is_a_dataclass_with_replaceable_fields():
    cfg = make_config_from_hf(M.EVEN)
    assert dataclasses.replace(cfg, vocab_size=11).vocab_size == 11 and cfg.num_layers == 5
