"""Configuration, specification, tensor list and page retention of the Lotilix decoder (no GPU)."""

import copy
import math

import pytest
import torch

from quanta_b200.config import ConfigError, LotilixConfig
from quanta_b200.config.registry import resolve
from tests.plain import lotilix_plain as P

RAW = {"architecture": "Lotilix", "vocab": 50, "width": 36, "norm": {"eps": 1e-4}, "token_side": {"dim": 7}, "layers": [
    {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 24},
     "mixer": {"heads": 3, "dim": 10, "rot_dim": 6, "vdim": 14, "q_rank": 20, "kv_rank": 18, "scale": 0.3, "mask": {"size": 9},
               "rot": {"base": 100.0, "dims": 6}}},
    {"type": "channel_delta", "mlp": None,
     "mixer": {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 14, "conv": 5, "decay_rank": 4, "gate_rank": 9}},
    {"type": "attention", "mlp": {"kind": "dense", "ff": 40},
     "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 12, "scale": 0.25, "mask": {"size": 11},
               "rot": {"dims": 8, "base": 30.0, "scaling": {"factor": 3.0, "low": 1.0, "high": 3.0, "original": 40}}}}]}


def test_registry_finds_the_architecture_by_its_key():
    assert resolve(RAW).name == "Lotilix"
    assert resolve({"architectures": ["Lotilix"]}).config_cls is LotilixConfig


def test_fields_and_round_trip():
    cfg = LotilixConfig.from_dict(RAW)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.side_dim) == (50, 36, 1e-4, 7)
    assert [l.type for l in cfg.layers] == ["latent_attention", "channel_delta", "attention"]
    again = LotilixConfig.from_dict(cfg.to_dict())
    assert again == cfg and again.to_dict() == cfg.to_dict()


@pytest.mark.parametrize("change,what", [
    (lambda r: r["layers"][0].update(type="softmax"), "type"),
    (lambda r: r["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda r: r["layers"][2]["mlp"].update(ff=0), "ff"),
    (lambda r: r["layers"][0]["mixer"].pop("q_rank"), "lacks"),
    (lambda r: r["layers"][0]["mixer"].update(kv_rank=600), "kv_rank"),
    (lambda r: r["layers"][0]["mixer"].update(rot_dim=5), "even"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=4), "rot_dim"),
    (lambda r: r["layers"][0]["mixer"]["mask"].update(size=0), "mask"),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda r: r["layers"][1]["mixer"].update(dim=300), "between"),
    (lambda r: r["layers"][1]["mixer"].update(conv=0), "tap"),
    (lambda r: r["layers"][2]["mixer"].update(vdim=16), "keys"),
    (lambda r: r["layers"][2]["mixer"]["rot"].update(dims=7), "even"),
    (lambda r: r["layers"][2]["mixer"]["rot"]["scaling"].pop("low"), "scaling"),
    (lambda r: r["layers"][2]["mixer"]["rot"]["scaling"].update(high=0.5), "low < high"),
    (lambda r: r["layers"][2]["mixer"].pop("mask"), "lacks"),
    (lambda r: r.pop("token_side"), "token_side"),
    (lambda r: r.pop("norm"), "norm"),
])
def test_refusals(change, what):
    raw = copy.deepcopy(RAW)
    change(raw)
    with pytest.raises(ConfigError, match=what):
        LotilixConfig.from_dict(raw)


def test_inner_ranks_come_from_the_tensor_shapes():
    raw = copy.deepcopy(RAW)
    for key in ("decay_rank", "gate_rank"):
        raw["layers"][1]["mixer"].pop(key)
    shapes = P.tensor_shapes(raw, inner_ranks=(11, 3))
    cfg = LotilixConfig.from_dict(raw).with_tensor_shapes(shapes.get)
    assert (cfg.layers[1].mixer["decay_rank"], cfg.layers[1].mixer["gate_rank"]) == (11, 3)
    assert "decay_rank" not in cfg.layers[0].mixer


def test_the_model_asks_for_exactly_the_tensors_of_the_design():
    from quanta_b200 import models  # noqa: F401
    from quanta_b200.engine.model import Model
    from quanta_b200.weights.loader import DictSource, WeightError
    cfg = LotilixConfig.from_dict(RAW)
    arch = resolve(RAW)
    model = Model(arch.build_spec(cfg), dtype=torch.float32, device="cpu")
    want = P.tensor_shapes(RAW, inner_ranks=(4, 9))
    assert {s.name: tuple(s.shape) for s in model.tensor_specs()} == want
    weights = P.draw_weights(RAW, seed=1, inner_ranks=(4, 9))
    model.load(DictSource(weights))
    # one table for all layers, loaded once
    assert len({b.token_input.table.data_ptr() for b in model.blocks}) == 1
    weights.pop("l1.mix.g2")
    with pytest.raises(WeightError, match="l1.mix.g2"):
        Model(arch.build_spec(cfg), dtype=torch.float32, device="cpu").load(DictSource(weights))


def test_cache_and_state_needs():
    from quanta_b200 import models  # noqa: F401
    from quanta_b200.engine.model import Model
    from quanta_b200.parts import OwnChunk, Window
    model = Model(resolve(RAW).build_spec(LotilixConfig.from_dict(RAW)), dtype=torch.float32, device="cpu")
    latent, none, attn = model.cache_needs()
    assert none is None and latent.retention == Window(9) and attn.retention == OwnChunk(11)
    assert [(s.heads, s.width) for s in latent.streams] == [(1, 24)]
    assert [(s.heads, s.width) for s in attn.streams] == [(2, 12), (2, 12)]
    state = model.state_needs()
    assert state[0] == {} and state[2] == {}
    assert sorted(shape for shape, _ in state[1].values()) == [(4, 2 * 3 * 10 + 6 * 14), (6, 10, 14)]


@pytest.mark.parametrize("chunk,page", [(11, 4), (8, 4), (3, 4), (1, 4), (20, 4), (4, 8)])
def test_pages_of_finished_chunks_go_back(chunk, page):
    """After every step a request holds exactly the pages of its open chunk; positions of earlier chunks that share a
    page with it stay."""
    from quanta_b200.cache.manager import CacheManager
    from quanta_b200.parts import CacheSpec, CacheStream, OwnChunk
    mgr = CacheManager([CacheSpec((CacheStream("k", 1, 4),), OwnChunk(chunk))], page, 40, 2)
    mgr.add_request("a")
    n = 0
    for step in (1, 2, 1, 7, 5, 1, 1, 13, 2, 30, 1):
        mgr.reserve("a", n + step)
        mgr.advance("a", step)
        n += step
        first = n // chunk * chunk                      # what the next token's chunk starts with
        table = mgr.block_table_rows(0, ["a"])[0]
        for i, p in enumerate(table):
            needed = (i + 1) * page > first
            assert (p >= 0) == needed, (n, i, table)
        mgr.check_invariants()
    mgr.free("a")
    assert mgr.stats()["groups"][0]["used"] == 0


def test_rotation_ladder_is_float64_rounded_once():
    from quanta_b200.parts.rotary import PartialRotary
    for rot in ({"dims": 16, "base": 500000.0}, {"dims": 10, "base": 30.0},
                {"dims": 40, "base": 9000.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 256}}):
        sc = rot.get("scaling")
        part = PartialRotary(head_dim=rot["dims"], rotary_dim=rot["dims"], theta=rot["base"], interleaved=True,
                             float64_ladder=True,
                             wavelength_scaling=None if sc is None else tuple(sc[k] for k in ("factor", "low", "high", "original")))
        want = torch.tensor(P.frequencies(rot), dtype=torch.float64)
        assert torch.equal(part.inv_freq(), want.float())
        if sc is not None:          # all three ranges are there: kept, blended, slowed down
            plain = torch.tensor(P.frequencies({k: rot[k] for k in ("dims", "base")}), dtype=torch.float64)
            ratio = plain / want
            assert float(ratio.min()) == 1.0 and math.isclose(float(ratio.max()), sc["factor"])
            assert bool(((ratio > 1.001) & (ratio < sc["factor"] - 0.001)).any())
