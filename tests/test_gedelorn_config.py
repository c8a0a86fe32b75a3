"""Configuration, specification, tensor list, page retention and per-request state of the Gedelorn decoder (no GPU)."""

import copy

import pytest
import torch

from quanta_b200.config import ConfigError, GedelornConfig
from quanta_b200.config.registry import resolve
from tests.plain import gedelorn_plain as P

RAW = {"architecture": "Gedelorn", "vocab": 50, "width": 36, "norm": {"eps": 1e-4}, "layers": [
    {"type": "mlstm", "mixer": {"heads": 3, "dim": 10, "vdim": 14, "gate_cap": 7.0},
     "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 5, "top": 2, "scale": 1.4}, "shared": {"ff": 20}}},
    {"type": "mamba2", "mlp": {"kind": "dense", "ff": 24},
     "mixer": {"heads": 6, "vdim": 8, "state": 9, "groups": 3, "conv": 5, "norm_groups": 4}},
    {"type": "parallel", "mlp": None,
     "mixer": {"left": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 12, "scale": 0.25, "softcap": 5.0, "mask": {"size": 11},
                        "rot": {"dims": 8, "base": 30.0}},
               "right": {"heads": 2, "dim": 6, "vdim": 10, "decay": [0.5, 0.99]}, "left_scale": 0.7, "right_scale": 1.3}}]}


def test_registry_finds_the_architecture_by_its_key():
    assert resolve(RAW).name == "Gedelorn"
    assert resolve({"architectures": ["Gedelorn"]}).config_cls is GedelornConfig


def test_fields_and_round_trip():
    cfg = GedelornConfig.from_dict(RAW)
    assert (cfg.vocab, cfg.width, cfg.norm_eps) == (50, 36, 1e-4)
    assert [l.type for l in cfg.layers] == ["mlstm", "mamba2", "parallel"]
    again = GedelornConfig.from_dict(cfg.to_dict())
    assert again == cfg and again.to_dict() == cfg.to_dict()


LEFT, RIGHT = (lambda r: r["layers"][2]["mixer"]["left"]), (lambda r: r["layers"][2]["mixer"]["right"])


@pytest.mark.parametrize("change,what", [
    (lambda r: r["layers"][0].update(type="attention"), "type"),
    (lambda r: r["layers"][1]["mlp"].update(kind="sparse"), "kind"),
    (lambda r: r["layers"][1]["mlp"].update(ff=0), "ff"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda r: r["layers"][0]["mlp"]["router"].pop("scale"), "lacks"),
    (lambda r: r["layers"][0]["mlp"]["shared"].update(ff=0), "shared"),
    (lambda r: r["layers"][0]["mixer"].pop("gate_cap"), "lacks"),
    (lambda r: r["layers"][0]["mixer"].update(gate_cap=0.0), "gate_cap"),
    (lambda r: r["layers"][0]["mixer"].update(dim=300), "between"),
    (lambda r: r["layers"][1]["mixer"].update(groups=4), "multiple"),
    (lambda r: r["layers"][1]["mixer"].update(norm_groups=5), "divide"),
    (lambda r: r["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda r: r["layers"][1]["mixer"].update(state=257), "between"),
    (lambda r: LEFT(r).update(kv_heads=3), "multiple"),
    (lambda r: LEFT(r).update(vdim=16), "keys"),
    (lambda r: LEFT(r)["mask"].update(size=0), "mask"),
    (lambda r: LEFT(r).update(softcap=0.0), "softcap"),
    (lambda r: LEFT(r)["rot"].update(dims=7), "even"),
    (lambda r: LEFT(r)["rot"].update(dims=14), "at most"),
    (lambda r: RIGHT(r).update(decay=[0.5]), "decay"),
    (lambda r: RIGHT(r).update(decay=[0.5, 1.5]), "decay"),
    (lambda r: r["layers"][2]["mixer"].pop("right_scale"), "lacks"),
    (lambda r: r.pop("norm"), "norm"),
])
def test_refusals(change, what):
    raw = copy.deepcopy(RAW)
    change(raw)
    with pytest.raises(ConfigError, match=what):
        GedelornConfig.from_dict(raw)


def _model(raw=RAW):
    from quanta_b200 import models  # noqa: F401
    from quanta_b200.engine.model import Model
    return Model(resolve(raw).build_spec(GedelornConfig.from_dict(raw)), dtype=torch.float32, device="cpu")


def test_the_model_asks_for_exactly_the_tensors_of_the_design():
    from quanta_b200.weights.loader import DictSource, WeightError
    want = P.tensor_shapes(RAW)
    assert {s.name: tuple(s.shape) for s in _model().tensor_specs()} == want
    weights = P.draw_weights(RAW, seed=1)
    model = _model()
    model.load(DictSource(weights))
    # gains are stored minus one; the fused projection holds the named matrices below each other
    assert torch.equal(model.blocks[0].mixer_norm.weight, 1 + weights["l0.norm1"].float())
    memory = model.blocks[0].mixer
    for name, at in (("q", 0), ("k", 30), ("v", 60), ("g", memory.g_off), ("i", memory.i_off), ("f", memory.i_off + 3)):
        rows = weights[f"l0.mix.{name}"].float()
        assert torch.equal(memory.w_in[at: at + rows.shape[0]], rows), name
    left = model.blocks[2].mixer.left
    assert torch.equal(left.b_qkv, torch.cat([weights["l2.mix.left.q.b"], weights["l2.mix.left.k.b"]]).float())
    assert left.w_qkv.shape[0] == 72 and left.b_o is None          # 48 + 24 rows: the values have none of their own
    weights.pop("l1.mix.conv.b")
    with pytest.raises(WeightError, match="l1.mix.conv.b"):
        _model().load(DictSource(weights))


def test_a_layer_without_shared_expert_or_feed_forward_asks_for_neither():
    raw = copy.deepcopy(RAW)
    raw["layers"][0]["mlp"]["shared"] = None
    raw["layers"][1]["mlp"] = None
    names = {s.name for s in _model(raw).tensor_specs()}
    assert names == set(P.tensor_shapes(raw))
    assert not any("shared" in n for n in names) and "l1.norm2" not in names


def test_cache_and_state_needs():
    from quanta_b200.parts import Window
    model = _model()
    memory, ssm, par = model.cache_needs()
    assert memory is None and ssm is None and par.retention == Window(11)
    assert [(s.heads, s.width) for s in par.streams] == [(2, 12), (2, 12)]
    state = model.state_needs()
    assert sorted(shape for shape, _ in state[0].values()) == [(3,), (3, 10), (3, 10, 14)]
    assert sorted(shape for shape, _ in state[1].values()) == [(4, 6 * 8 + 2 * 3 * 9), (6, 9, 8)]
    assert [shape for shape, _ in state[2].values()] == [(2, 6, 10)]
    assert all(dtype == torch.float32 for s in state for _, dtype in s.values())
    raw = copy.deepcopy(RAW)
    raw["layers"][1]["mixer"]["conv"] = 1                        # one tap looks at no earlier token
    assert list(_model(raw).state_needs()[1].values()) == [((6, 9, 8), torch.float32)]


def test_constant_decays_are_taken_as_float32_in_both_forms():
    from quanta_b200.kernels import DecayGates
    gates = DecayGates.constant(torch.tensor([0.999, 1.0, 0.0, 0.5]))
    back = torch.exp(gates.t["log_decay"].double())
    assert float((back - gates.t["decay"].double()).abs().max()) < 3e-9 and float(gates.t["log_decay"][1]) == 0.0


def test_entry_points_of_the_recurrence_are_a_unit_of_their_own():
    from quanta_b200.csrc import build
    where = build.entry_points()
    assert build.UNITS["decay_state"] == ["decay_state.cu"] and build.UNITS["short_conv"] == ["short_conv.cu"]
    assert {where[n] for n in ("qb_decay_chain", "qb_decay_chunks", "qb_memory_gates", "qb_decay_out", "qb_rows_act")} == {"decay_state"}
