"""Gedelorn decoder: from its configuration to a model specification.

A token table; layers ``l<i>.`` with an RMS norm before and one after each sublayer, gains stored around zero,
``x += norm1b(mixer(norm1(x)))`` and, where the layer has a feed-forward, ``x += norm2b(ff(norm2(x)))``.  Three mixers:
``mlstm`` (a matrix memory with exponential gates, a running maximum and a normaliser), ``mamba2`` (a state-space
recurrence with one decay a head behind a short convolution, gated before its norm in parts) and ``parallel`` (the
weighted sum of a windowed grouped-query attention with capped scores, interleaved rotation and values that are its
projected keys, and linear attention with a constant decay a head).  Feed-forwards are gated dense layers with silu, or
sigmoid-routed ungated experts with a shared one.  The head is an RMS norm and an output matrix of its own.
"""

from __future__ import annotations

from ..config.gedelorn import GedelornConfig
from ..config.registry import register_architecture
from ..parts.spec import ModelSpec


def window_attention(cfg: GedelornConfig, p: str, m: dict) -> tuple[str, dict]:
    D = int(m["dim"])
    rot = m["rot"] or {}
    dims = int(rot.get("dims") or 0)
    position = ("partial_rotary", dict(head_dim=D, rotary_dim=dims, theta=float(rot["base"]), interleaved=True,
                                       float64_ladder=True)) if dims else ("none", {})
    return ("window_attention", dict(
        hidden_size=cfg.width, n_q_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), head_dim=D, scale=float(m["scale"]),
        window=int(m["mask"]["size"]), norm_eps=cfg.norm_eps, position=position, biases=True, softcap=float(m["softcap"]),
        values_from_keys=True, names={"q": p + "q", "q_b": p + "q.b", "k": p + "k", "k_b": p + "k.b", "o": p + "o"}))


def mixer(cfg: GedelornConfig, i: int) -> tuple[str, dict]:
    layer = cfg.layers[i]
    m, p = layer.mixer, f"l{i}.mix."
    if layer.type == "mlstm":
        return ("matrix_memory", dict(
            hidden_size=cfg.width, n_heads=int(m["heads"]), dim=int(m["dim"]), value_dim=int(m["vdim"]),
            gate_cap=float(m["gate_cap"]), norm_eps=cfg.norm_eps,
            names=dict({k: p + k for k in ("q", "k", "v", "g", "i", "f", "norm", "o")}, i_b=p + "i.b", f_b=p + "f.b")))
    if layer.type == "mamba2":
        return ("state_space_dual", dict(
            hidden_size=cfg.width, n_heads=int(m["heads"]), n_groups=int(m["groups"]), n_state=int(m["state"]),
            value_dim=int(m["vdim"]), conv_taps=int(m["conv"]), norm_groups=int(m["norm_groups"]), norm_eps=cfg.norm_eps,
            names=dict({k: p + k for k in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")}, conv_b=p + "conv.b")))
    right = m["right"]
    linear = ("constant_decay_attention", dict(
        hidden_size=cfg.width, n_heads=int(right["heads"]), dim=int(right["dim"]), value_dim=int(right["vdim"]),
        decay=tuple(float(d) for d in right["decay"]), norm_eps=cfg.norm_eps,
        names={k: p + "right." + k for k in ("q", "k", "v", "g", "norm", "o")}))
    return ("parallel_mixers", dict(left=window_attention(cfg, p + "left.", m["left"]), right=linear,
                                    left_scale=float(m["left_scale"]), right_scale=float(m["right_scale"])))


def feed_forward(cfg: GedelornConfig, i: int) -> tuple[str, dict]:
    mlp, p = cfg.layers[i].mlp, f"l{i}.mlp."
    if mlp["kind"] == "dense":
        return ("gated_dense", dict(hidden_size=cfg.width, inner_size=int(mlp["ff"]),
                                    names={k: p + k for k in ("gate", "up", "down")}))
    router, shared = mlp["router"], mlp.get("shared")
    return ("sigmoid_ungated_experts", dict(
        hidden_size=cfg.width, expert_size=int(mlp["expert"]["ff"]), n_experts=int(router["experts"]), top_k=int(router["top"]),
        scaling=float(router["scale"]), shared_size=0 if shared is None else int(shared["ff"]),
        names={"gate": p + "router", "up": p + "e{e}.up", "down": p + "e{e}.down", "shared_up": p + "shared.up",
               "shared_down": p + "shared.down"}))


def norm(cfg: GedelornConfig, name: str) -> tuple[str, dict]:
    return ("rms_norm", dict(width=cfg.width, eps=cfg.norm_eps, weight_name=name, around_zero=True))


def layer_choice(cfg: GedelornConfig, i: int) -> tuple[str, dict]:
    p = f"l{i}."
    params = dict(hidden_size=cfg.width, mixer=mixer(cfg, i), mixer_norm=norm(cfg, p + "norm1"),
                  mixer_post_norm=norm(cfg, p + "norm1b"))
    if cfg.layers[i].mlp is not None:
        params.update(feed_forward=feed_forward(cfg, i), feed_forward_norm=norm(cfg, p + "norm2"),
                      feed_forward_post_norm=norm(cfg, p + "norm2b"))
    return ("sandwich_norm", params)


def build_spec(cfg: GedelornConfig) -> ModelSpec:
    return ModelSpec(
        name="Gedelorn", vocab_size=cfg.vocab, hidden_size=cfg.width, embedding_name="embed",
        layers=[layer_choice(cfg, i) for i in range(len(cfg.layers))], final_norm=norm(cfg, "final.norm"), head_name="head",
        tied_head=False)


ARCHITECTURE = register_architecture(["Gedelorn", "gedelorn"], GedelornConfig, build_spec)
