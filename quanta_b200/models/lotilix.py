"""Lotilix decoder: from its configuration to a model specification.

A token table; layers ``l<i>.`` whose mixer and feed-forward read one RMS norm of the stream and join it together,
``x += mixer(h) + ff(h)``, followed by the token's own input: the layer's part of the token's row of a second table,
gated by a projection of the new stream, projected back and RMS-normed.  Three mixers: ``latent_attention`` (softmax
attention through low-rank latents over a sliding window, one rotated key part for all heads, a sigmoid gate per
head), ``channel_delta`` (a gated delta rule with a decay per key channel and a low-rank sigmoid output gate) and
``attention`` (grouped-query softmax attention inside chunks of the sequence whose values are the projected,
unrotated keys; frequencies rescaled by wavelength).  All rotations pair neighbouring coordinates.  Feed-forwards are
gated dense layers with the tanh form of gelu.  The head is an RMS norm and an output matrix of its own.
"""

from __future__ import annotations

from ..config.lotilix import DEFAULT_INNER_RANK, LotilixConfig
from ..config.registry import register_architecture
from ..parts.spec import ModelSpec

# what the design fixes
UNIT_EPS = 1e-6                # under the root that makes the recurrence's q and k unit vectors


def rotation(rot: dict | None, head_dim: int, dims: int) -> tuple[str, dict]:
    if not dims:
        return ("none", {})
    sc = rot.get("scaling")
    scaling = None if sc is None else (float(sc["factor"]), float(sc["low"]), float(sc["high"]), float(sc["original"]))
    return ("partial_rotary", dict(head_dim=head_dim, rotary_dim=dims, theta=float(rot["base"]),
                                   wavelength_scaling=scaling, interleaved=True, float64_ladder=True))


def mixer(cfg: LotilixConfig, i: int) -> tuple[str, dict]:
    layer = cfg.layers[i]
    m, p = layer.mixer, f"l{i}.mix."
    if layer.type == "latent_attention":
        R = int(m["rot_dim"])
        return ("latent_attention", dict(
            hidden_size=cfg.width, n_heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=R, value_dim=int(m["vdim"]),
            q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), norm_eps=cfg.norm_eps,
            position=rotation(m["rot"], R, R), sink=False, window=int(m["mask"]["size"]), float32_weights=True,
            names={"dq": p + "dq", "dq_norm": p + "dq.norm", "uq": p + "uq", "dkv": p + "dkv", "dkv_norm": p + "dkv.norm",
                   "uk": p + "uk", "uv": p + "uv", "g": p + "g", "o": p + "o"}))
    if layer.type == "channel_delta":
        names = {k: p + k for k in ("q", "k", "v", "b", "A_log", "dt_bias", "norm", "a1", "a2", "g1", "g2", "o")}
        names.update({f"{k}_conv": f"{p}{k}.conv" for k in ("q", "k", "v")})
        return ("gated_delta_rule", dict(
            hidden_size=cfg.width, n_heads=int(m["heads"]), n_groups=int(m["kv_heads"]), dim=int(m["dim"]),
            value_dim=int(m["vdim"]), conv_taps=int(m["conv"]), q_scale=float(int(m["dim"]) ** -0.5), unit_eps=UNIT_EPS,
            norm_eps=cfg.norm_eps, decay_rank=int(m.get("decay_rank", DEFAULT_INNER_RANK)),
            gate_rank=int(m.get("gate_rank", DEFAULT_INNER_RANK)), gate_activation="sigmoid", names=names))
    D = int(m["dim"])
    rot = m.get("rot")
    return ("gqa_attention", dict(
        hidden_size=cfg.width, n_q_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), head_dim=D,
        scale=float(m["scale"]), position=rotation(rot, D, 0 if rot is None else int(rot.get("dims") or 0)),
        qk_norm=None, qk_norm_eps=cfg.norm_eps, names={"q": p + "q", "k": p + "k", "o": p + "o"}, float32_output=True,
        float32_weights=True, float32_projection=True, values_from_keys=True, chunk=int(m["mask"]["size"])))


def layer_choice(cfg: LotilixConfig, i: int) -> tuple[str, dict]:
    layer, p = cfg.layers[i], f"l{i}."
    norm = lambda n: ("rms_norm", dict(width=cfg.width, eps=cfg.norm_eps, weight_name=p + n))  # noqa: E731
    feed_forward = None
    if layer.mlp is not None:
        feed_forward = ("gated_dense", dict(hidden_size=cfg.width, inner_size=int(layer.mlp["ff"]), activation="gelu_tanh",
                                            names={k: f"{p}mlp.{k}" for k in ("gate", "up", "down")}))
    side = ("gated_token_row", dict(hidden_size=cfg.width, vocab_size=cfg.vocab, dim=cfg.side_dim, index=i,
                                    layers=len(cfg.layers), norm=norm("side.norm"),
                                    names={"table": "side.embed", "gate": p + "side.gate", "proj": p + "side.proj"}))
    return ("parallel_residual", dict(hidden_size=cfg.width, mixer=mixer(cfg, i), norm=norm("norm1"),
                                      feed_forward=feed_forward, token_input=side))


def build_spec(cfg: LotilixConfig) -> ModelSpec:
    return ModelSpec(
        name="Lotilix", vocab_size=cfg.vocab, hidden_size=cfg.width, embedding_name="embed",
        layers=[layer_choice(cfg, i) for i in range(len(cfg.layers))],
        final_norm=("rms_norm", dict(width=cfg.width, eps=cfg.norm_eps, weight_name="final.norm")), head_name="head",
        tied_head=False)


ARCHITECTURE = register_architecture(["Lotilix", "lotilix"], LotilixConfig, build_spec)
