"""Plain, slow implementation of the Lotilix decoder, one function per mechanism, whole sequences only.

It shares no code with the engine: float torch (float32, or float64 on request) on whatever device the weights are
on, token by token where the design is a recurrence.  ``forward(weights, config, tokens)`` returns the logits at
every position and, on request, the residual stream after every layer.

The design: a token table; layers ``x += mixer(h) + ff(h)`` whose two sublayers read one RMS norm ``h`` of the
stream; after that each layer adds an input that belongs to the token itself: a row of a second token table (one
part of it per layer), gated by a projection of the stream, projected to the width and RMS-normed.  Three mixers:
softmax attention through low-rank latents over a sliding window (pairs of neighbouring coordinates rotated, a
sigmoid gate per head); a delta rule whose state decays per key channel (short convolutions with silu, unit
queries and keys, a low-rank decay and a low-rank sigmoid output gate); and grouped-query softmax attention inside
chunks of the sequence whose values are its projected, unrotated keys.  The feed-forward is a gated dense layer
with the tanh form of gelu.  The head is an RMS norm and an output matrix.
"""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch
import torch.nn.functional as F


def read_config(model_dir) -> dict:
    return json.loads((Path(model_dir) / "config.json").read_text())


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


# ---- rotation ---------------------------------------------------------------------------------------
def frequencies(rot: dict) -> list[float]:
    """``base^(-2i/dims)``; with ``scaling``, long wavelengths slowed down by ``factor``, short ones kept, those
    between blended linearly in ``original / wavelength``."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            factor, low, high, orig = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            lam = 2.0 * math.pi / f
            if lam > orig / low:
                f = f / factor
            elif lam >= orig / high:
                s = (orig / lam - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate_neighbours(x, positions, rot: dict):
    """``x`` [T, ..., d]: coordinates 2i and 2i + 1 of the first ``dims`` turn by ``position * f_i``."""
    dims = int(rot["dims"])
    f = torch.tensor(frequencies(rot), dtype=torch.float64)
    ang = positions.double().cpu()[:, None] * f[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (dims // 2,)
    c = torch.cos(ang).to(x.device, x.dtype).view(shape)
    s = torch.sin(ang).to(x.device, x.dtype).view(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], -1)


# ---- which keys a position sees -------------------------------------------------------------------------
def window_mask(T: int, size: int, device=None):
    i, j = torch.arange(T, device=device)[:, None], torch.arange(T, device=device)[None, :]
    return (j <= i) & (i - j < size)


def chunk_mask(T: int, size: int, device=None):
    i, j = torch.arange(T, device=device)[:, None], torch.arange(T, device=device)[None, :]
    return (j <= i) & (i // size == j // size)


# ---- mixers -------------------------------------------------------------------------------------------
def latent_attention(w, p: str, h, m: dict, eps: float):
    T = h.shape[0]
    H, D, R, V, C = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    pos = torch.arange(T, device=h.device)
    c_q = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (c_q @ w[p + "uq"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :C], eps) * w[p + "dkv.norm"]
    q_rot = rotate_neighbours(q[..., D:], pos, m["rot"])
    k_rot = rotate_neighbours(down[:, C:], pos, m["rot"])
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    seen = window_mask(T, int(m["mask"]["size"]), h.device)
    out = h.new_zeros(T, H, V)
    for head in range(H):
        s = (q[:, head, :D] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * float(m["scale"])
        out[:, head] = torch.softmax(s.masked_fill(~seen, float("-inf")), -1) @ v[:, head]
    out = out * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return out.reshape(T, H * V) @ w[p + "o"].T


def causal_conv(u, w):
    """``u`` [T, C], ``w`` [C, taps]: ``y_t = sum_j w[:, j] u_(t - taps + 1 + j)``, zeros before the start."""
    T, C = u.shape
    taps = w.shape[1]
    padded = torch.cat([u.new_zeros(taps - 1, C), u], 0)
    return sum(w[:, j] * padded[j: j + T] for j in range(taps))


def delta_recurrence(q, k, v, decay, beta, S=None):
    """``q``, ``k`` [T, G, D]; ``v`` [T, H, V]; ``decay`` [T, H, D]; ``beta`` [T, H].  Per head, in this order:
    ``S <- diag(decay) S``; ``u = beta (v - S^T k)``; ``S <- S + k u^T``; ``o = S^T q``.  Returns (o [T, H, V], S)."""
    T, H, V = v.shape
    G, D = k.shape[1], k.shape[2]
    S = v.new_zeros(H, D, V) if S is None else S.clone()
    group = torch.arange(H, device=v.device) // (H // G)
    o = v.new_zeros(T, H, V)
    for t in range(T):
        kt, qt = k[t, group], q[t, group]                       # [H, D]
        S = decay[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, kt))
        S = S + kt[:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, qt)
    return o, S


def channel_delta(w, p: str, h, m: dict, eps: float):
    T = h.shape[0]
    H, G, D, V = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    q, k, v = (F.silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q, k, v = q.view(T, G, D), k.view(T, G, D), v.view(T, H, V)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    step = F.softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(T, H, D)
    decay = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * step)
    o, _ = delta_recurrence(q, k, v, decay, beta)
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, V)
    o = rms(o, eps) * w[p + "norm"] * gate
    return o.reshape(T, H * V) @ w[p + "o"].T


def chunk_attention(w, p: str, h, m: dict):
    T = h.shape[0]
    H, G, D = (int(m[k]) for k in ("heads", "kv_heads", "dim"))
    pos = torch.arange(T, device=h.device)
    q = (h @ w[p + "q"].T).view(T, H, D)
    v = (h @ w[p + "k"].T).view(T, G, D)                        # the values are the keys before their rotation
    q, k = rotate_neighbours(q, pos, m["rot"]), rotate_neighbours(v, pos, m["rot"])
    out = attend(q, k, v, float(m["scale"]), chunk_mask(T, int(m["mask"]["size"]), h.device))
    return out.reshape(T, H * D) @ w[p + "o"].T


def attend(q, k, v, scale: float, seen):
    """``q`` [T, H, D], ``k`` [T, G, D], ``v`` [T, G, V], ``seen`` [T, T] -> [T, H, V]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = q.new_zeros(T, H, v.shape[2])
    for head in range(H):
        g = head // (H // G)
        s = ((q[:, head] @ k[:, g].T) * scale).masked_fill(~seen, float("-inf"))
        out[:, head] = torch.softmax(s, -1) @ v[:, g]
    return out


# ---- feed-forward, the token's own input ------------------------------------------------------------------
def gated_ff(w, p: str, h):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def token_input(w, p: str, x, e, eps: float):
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return rms(y, eps) * w[p + "norm"]


def forward(weights: dict, config: dict, tokens, dtype=torch.float32, details: bool = False, disturb=None):
    """Logits ``[T, vocab]`` of one whole sequence; ``details``: also the stream after every layer; ``disturb``: applied to
    what every sublayer reads (to see how much a model makes of a rounding)."""
    seen = disturb or (lambda t: t)
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps, side = float(config["norm"]["eps"]), int(config["token_side"]["dim"])
    ids = torch.as_tensor(tokens, dtype=torch.long, device=w["embed"].device)
    x = w["embed"][ids]
    after = []
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = seen(rms(x, eps) * w[p + "norm1"])
        if layer["type"] == "latent_attention":
            y = latent_attention(w, p + "mix.", h, m, eps)
        elif layer["type"] == "channel_delta":
            y = channel_delta(w, p + "mix.", h, m, eps)
        elif layer["type"] == "attention":
            y = chunk_attention(w, p + "mix.", h, m)
        else:
            raise ValueError(f"layer type {layer['type']!r}")
        if layer.get("mlp") is not None:
            y = y + gated_ff(w, p + "mlp.", h)
        x = x + y
        x = x + token_input(w, p + "side.", seen(x), w["side.embed"][ids, i * side: (i + 1) * side], eps)
        after.append(x)
    logits = seen(rms(x, eps) * w["final.norm"]) @ w["head"].T
    return (logits, torch.stack(after)) if details else logits


def generate(weights: dict, config: dict, prompt, n_new: int) -> list[int]:
    """Greedy continuation, the whole sequence run again for every token."""
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(weights, config, toks)[-1].argmax()))
    return toks[len(prompt):]


# ---- random weights of a configuration --------------------------------------------------------------------
def tensor_shapes(config: dict, inner_ranks=(5, 7)) -> dict:
    """``inner_ranks``: the inner sizes of a recurrent layer's low-rank decay and output gate, which only the
    tensors' shapes give."""
    W, V, S = int(config["width"]), int(config["vocab"]), int(config["token_side"]["dim"])
    shapes = {"embed": (V, W), "side.embed": (V, S * len(config["layers"])), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        shapes.update({p + "norm1": (W,), p + "side.gate": (S, W), p + "side.proj": (W, S), p + "side.norm": (W,)})
        H = int(m["heads"])
        if layer["type"] == "latent_attention":
            D, R, Vd, C, Q = (int(m[k]) for k in ("dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            shapes.update({q + "dq": (Q, W), q + "dq.norm": (Q,), q + "uq": (H * (D + R), Q), q + "dkv": (C + R, W),
                           q + "dkv.norm": (C,), q + "uk": (H * D, C), q + "uv": (H * Vd, C), q + "g": (H, W),
                           q + "o": (W, H * Vd)})
        elif layer["type"] == "channel_delta":
            G, D, Vd, taps = (int(m[k]) for k in ("kv_heads", "dim", "vdim", "conv"))
            for n, c in (("q", G * D), ("k", G * D), ("v", H * Vd)):
                shapes.update({q + n: (c, W), q + n + ".conv": (c, taps)})
            ra, rg = inner_ranks
            shapes.update({q + "b": (H, W), q + "A_log": (H,), q + "norm": (Vd,), q + "a1": (ra, W), q + "a2": (H * D, ra),
                           q + "dt_bias": (H * D,), q + "g1": (rg, W), q + "g2": (H * Vd, rg), q + "o": (W, H * Vd)})
        else:
            G, D = int(m["kv_heads"]), int(m["dim"])
            shapes.update({q + "q": (H * D, W), q + "k": (G * D, W), q + "o": (W, H * D)})
        if layer.get("mlp") is not None:
            Fs = int(layer["mlp"]["ff"])
            shapes.update({p + "mlp.gate": (Fs, W), p + "mlp.up": (Fs, W), p + "mlp.down": (W, Fs)})
    return shapes


def draw_weights(config: dict, seed: int, inner_ranks=(5, 7)) -> dict:
    """bfloat16 tensors by name, drawn so that no constant of the design is near neutral: gains away from one, taps of
    every age, decays between slow and fast that differ from channel to channel."""
    g = torch.Generator().manual_seed(seed)
    uni = lambda shape, lo, hi: torch.empty(shape).uniform_(lo, hi, generator=g)  # noqa: E731
    out = {}
    for name, shape in tensor_shapes(config, inner_ranks).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "conv":
            t = uni(shape, -0.5, 0.5)
            t[:, -1] += 1.0
        elif leaf in ("norm1", "norm"):
            t = uni(shape, 0.6, 1.4)
        elif leaf == "A_log":
            t = uni(shape, -2.5, 0.0)
        elif leaf == "dt_bias":
            t = uni(shape, -3.0, 1.0)
        elif name in ("embed", "side.embed"):
            t = torch.randn(shape, generator=g)
        elif name.endswith("side.gate"):      # the stream is several times as large as a normed input
            t = torch.randn(shape, generator=g) * 0.25 / math.sqrt(shape[-1])
        else:
            t = torch.randn(shape, generator=g) * 1.5 / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
