"""Plain, slow implementation of the Gedelorn decoder, one function per mechanism, whole sequences only.

It shares no code with the engine: float torch (float32, or float64 on request) on whatever device the weights are
on, token by token where the design is a recurrence.  ``forward(weights, config, tokens)`` returns the logits at
every position and, on request, the residual stream after every layer.

The design: a token table; layers with a norm before and a norm after each sublayer (gains stored around zero);
three mixers, ``mlstm`` (a matrix memory with exponential input gates, a running maximum and a normaliser),
``mamba2`` (a state-space recurrence with one decay a head behind a short convolution, a gate and a norm in parts)
and ``parallel`` (the weighted sum of a windowed softmax attention whose values are its unrotated keys, with capped
scores, and linear attention with a constant decay a head); gated dense feed-forwards or sigmoid-routed ungated
experts with a shared one; a final norm and an output matrix.
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


def around_zero_norm(x, w, eps: float):
    return rms(x, eps) * (1.0 + w)


# ---- matrix memory with exponential gates ---------------------------------------------------------------
def memory_rows(q, k, v, i_gate, f_gate, state=None):
    """``q``, ``k`` [T, H, D]; ``v`` [T, H, V]; log gates ``i_gate``, ``f_gate`` [T, H].  With a running maximum m:
    ``m' = max(f + m, i)``, ``S <- exp(f + m - m') S + exp(i - m') k v^T``, n likewise with k alone,
    ``o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)``.  Returns (o [T, H, V], (S, n, m))."""
    T, H, D = k.shape
    V = v.shape[2]
    if state is None:
        S, n, m = v.new_zeros(H, D, V), v.new_zeros(H, D), v.new_zeros(H)
    else:
        S, n, m = (t.clone() for t in state)
    o = v.new_zeros(T, H, V)
    for t in range(T):
        top = torch.maximum(f_gate[t] + m, i_gate[t])
        keep, put = torch.exp(f_gate[t] + m - top), torch.exp(i_gate[t] - top)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = top
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        o[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return o, (S, n, m)


def matrix_memory(w, p: str, h, m: dict, eps: float):
    T = h.shape[0]
    H, D, V, cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k, v = (h @ w[p + "k"].T).view(T, H, D), (h @ w[p + "v"].T).view(T, H, V)
    i_gate = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f_gate = F.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o, _ = memory_rows(q, k, v, i_gate, f_gate)
    o = rms(o, eps).reshape(T, H * V) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---- state-space recurrence with one decay a head ---------------------------------------------------------
def causal_conv(u, w, b):
    """``u`` [T, C], ``w`` [C, taps]: ``y_t = b + sum_j w[:, j] u_(t - taps + 1 + j)``, zeros before the start."""
    T, C = u.shape
    taps = w.shape[1]
    padded = torch.cat([u.new_zeros(taps - 1, C), u], 0)
    return sum(w[:, j] * padded[j: j + T] for j in range(taps)) + b


def decayed_rows(q, k, v, decay, put, S=None):
    """``q``, ``k`` [T, H, D]; ``v`` [T, H, V]; ``decay``, ``put`` [T, H]: ``S <- decay S + put k v^T``, ``o = S^T q``.
    Returns (o [T, H, V], S [H, D, V])."""
    T, H, D = k.shape
    S = v.new_zeros(H, D, v.shape[2]) if S is None else S.clone()
    o = v.new_zeros(T, H, v.shape[2])
    for t in range(T):
        S = decay[t][:, None, None] * S + put[t][:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def state_space(w, p: str, h, m: dict, eps: float):
    T = h.shape[0]
    H, V, N, G, parts = (int(m[k]) for k in ("heads", "vdim", "state", "groups", "norm_groups"))
    inner = H * V
    z, u, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], 1)
    u = F.silu(causal_conv(u, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(u, [inner, G * N, G * N], 1)
    x = x.reshape(T, H, V)
    group = torch.arange(H, device=h.device) // (H // G)
    B, C = B.reshape(T, G, N)[:, group], C.reshape(T, G, N)[:, group]
    dt = F.softplus(dt + w[p + "dt_bias"])
    y, _ = decayed_rows(C, B, x, torch.exp(-torch.exp(w[p + "A_log"]) * dt), dt)
    y = (y + w[p + "D"][:, None] * x).reshape(T, inner) * F.silu(z)
    y = rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


# ---- windowed attention whose values are its keys ------------------------------------------------------------
def rotate_neighbours(x, positions, rot: dict):
    """``x`` [T, heads, d]: coordinates 2i and 2i + 1 of the first ``dims`` turn by ``position * base^(-2i/dims)``."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    ang = positions.double().cpu()[:, None] * f[None, :]
    c, s = torch.cos(ang).to(x.device, x.dtype)[:, None, :], torch.sin(ang).to(x.device, x.dtype)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., dims:]], -1)


def window_mask(T: int, size: int, device=None):
    i, j = torch.arange(T, device=device)[:, None], torch.arange(T, device=device)[None, :]
    return (j <= i) & (i - j < size)


def capped_attend(q, k, v, scale: float, cap: float, seen):
    """``q`` [T, H, D], ``k`` [T, G, D], ``v`` [T, G, V], ``seen`` [T, T] -> [T, H, V]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = q.new_zeros(T, H, v.shape[2])
    for head in range(H):
        g = head // (H // G)
        s = cap * torch.tanh((q[:, head] @ k[:, g].T) * scale / cap)
        out[:, head] = torch.softmax(s.masked_fill(~seen, float("-inf")), -1) @ v[:, g]
    return out


def key_valued_attention(w, p: str, h, m: dict):
    T = h.shape[0]
    H, G, D = (int(m[k]) for k in ("heads", "kv_heads", "dim"))
    pos = torch.arange(T, device=h.device)
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, D)
    v = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, D)              # the values are the keys before their rotation
    q, k = rotate_neighbours(q, pos, m["rot"]), rotate_neighbours(v, pos, m["rot"])
    out = capped_attend(q, k, v, float(m["scale"]), float(m["softcap"]), window_mask(T, int(m["mask"]["size"]), h.device))
    return out.reshape(T, H * D) @ w[p + "o"].T


# ---- linear attention with a constant decay a head -----------------------------------------------------------
def constant_decay_attention(w, p: str, h, m: dict, eps: float):
    T = h.shape[0]
    H, D, V = (int(m[k]) for k in ("heads", "dim", "vdim"))
    q, k, v = (F.silu(h @ w[p + n].T).view(T, H, d) for n, d in (("q", D), ("k", D), ("v", V)))
    decay = torch.tensor([float(x) for x in m["decay"]], dtype=h.dtype, device=h.device).expand(T, H)
    o, _ = decayed_rows(q, k, v, decay, torch.ones_like(decay))
    return (rms(o.reshape(T, H * V), eps) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(w, p: str, h, m: dict, eps: float):
    return float(m["left_scale"]) * key_valued_attention(w, p + "left.", h, m["left"]) + \
        float(m["right_scale"]) * constant_decay_attention(w, p + "right.", h, m["right"], eps)


# ---- feed-forwards -------------------------------------------------------------------------------------------
def gated_ff(w, p: str, h):
    return (F.silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def squared_expert(w, p: str, h):
    return (F.relu(h @ w[p + "up"].T) ** 2) @ w[p + "down"].T


def routed_ff(w, p: str, h, m: dict, chosen=None):
    """The ``top`` largest of the sigmoid scores (or the experts ``chosen`` [T, top]); their weights are the scores divided
    by their sum, times ``scale``; a shared expert is added.  Returns (output, chosen [T, top], margin [T]: last chosen over first not chosen)."""
    E, top, scale = int(m["router"]["experts"]), int(m["router"]["top"]), float(m["router"]["scale"])
    s = torch.sigmoid(h @ w[p + "router"].T)
    order = torch.sort(s, dim=-1, descending=True, stable=True)
    idx, val = order.indices[:, :top], order.values[:, :top]
    margin = val[:, -1] - order.values[:, top] if E > top else torch.full_like(s[:, 0], 1e9)
    if chosen is not None:
        idx = chosen.long()
        val = s.gather(1, idx)
    weight = val / (val.sum(-1, keepdim=True) + 1e-20) * scale
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(top):
            out[t] += weight[t, j] * squared_expert(w, f"{p}e{int(idx[t, j])}.", h[t:t + 1])[0]
    if m.get("shared") is not None:
        out = out + squared_expert(w, p + "shared.", h)
    return out, idx, margin


# ---- the whole model -----------------------------------------------------------------------------------------
def forward(weights: dict, config: dict, tokens, dtype=torch.float32, details: bool = False, disturb=None,
            margins: list | None = None, chosen=None):
    """Logits ``[T, vocab]`` of one whole sequence; ``details``: also the stream after every layer; ``disturb``: applied
    to what every sublayer reads (to see how much a model makes of a rounding); ``margins`` receives the routers'; ``chosen``: per
    routed layer, experts [T, top] to take instead of choosing."""
    seen = disturb or (lambda t: t)
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    ids = torch.as_tensor(tokens, dtype=torch.long, device=w["embed"].device)
    x = w["embed"][ids]
    after, routed = [], 0
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = seen(around_zero_norm(x, w[p + "norm1"], eps))
        if layer["type"] == "mlstm":
            y = matrix_memory(w, p + "mix.", h, m, eps)
        elif layer["type"] == "mamba2":
            y = state_space(w, p + "mix.", h, m, eps)
        elif layer["type"] == "parallel":
            y = side_by_side(w, p + "mix.", h, m, eps)
        else:
            raise ValueError(f"layer type {layer['type']!r}")
        x = x + around_zero_norm(y, w[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = seen(around_zero_norm(x, w[p + "norm2"], eps))
            if mlp["kind"] == "dense":
                y = gated_ff(w, p + "mlp.", h)
            else:
                y, _, margin = routed_ff(w, p + "mlp.", h, mlp, None if chosen is None else chosen[routed])
                routed += 1
                if margins is not None:
                    margins.append(margin)
            x = x + around_zero_norm(y, w[p + "norm2b"], eps)
        after.append(x)
    logits = seen(around_zero_norm(x, w["final.norm"], eps)) @ w["head"].T
    return (logits, torch.stack(after)) if details else logits


def generate(weights: dict, config: dict, prompt, n_new: int) -> list[int]:
    """Greedy continuation, the whole sequence run again for every token."""
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(weights, config, toks)[-1].argmax()))
    return toks[len(prompt):]


# ---- random weights of a configuration --------------------------------------------------------------------
def tensor_shapes(config: dict) -> dict:
    W, vocab = int(config["width"]), int(config["vocab"])
    shapes = {"embed": (vocab, W), "final.norm": (W,), "head": (vocab, W)}
    for i, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        q = p + "mix."
        shapes.update({p + "norm1": (W,), p + "norm1b": (W,)})
        if layer["type"] == "mlstm":
            H, D, V = (int(m[k]) for k in ("heads", "dim", "vdim"))
            shapes.update({q + "q": (H * D, W), q + "k": (H * D, W), q + "v": (H * V, W), q + "g": (H * V, W),
                           q + "o": (W, H * V), q + "norm": (H * V,), q + "i": (H, W), q + "i.b": (H,), q + "f": (H, W),
                           q + "f.b": (H,)})
        elif layer["type"] == "mamba2":
            H, V, N, G, taps = (int(m[k]) for k in ("heads", "vdim", "state", "groups", "conv"))
            C = H * V + 2 * G * N
            shapes.update({q + "in": (H * V + C + H, W), q + "conv": (C, taps), q + "conv.b": (C,), q + "dt_bias": (H,),
                           q + "A_log": (H,), q + "D": (H,), q + "norm": (H * V,), q + "o": (W, H * V)})
        else:
            L, R = m["left"], m["right"]
            H, G, D = (int(L[k]) for k in ("heads", "kv_heads", "dim"))
            shapes.update({q + "left.q": (H * D, W), q + "left.q.b": (H * D,), q + "left.k": (G * D, W),
                           q + "left.k.b": (G * D,), q + "left.o": (W, H * D)})
            H, D, V = (int(R[k]) for k in ("heads", "dim", "vdim"))
            shapes.update({q + "right.q": (H * D, W), q + "right.k": (H * D, W), q + "right.v": (H * V, W),
                           q + "right.g": (H * V, W), q + "right.o": (W, H * V), q + "right.norm": (H * V,)})
        if mlp is None:
            continue
        shapes.update({p + "norm2": (W,), p + "norm2b": (W,)})
        if mlp["kind"] == "dense":
            I = int(mlp["ff"])
            shapes.update({p + "mlp.gate": (I, W), p + "mlp.up": (I, W), p + "mlp.down": (W, I)})
        else:
            I = int(mlp["expert"]["ff"])
            shapes[p + "mlp.router"] = (int(mlp["router"]["experts"]), W)
            for e in range(int(mlp["router"]["experts"])):
                shapes.update({f"{p}mlp.e{e}.up": (I, W), f"{p}mlp.e{e}.down": (W, I)})
            if mlp.get("shared") is not None:
                I = int(mlp["shared"]["ff"])
                shapes.update({p + "mlp.shared.up": (I, W), p + "mlp.shared.down": (W, I)})
    return shapes


def draw_weights(config: dict, seed: int) -> dict:
    """bfloat16 tensors by name, drawn so that no constant of the design is near neutral: gains away from one, taps of
    every age, decays between slow and fast, input gates that take over the running maximum now and then."""
    g = torch.Generator().manual_seed(seed)
    uni = lambda shape, lo, hi: torch.empty(shape).uniform_(lo, hi, generator=g)  # noqa: E731
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            t = uni(shape, -0.4, 0.4)
        elif leaf == "norm":
            t = uni(shape, 0.6, 1.4)
        elif leaf == "conv":
            t = uni(shape, -0.5, 0.5)
            t[:, -1] += 1.0
        elif leaf == "A_log":
            t = uni(shape, -2.5, 0.5)
        elif leaf == "dt_bias":
            t = uni(shape, -3.0, 1.0)
        elif leaf == "D":
            t = uni(shape, -1.0, 1.0)
        elif name.endswith(".f.b"):
            t = uni(shape, 0.0, 4.0)
        elif name.endswith(".i.b"):
            t = uni(shape, -2.0, 1.0)
        elif leaf == "b":
            t = uni(shape, -0.5, 0.5)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * 1.5 / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
