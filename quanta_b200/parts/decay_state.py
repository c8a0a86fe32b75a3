"""Recurrences whose state is a matrix S [key channel, value channel] per head with ONE decay a (token, head):
``S <- a S + w k v^T``, ``o = S^T q``.  Three mixers that share the kernels (``kernels.decay_state``):

``matrix_memory``: exponential gates with a running maximum m (zero at admission) and a normaliser.  ``q = W_q x *
q_scale``, ``k = W_k x``, ``v = W_v x``; per head ``i = cap tanh((W_i x + b_i) / cap)``, ``f = logsigmoid(cap tanh((W_f x +
b_f) / cap))``, ``m' = max(f + m, i)``, ``a = exp(f + m - m')``, ``w = exp(i - m')``, n like S with k alone, ``o = S^T q /
(max(|n . q|, exp(-m')) + 1e-6)``.  Each head's o is divided by its root mean square, the heads together are multiplied by a
gain and by ``sigmoid(W_g x)`` and projected by W_o.

``state_space_dual``: ``[z | x | B | C | dt] = W_in h``; x, B and C pass a short causal convolution per channel with a bias
and silu; ``dt = softplus(dt + bias)``, ``a = exp(-exp(A_log) dt)``, ``w = dt``, with B the keys and C the queries of a group of
heads and x the values; ``y = S^T C + D x``, times ``silu(z)``, normed in equal parts of the row, times a gain, W_o.

``constant_decay_attention``: ``q, k, v = silu(W x)``, ``a`` a constant per head, ``w = 1``; the heads together are normed,
multiplied by a gain and by ``sigmoid(W_g x)`` and projected by W_o.

S, n, m and the convolution's last ``taps - 1`` inputs are per-request state, float32, zero at admission.  The projections that
read x are one library product each; its float32 accumulators feed the kernels.  Gates, decays, sums and norms are float32.
In bfloat16 mode portions of many tokens read q, k and v rounded to bfloat16 and run in chunks on the tensor cores; single
tokens, short portions and the float32 mode run token by token.
"""

from __future__ import annotations

import torch

from .. import kernels
from ..matmul import empty_rows, linear
from .base import Mixer, TensorSpec, register


def _fused(fetch, names: list[str], hidden: int) -> torch.Tensor:
    """The named matrices below each other, the rows padded to a multiple of 8 (every product row starts on 16 bytes)."""
    parts = [fetch(n) for n in names]
    rows = sum(p.shape[0] for p in parts)
    w = torch.zeros((-(-rows // 8) * 8, hidden), dtype=parts[0].dtype, device=parts[0].device)
    at = 0
    for p in parts:
        w[at: at + p.shape[0]].copy_(p)
        at += p.shape[0]
    return w


class _DecayState(Mixer):
    """What the three share: sizes, the state, and how the recurrence is run."""

    graph_safe = True
    kind = "decay_state"

    def _sizes(self, hidden_size, n_heads, n_groups, dim, value_dim, norm_eps, names, state_name):
        if n_heads <= 0 or n_groups <= 0 or n_heads % n_groups:
            raise ValueError(f"{self.kind}: {n_heads} heads are not a positive multiple of {n_groups} groups")
        if not 0 < dim <= kernels.DECAY_MAX_DIM or value_dim <= 0:
            raise ValueError(f"{self.kind}: {dim} key channels a head are outside the kernel's 1 to {kernels.DECAY_MAX_DIM}, "
                             f"or no value channels ({value_dim})")
        self.hidden, self.H, self.G, self.D, self.E = int(hidden_size), int(n_heads), int(n_groups), int(dim), int(value_dim)
        self.eps, self.names, self.state_name = float(norm_eps), dict(names), state_name
        self.w_in = self.w_o = self.gain = None

    def state_spec(self):
        return {self.state_name: ((self.H, self.D, self.E), torch.float32)}

    def _chunks(self, T: int, ctx, dtype) -> bool:
        return dtype == torch.bfloat16 and kernels.decay_chunks_take(T, int(ctx.req_slot.numel()), ctx.max_new_tokens_per_req,
                                                                     self.D, self.E)

    def _columns(self, rows):
        """q, k and v out of rows ``[q | k | v | ...]``."""
        a, b = self.G * self.D, 2 * self.G * self.D
        return rows[:, :a], rows[:, a:b], rows[:, b: b + self.H * self.E]

    def _from_projection(self, proj, ctx, dtype, gates, state, silu: bool, **extra):
        """The recurrence over rows ``[q | k | v | ...]`` of a projection's float32 accumulators."""
        T = proj.shape[0]
        rows16 = None
        if self._chunks(T, ctx, dtype):
            n = 2 * self.G * self.D + self.H * self.E
            act = torch.empty((T, n), dtype=dtype, device=proj.device)
            kernels.rows_act(proj[:, :n], act, silu=silu)
            rows16 = self._columns(act)
        o = torch.empty((T, self.H, self.E), dtype=torch.float32, device=proj.device)
        kernels.decay_state(*self._columns(proj), gates, state[self.state_name], o, ctx.req_start, ctx.req_slot, self.H, self.G,
                            self.D, self.E, silu=silu, rows16=rows16, longest=ctx.max_new_tokens_per_req, **extra)
        return o


@register("mixer", "matrix_memory")
class MatrixMemory(_DecayState):
    kind = "matrix_memory"

    def __init__(self, hidden_size: int, n_heads: int, dim: int, value_dim: int, gate_cap: float, norm_eps: float, names: dict,
                 q_scale: float | None = None, state_name: str = "matrix_memory"):
        """``names``: q, k, v, g, i, f, i_b, f_b, norm (all heads' size), o.  ``q_scale`` None: ``dim ** -0.5``."""
        self._sizes(hidden_size, n_heads, n_heads, dim, value_dim, norm_eps, names, state_name)
        if not gate_cap > 0:
            raise ValueError(f"matrix_memory: the gates' cap {gate_cap} must be positive")
        self.cap, self.q_scale = float(gate_cap), float(int(dim) ** -0.5 if q_scale is None else q_scale)
        self.g_off = self.H * (2 * self.D + self.E)
        self.i_off = self.g_off + self.H * self.E
        self.b_i = self.b_f = None

    def tensor_specs(self):
        n, W, HD, HE, H = self.names, self.hidden, self.H * self.D, self.H * self.E, self.H
        return [TensorSpec(n["q"], (HD, W)), TensorSpec(n["k"], (HD, W)), TensorSpec(n["v"], (HE, W)), TensorSpec(n["g"], (HE, W)),
                TensorSpec(n["i"], (H, W)), TensorSpec(n["f"], (H, W)), TensorSpec(n["i_b"], (H,), "f32", "bias"),
                TensorSpec(n["f_b"], (H,), "f32", "bias"), TensorSpec(n["norm"], (HE,), "f32", "gain"), TensorSpec(n["o"], (W, HE))]

    def load(self, fetch):
        n = self.names
        self.w_in = _fused(fetch, [n[k] for k in ("q", "k", "v", "g", "i", "f")], self.hidden)
        self.b_i, self.b_f = fetch(n["i_b"]).contiguous(), fetch(n["f_b"]).contiguous()
        self.gain, self.w_o = fetch(n["norm"]).contiguous(), fetch(n["o"])

    def state_spec(self):
        return {self.state_name: ((self.H, self.D, self.E), torch.float32),
                self.state_name + "_norm": ((self.H, self.D), torch.float32),
                self.state_name + "_max": ((self.H,), torch.float32)}

    def forward(self, x, ctx, cache, state):
        T = x.shape[0]
        proj = linear(x, self.w_in, out_dtype=torch.float32)
        log_decay, weight, floor = kernels.memory_gates(proj, self.i_off, self.i_off + self.H, self.b_i, self.b_f, self.cap,
                                                        state[self.state_name + "_max"], ctx.req_start, ctx.req_slot, self.H)
        den = torch.empty((T, self.H), dtype=torch.float32, device=x.device)
        o = self._from_projection(proj, ctx, x.dtype, kernels.DecayGates.given(log_decay, weight), state, False,
                                  q_scale=self.q_scale, n_state=state[self.state_name + "_norm"], floor=floor, den=den)
        y = empty_rows(T, self.H * self.E, dtype=x.dtype, device=x.device)
        kernels.decay_out(o, proj[:, self.g_off: self.i_off], self.gain, y, self.H, self.E, self.H, self.eps, den=den)
        return linear(y, self.w_o, out_dtype=torch.float32)


@register("mixer", "state_space_dual")
class StateSpaceDual(_DecayState):
    kind = "state_space_dual"

    def __init__(self, hidden_size: int, n_heads: int, n_groups: int, n_state: int, value_dim: int, conv_taps: int,
                 norm_groups: int, norm_eps: float, names: dict, state_name: str = "state_space",
                 conv_state_name: str = "state_space_conv_inputs"):
        """``names``: in, conv, conv_b, dt_bias, A_log, D, norm, o."""
        self._sizes(hidden_size, n_heads, n_groups, n_state, value_dim, norm_eps, names, state_name)
        if conv_taps < 1 or norm_groups < 1 or (n_heads * value_dim) % norm_groups:
            raise ValueError(f"state_space_dual: {conv_taps} taps, or {norm_groups} parts that do not divide {n_heads * value_dim}")
        self.taps, self.parts, self.conv_state_name = int(conv_taps), int(norm_groups), conv_state_name
        self.inner = self.H * self.E
        self.n_conv = self.inner + 2 * self.G * self.D
        self.conv_w = self.conv_b = self.dt_bias = self.A_log = self.skip = None

    def tensor_specs(self):
        n, W, C = self.names, self.hidden, self.n_conv
        return [TensorSpec(n["in"], (self.inner + C + self.H, W)), TensorSpec(n["conv"], (C, self.taps), "f32", "conv"),
                TensorSpec(n["conv_b"], (C,), "f32", "bias"), TensorSpec(n["dt_bias"], (self.H,), "f32", "bias"),
                TensorSpec(n["A_log"], (self.H,), "f32", "gain"), TensorSpec(n["D"], (self.H,), "f32", "gain"),
                TensorSpec(n["norm"], (self.inner,), "f32", "gain"), TensorSpec(n["o"], (W, self.inner))]

    def load(self, fetch):
        n = self.names
        self.w_in = _fused(fetch, [n["in"]], self.hidden)
        self.conv_w, self.conv_b = fetch(n["conv"]).contiguous(), fetch(n["conv_b"]).contiguous()
        self.dt_bias, self.A_log, self.skip = (fetch(n[k]).contiguous() for k in ("dt_bias", "A_log", "D"))
        self.gain, self.w_o = fetch(n["norm"]).contiguous(), fetch(n["o"])

    def state_spec(self):
        spec = super().state_spec()
        if self.taps > 1:
            spec[self.conv_state_name] = ((self.taps - 1, self.n_conv), torch.float32)
        return spec

    def forward(self, x, ctx, cache, state):
        T, I, C, GD = x.shape[0], self.inner, self.n_conv, self.G * self.D
        proj = linear(x, self.w_in, out_dtype=torch.float32)
        u = torch.empty((T, C), dtype=x.dtype, device=x.device)
        hist = state[self.conv_state_name] if self.taps > 1 else torch.empty((0, 0, C), dtype=torch.float32, device=x.device)
        kernels.short_conv(proj[:, I: I + C], self.conv_w, hist, u, ctx.tok_req, ctx.req_start, ctx.req_slot, bias=self.conv_b,
                           silu=True)
        values, keys, queries = u[:, :I], u[:, I: I + GD], u[:, I + GD: I + 2 * GD]
        rows16 = None
        if self._chunks(T, ctx, x.dtype) and all(n % 8 == 0 for n in (C, I, GD)):
            rows16 = (queries, keys, values)
        o = torch.empty((T, self.H, self.E), dtype=torch.float32, device=x.device)
        gates = kernels.DecayGates.step(proj[:, I + C: I + C + self.H], self.dt_bias, self.A_log)
        kernels.decay_state(queries, keys, values, gates, state[self.state_name], o, ctx.req_start, ctx.req_slot, self.H, self.G,
                            self.D, self.E, rows16=rows16, longest=ctx.max_new_tokens_per_req)
        y = empty_rows(T, I, dtype=x.dtype, device=x.device)
        kernels.decay_out(o, proj[:, :I], self.gain, y, self.H, self.E, self.parts, self.eps, x=values, skip=self.skip,
                          gate_first=True)
        return linear(y, self.w_o, out_dtype=torch.float32)


@register("mixer", "constant_decay_attention")
class ConstantDecayAttention(_DecayState):
    kind = "constant_decay_attention"

    def __init__(self, hidden_size: int, n_heads: int, dim: int, value_dim: int, decay, norm_eps: float, names: dict,
                 state_name: str = "constant_decay"):
        """``decay``: one number a head in 0 .. 1; ``names``: q, k, v, g, norm, o."""
        self._sizes(hidden_size, n_heads, n_heads, dim, value_dim, norm_eps, names, state_name)
        self.decay = tuple(float(d) for d in decay)
        if len(self.decay) != self.H or any(not 0.0 <= d <= 1.0 for d in self.decay):
            raise ValueError(f"constant_decay_attention: {len(self.decay)} decays for {self.H} heads, or one outside 0 .. 1")
        self.g_off = self.H * (2 * self.D + self.E)
        self.gates = None

    def tensor_specs(self):
        n, W, HD, HE = self.names, self.hidden, self.H * self.D, self.H * self.E
        return [TensorSpec(n["q"], (HD, W)), TensorSpec(n["k"], (HD, W)), TensorSpec(n["v"], (HE, W)), TensorSpec(n["g"], (HE, W)),
                TensorSpec(n["norm"], (HE,), "f32", "gain"), TensorSpec(n["o"], (W, HE))]

    def load(self, fetch):
        n = self.names
        self.w_in = _fused(fetch, [n[k] for k in ("q", "k", "v", "g")], self.hidden)
        self.gain, self.w_o = fetch(n["norm"]).contiguous(), fetch(n["o"])
        self.gates = kernels.DecayGates.constant(torch.tensor(self.decay, dtype=torch.float32, device=self.gain.device))

    def forward(self, x, ctx, cache, state):
        T = x.shape[0]
        proj = linear(x, self.w_in, out_dtype=torch.float32)
        o = self._from_projection(proj, ctx, x.dtype, self.gates, state, True)
        y = empty_rows(T, self.H * self.E, dtype=x.dtype, device=x.device)
        kernels.decay_out(o, proj[:, self.g_off: self.g_off + self.H * self.E], self.gain, y, self.H, self.E, 1, self.eps)
        return linear(y, self.w_o, out_dtype=torch.float32)
