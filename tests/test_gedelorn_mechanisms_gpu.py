"""Every mechanism of the Gedelorn decoder alone: the framework's kernel or part against the plain function of the same
mechanism (tests/plain/gedelorn_plain.py), for prompts, portions and single tokens, on caches whose pages are shuffled
and partly given back and in state slots that hold other requests' numbers.  Where random numbers would hide a fault the
inputs are made so that it shows: one key whose score outweighs all others just inside or just outside a window, one
pair written hundreds of tokens ago into a head that hardly decays, steps that wipe a state out, a running maximum that
is taken over late."""

import math

import pytest
import torch

from tests.plain import gedelorn_plain as P

DEV = "cuda:0"
pytestmark = pytest.mark.gpu


def _close(got, want, tol, what=""):
    scale = float(want.abs().max()) or 1.0
    err = float((got.double().cpu() - want.double().cpu()).abs().max()) / scale
    assert err < tol, (what, err)


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def _steps(lens, cuts):
    """Portions of several requests side by side: per step, (request, first position, tokens) of those that go on."""
    at = [0] * len(lens)
    for turn in range(max(len(c) for c in cuts)):
        step = []
        for r, c in enumerate(cuts):
            if turn < len(c):
                step.append((r, at[r], c[turn]))
                at[r] += c[turn]
        yield step
    assert at == list(lens)


def _starts(step):
    starts = [0]
    for _, _, n in step:
        starts.append(starts[-1] + n)
    return starts


# ---- the recurrence -------------------------------------------------------------------------------------------
def _constants(H):
    """Decays, step biases and rates of H heads, the same for every request."""
    g = torch.Generator().manual_seed(H)
    decay = torch.tensor(([0.0, 1.0, 0.999, 0.6, 0.2, 0.97] + [0.9] * H)[:H])
    return decay, torch.randn(H, generator=g), torch.randn(H, generator=g)


def _gate_inputs(n, H, kind, g):
    """(columns a token that the gates are made from, plain decay, plain weight), all ``[n, H]``."""
    decay, bias, A_log = _constants(H)
    if kind == "constant":
        return [], decay.double().expand(n, H), torch.ones(n, H, dtype=torch.float64)
    if kind == "step":
        pre = torch.randn(n, H, generator=g) * 2
        pre[n // 2] = 40.0                      # a step far in softplus's linear range: the state is wiped out
        dt = torch.nn.functional.softplus(pre.double() + bias.double())
        return [pre], torch.exp(-torch.exp(A_log.double()) * dt), dt
    la, w = -torch.rand(n, H, generator=g) ** 4 * 6, torch.rand(n, H, generator=g)
    return [la, w], torch.exp(la.double()), w.double()


def _gates(kind, H, columns):
    from quanta_b200 import kernels
    decay, bias, A_log = (t.to(DEV) for t in _constants(H))
    if kind == "constant":
        return kernels.DecayGates.constant(decay)
    if kind == "step":
        wide = torch.full((columns[0].shape[0], H + 3), 5.0)                   # columns of wider rows
        wide[:, 2: 2 + H] = columns[0]
        return kernels.DecayGates.step(wide.to(DEV)[:, 2: 2 + H], bias, A_log)
    return kernels.DecayGates.given(*(c.contiguous().to(DEV) for c in columns))


def _plain_recurrence(q, k, v, a, w, H, G, D, E):
    """(o [n, H, E], n . q [n, H], S, n) in float64."""
    n = q.shape[0]
    group = torch.arange(H) // (H // G)
    q, k = q.double().view(n, G, D)[:, group], k.double().view(n, G, D)[:, group]
    v = torch.cat([v.double().view(n, H, E), torch.ones(n, H, 1, dtype=torch.float64)], -1)     # the normaliser: values of one
    o, S = P.decayed_rows(q, k, v, a, w)
    return o[..., :E], o[..., E], S[..., :E], S[..., E]


SHAPES = [(4, 2, 12, 20), (3, 3, 16, 8), (2, 1, 40, 24), (4, 4, 64, 64), (6, 2, 128, 64), (1, 1, 256, 96), (2, 2, 24, 6),
          (8, 1, 8, 48), (5, 5, 33, 13), (2, 2, 96, 40), (3, 1, 200, 16), (2, 1, 16, 136)]


@pytest.mark.parametrize("kind", ["constant", "step", "given"])
@pytest.mark.parametrize("H,G,D,E", SHAPES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_recurrence_in_portions(H, G, D, E, kind, dtype):
    """Two requests side by side in portions that begin and end anywhere in a chunk, single tokens beside long portions;
    in bfloat16, with sizes that allow it, portions run in chunks on the tensor cores."""
    from quanta_b200 import kernels
    lens, cuts = [161, 90], [[1, 64, 2, 17, 15, 1, 61], [35, 1, 2, 51, 1]]
    rows, columns, want = [], [], []
    for r, n in enumerate(lens):
        g = torch.Generator().manual_seed(10 * r + D)
        qkv = torch.randn(n, 2 * G * D + H * E, generator=g).to(dtype)
        cols, a, w = _gate_inputs(n, H, kind, g)
        rows.append(qkv)
        columns.append(cols)
        want.append(_plain_recurrence(qkv[:, : G * D], qkv[:, G * D: 2 * G * D], qkv[:, 2 * G * D:], a, w, H, G, D, E))
    norms = kind == "given"
    slots = [2, 0]
    state, n_state = torch.full((4, H, D, E), 3.0, device=DEV), torch.full((4, H, D), 3.0, device=DEV)
    state[slots] = 0.0
    n_state[slots] = 0.0
    chunked = dtype == torch.bfloat16 and D % 8 == 0 and E % 8 == 0
    tol = 5e-5 if chunked else 1e-5
    for step in _steps(lens, cuts):
        starts = _starts(step)
        T = starts[-1]
        x = torch.cat([rows[r][p: p + n] for r, p, n in step]).contiguous().to(DEV)
        gates = _gates(kind, H, [torch.cat([columns[r][c][p: p + n] for r, p, n in step]) for c in range(len(columns[0]))])
        qkv = x[:, : G * D], x[:, G * D: 2 * G * D], x[:, 2 * G * D:]
        o = torch.full((T, H, E), float("nan"), device=DEV)
        den = torch.full((T, H), float("nan"), device=DEV)
        extra = dict(n_state=n_state, floor=torch.full((T, H), 0.25, device=DEV), den=den) if norms else {}
        kernels.decay_state(*qkv, gates, state, o, _i32(starts), _i32([slots[r] for r, _, _ in step]), H, G, D, E, q_scale=0.7,
                            rows16=qkv if chunked and T > len(step) else None, **extra)
        for i, (r, p, n) in enumerate(step):
            _close(o[starts[i]: starts[i + 1]], 0.7 * want[r][0][p: p + n], tol, f"request {r}, tokens {p}:{p + n}")
            if norms:
                _close(den[starts[i]: starts[i + 1]], torch.clamp_min((0.7 * want[r][1][p: p + n]).abs(), 0.25) + 1e-6, tol,
                       f"normaliser of {r}, tokens {p}:{p + n}")
    for r in range(2):
        _close(state[slots[r]], want[r][2], tol, f"state of {r}")
        if norms:
            _close(n_state[slots[r]], want[r][3], tol, f"normaliser state of {r}")
    assert float(state[[1, 3]].min()) == 3.0 == float(state[[1, 3]].max())


@pytest.mark.parametrize("H,G,D,E,kind", [(2, 1, 32, 48, "step"), (4, 4, 64, 64, "constant"), (3, 3, 128, 72, "given"), (1, 1, 192, 40, "given")])
def test_long_prompts_run_as_segments(H, G, D, E, kind):
    """A step whose heads do not fill the GPU: segments of several chunks in three passes, beside one pass and beside a
    request of a few tokens; the state goes on from where an earlier portion left it."""
    from quanta_b200 import kernels
    lens = [1500, 9]
    data = []
    for r, n in enumerate(lens):
        g = torch.Generator().manual_seed(r)
        qkv = torch.randn(n, 2 * G * D + H * E, generator=g).to(torch.bfloat16)
        cols, a, w = _gate_inputs(n, H, kind, g)
        data.append((qkv, cols, _plain_recurrence(qkv[:, : G * D], qkv[:, G * D: 2 * G * D], qkv[:, 2 * G * D:], a, w, H, G, D, E)))
    norms = kind == "given"
    for segments in (None, False):
        state, n_state = torch.zeros(3, H, D, E, device=DEV), torch.zeros(3, H, D, device=DEV)
        for step in ([(0, 0, 70)], [(0, 70, 1430), (1, 0, 9)]):
            starts = _starts(step)
            T = starts[-1]
            x = torch.cat([data[r][0][p: p + n] for r, p, n in step]).to(DEV)
            gates = _gates(kind, H, [torch.cat([data[r][1][c][p: p + n] for r, p, n in step]) for c in range(len(data[0][1]))])
            qkv = x[:, : G * D], x[:, G * D: 2 * G * D], x[:, 2 * G * D:]
            o, den = torch.full((T, H, E), float("nan"), device=DEV), torch.full((T, H), float("nan"), device=DEV)
            extra = dict(n_state=n_state, floor=torch.full((T, H), 0.25, device=DEV), den=den) if norms else {}
            before = kernels.LAUNCHES
            kernels.decay_state(*qkv, gates, state, o, _i32(starts), _i32([r + 1 for r, _, _ in step]), H, G, D, E, rows16=qkv,
                                segments=segments, **extra)
            if T > 1000:
                assert kernels.LAUNCHES - before == (5 if segments is None else 2)
            for i, (r, p, n) in enumerate(step):
                _close(o[starts[i]: starts[i + 1]], data[r][2][0][p: p + n], 5e-5, f"{segments} request {r}, tokens {p}:{p + n}")
                if norms:
                    _close(den[starts[i]: starts[i + 1]], torch.clamp_min(data[r][2][1][p: p + n].abs(), 0.25) + 1e-6, 5e-5, "normaliser")
        for r in range(2):
            _close(state[r + 1], data[r][2][2], 5e-5, f"state of {r}")
            if norms:
                _close(n_state[r + 1], data[r][2][3], 5e-5, f"normaliser state of {r}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("at", [0, 63, 64, 300])
def test_a_pair_written_long_ago(dtype, at):
    """One key and value among hundreds of zeros, asked for by the last query, in heads that keep everything, decay slowly
    or fast: what comes back is ``decay^distance``; decoded alone and as part of the prompt."""
    from quanta_b200 import kernels
    n, D, E = 640, 16, 32
    decay = torch.tensor([1.0, 0.999, 0.98, 0.5, 0.0])
    H = decay.numel()
    g = torch.Generator().manual_seed(at)
    row = torch.zeros(n, 2 * H * D + H * E)
    row[at, H * D: 2 * H * D] = torch.eye(D)[3].repeat(H)
    row[at, 2 * H * D:] = torch.randn(H * E, generator=g)
    row[n - 1, : H * D] = torch.eye(D)[3].repeat(H)
    x = row.to(dtype).to(DEV)
    want = x[at, 2 * H * D:].view(H, E).double().cpu() * (decay.double() ** (n - 1 - at))[:, None]
    gates = kernels.DecayGates.constant(decay.to(DEV))
    for cuts in ([n], [n - 1, 1], [at + 1, 2, n - at - 4, 1]):
        state = torch.zeros(1, H, D, E, device=DEV)
        p = 0
        for m in cuts:
            part = x[p: p + m]
            qkv = part[:, : H * D], part[:, H * D: 2 * H * D], part[:, 2 * H * D:]
            o = torch.empty((m, H, E), device=DEV)
            kernels.decay_state(*qkv, gates, state, o, _i32([0, m]), _i32([0]), H, H, D, E,
                                rows16=qkv if dtype == torch.bfloat16 and m > 1 else None)
            p += m
        got = o[-1].double().cpu()
        for h in range(H):
            assert torch.allclose(got[h], want[h], atol=1e-7, rtol=6e-5), (cuts, h, got[h] / want[h])


# ---- exponential gates ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,cap", [(3, 15.0), (1, 2.0), (40, 4.0)])
def test_running_maximum(H, cap):
    """Input gates that take the maximum over now and then, forget gates near one and near zero; a prompt longer than a
    block's turn, then portions and single tokens of two requests."""
    from quanta_b200 import kernels
    lens, cuts = [2500, 60], [[2300, 1, 2, 190, 7], [3, 1, 40, 15, 1]]
    g = torch.Generator().manual_seed(H)
    b_i, b_f = torch.randn(H, generator=g), torch.randn(H, generator=g) + 1
    rows, want = [], []
    for n in lens:
        x = torch.randn(n, 2 * H + 5, generator=g) * 3
        x[:, 1: 1 + H] -= 2
        x[n // 3, 1: 1 + H] = 30.0
        i = cap * torch.tanh((x[:, 1: 1 + H].double() + b_i.double()) / cap)
        f = torch.nn.functional.logsigmoid(cap * torch.tanh((x[:, 3 + H: 3 + 2 * H].double() + b_f.double()) / cap))
        m, la, w, floor = torch.zeros(H, dtype=torch.float64), [], [], []
        for t in range(n):
            top = torch.maximum(f[t] + m, i[t])
            la.append(f[t] + m - top)
            w.append(torch.exp(i[t] - top))
            floor.append(torch.exp(-top))
            m = top
        rows.append(x)
        want.append((torch.stack(la), torch.stack(w), torch.stack(floor), m))
    m_state = torch.full((3, H), 9.0, device=DEV)
    m_state[[1, 2]] = 0.0
    for step in _steps(lens, cuts):
        starts = _starts(step)
        x = torch.cat([rows[r][p: p + n] for r, p, n in step]).to(DEV)
        got = kernels.memory_gates(x, 1, 3 + H, b_i.to(DEV), b_f.to(DEV), cap, m_state, _i32(starts), _i32([r + 1 for r, _, _ in step]), H)
        for i, (r, p, n) in enumerate(step):
            for j, what in enumerate(("log decay", "weight", "floor")):
                err = (got[j][starts[i]: starts[i + 1]].double().cpu() - want[r][j][p: p + n]).abs()
                assert float((err / (1 + want[r][j][p: p + n].abs())).max()) < 1e-5, (what, r, p)
    for r in range(2):
        assert torch.allclose(m_state[r + 1].double().cpu(), want[r][3], atol=1e-5)
    assert float(m_state[0].min()) == 9.0


# ---- from the recurrence to the output projection ----------------------------------------------------------------
@pytest.mark.parametrize("H,E,parts", [(4, 12, 4), (3, 10, 1), (2, 96, 2), (6, 20, 3), (8, 128, 1), (5, 7, 5), (16, 64, 2), (2, 300, 4), (32, 128, 1), (8, 640, 2), (4, 2500, 1), (40, 128, 2)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norm_in_parts_and_gate(H, E, parts, dtype):
    from quanta_b200 import kernels
    g = torch.Generator().manual_seed(H * E)
    T, C, eps = 5, H * E, 1e-2
    o = torch.randn(T, H, E, generator=g)
    proj = torch.randn(T, C + 8, generator=g) * 2
    gate, gain = proj[:, 4: 4 + C], torch.randn(C, generator=g)
    wide = torch.randn(T, C + 8, generator=g).to(dtype)
    x, skip, den = wide[:, :C], torch.randn(H, generator=g), torch.rand(T, H, generator=g) + 0.1

    def run(**kw):
        out = torch.empty((T, C), dtype=dtype, device=DEV)
        kernels.decay_out(o.to(DEV), proj.to(DEV)[:, 4: 4 + C], gain.to(DEV), out, H, E, parts, eps, **kw)
        return out

    def normed(y):
        return P.rms(y.view(T, parts, C // parts), eps).reshape(T, C) * gain

    tol = 3e-6 if dtype == torch.float32 else 6e-3
    _close(run(), normed(o.reshape(T, C)) * torch.sigmoid(gate), tol, "norm, then gate")
    _close(run(den=den.to(DEV)), normed((o / den[..., None]).reshape(T, C)) * torch.sigmoid(gate), tol, "denominator")
    y = (o + skip[:, None] * x.float().view(T, H, E)).reshape(T, C) * torch.nn.functional.silu(gate)
    _close(run(x=wide.to(DEV)[:, :C], skip=skip.to(DEV), gate_first=True), normed(y), tol, "skip, gate, then norm")


# ---- windowed attention with capped scores whose values are its keys -----------------------------------------------
class Pages:
    """Keys and values of one sequence in shuffled pages, stale numbers everywhere else; ``forget(before)`` gives the pages
    back that hold only positions below ``before``."""

    def __init__(self, k, v, page, dtype, seed):
        from quanta_b200 import kernels
        n, G, hd = k.shape
        count = -(-n // page)
        order = torch.randperm(count + 3, generator=torch.Generator().manual_seed(seed)).tolist()
        self.page = page
        self.k = torch.full((count + 3, G, page, hd), 37.0, dtype=dtype, device=DEV)
        self.v = torch.full((count + 3, G, page, v.shape[2]), -43.0, dtype=dtype, device=DEV)
        for p in range(n):
            self.k[order[p // page], :, p % page] = k[p].to(dtype).to(DEV)
            self.v[order[p // page], :, p % page] = v[p].to(dtype).to(DEV)
        self.table = _i32([order[:count]])
        self.status = kernels.new_status(DEV)

    def forget(self, before):
        self.table[0, : before // self.page] = -1

    def attend(self, q, p0, p1, scale, window, cap, **opts):
        from quanta_b200 import kernels
        rows = q[p0:p1].contiguous().to(DEV)
        out = torch.empty((p1 - p0, q.shape[1], self.v.shape[3]), dtype=q.dtype, device=DEV)
        kernels.window_attention(rows, self.k, self.v, out, _i32(list(range(p0, p1))), _i32([0] * (p1 - p0)), self.table, scale,
                                 window, self.status, softcap=cap, n_requests=1, **opts)
        assert int(self.status[0]) == 0
        return out.float().cpu()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window,page,hd,back", [(40, 16, 32, 0), (40, 16, 32, 1), (64, 16, 48, 0), (64, 16, 48, 1), (17, 4, 20, 0),
                                                 (17, 4, 20, 1), (128, 8, 64, 0), (128, 8, 64, 1), (1, 4, 16, 1)])
def test_a_key_at_the_edge_of_a_window(window, page, hd, back, dtype):
    """A key that outweighs all others although scores are capped: the last query that sees it (``back`` 0) and the first
    that does not (``back`` 1), in a prompt, in a portion of two tokens and decoded alone."""
    nq, G, n, cap, scale = 4, 2, 300, 9.0, 1.0
    g = torch.Generator().manual_seed(window + back)
    k, q, v = (torch.randn(n, h, hd, generator=g) * 0.1 for h in (G, nq, G))
    far = 131
    query = far + window - 1 + back
    k[far] = 0.0
    k[far, :, 3] = 20.0
    q[query] = 0.0
    q[query, :, 3] = 20.0
    q, k, v = (t.to(dtype) for t in (q, k, v))
    want = P.capped_attend(q.float(), k.float(), v.float(), scale, cap, P.window_mask(n, window))
    weight = math.exp(9.0) / (math.exp(9.0) + window - 1)
    seen = float((want[query, 0] - weight * v.float()[far, 0]).abs().max())
    assert (seen < 0.05) == (back == 0), "the case itself"
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    pages = Pages(k, v, page, dtype, seed=1)
    _close(pages.attend(q, 0, n, scale, window, cap), want, tol, "prompt")
    pages.forget(max(0, query - window + 1))
    _close(pages.attend(q, query, query + 2, scale, window, cap), want[query: query + 2], tol, "portion")
    for split in (1, 3, None):
        _close(pages.attend(q, query, query + 1, scale, window, cap, n_split=split), want[query: query + 1], tol, f"alone, {split}")


# ---- the mixers ---------------------------------------------------------------------------------------------------
def _part(raw_layer, seed, width=40, dtype=torch.float32, eps=1e-4):
    """(part, its weights as float32, page streams it wants) of one layer of a configuration."""
    from quanta_b200 import matmul
    from quanta_b200.config import GedelornConfig
    from quanta_b200.models.gedelorn import mixer
    from quanta_b200.parts.base import make
    matmul.configure()
    cfg = {"architecture": "Gedelorn", "vocab": 9, "width": width, "norm": {"eps": eps}, "layers": [dict(raw_layer, mlp=None)]}
    w = {k: v.float() for k, v in P.draw_weights(cfg, seed).items()}
    part = make("mixer", mixer(GedelornConfig.from_dict(cfg), 0))

    def load(p):
        kinds = {s.name: s.kind for s in p.tensor_specs()}
        p.load(lambda n: w[n].to(DEV, torch.float32 if kinds[n] == "f32" else dtype))
        for c in p.children():
            load(c)

    load(part)
    return part, w


MLSTM = [dict(heads=2, dim=12, vdim=20, gate_cap=3.0), dict(heads=3, dim=16, vdim=8, gate_cap=15.0), dict(heads=1, dim=64, vdim=72, gate_cap=1.0)]
MAMBA = [dict(heads=4, vdim=12, state=10, groups=2, conv=4, norm_groups=3), dict(heads=6, vdim=16, state=24, groups=1, conv=1, norm_groups=1),
         dict(heads=4, vdim=64, state=128, groups=4, conv=2, norm_groups=4), dict(heads=2, vdim=40, state=16, groups=2, conv=5, norm_groups=2)]
PARALLEL = [
    dict(left=dict(heads=4, kv_heads=2, dim=12, vdim=12, scale=0.4, softcap=3.0, mask=dict(size=7), rot=dict(dims=8, base=50.0)), left_scale=0.7,
         right=dict(heads=3, dim=10, vdim=14, decay=[0.9, 0.999, 0.3]), right_scale=1.4),
    dict(left=dict(heads=2, kv_heads=2, dim=16, vdim=16, scale=0.2, softcap=1.5, mask=dict(size=33), rot=dict(dims=16, base=1e4)), left_scale=1.1,
         right=dict(heads=2, dim=16, vdim=24, decay=[1.0, 0.95]), right_scale=0.6)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layer", [dict(type="mlstm", mixer=m) for m in MLSTM] + [dict(type="mamba2", mixer=m) for m in MAMBA] +
                         [dict(type="parallel", mixer=m) for m in PARALLEL])
def test_mixer_in_portions_against_the_plain_mixer(layer, dtype):
    """Projections, convolution and its state, gates, recurrence, attention over pages, norms: two requests in portions
    down to two tokens and single tokens, slots that were used before."""
    from quanta_b200 import kernels
    from quanta_b200.parts.base import Addends, LayerCache, StepContext
    width, eps, page = 40, 1e-4, 4
    part, w = _part(layer, 3, width, dtype, eps)
    lens, cuts = [100, 41], [[7, 2, 1, 1, 66, 2, 20, 1], [1, 2, 1, 30, 1, 5, 1]]
    xs = [torch.randn(n, width, generator=torch.Generator().manual_seed(n)).to(dtype) for n in lens]
    plain = {"mlstm": lambda x: P.matrix_memory(w, "l0.mix.", x, layer["mixer"], eps),
             "mamba2": lambda x: P.state_space(w, "l0.mix.", x, layer["mixer"], eps),
             "parallel": lambda x: P.side_by_side(w, "l0.mix.", x, layer["mixer"], eps)}[layer["type"]]
    want = [plain(x.float()) for x in xs]
    state = {n: torch.full((3, *shape), 2.0, dtype=dt, device=DEV) for n, (shape, dt) in part.state_spec().items()}
    for t in state.values():
        t[1:] = 0.0
    spec = part.cache_spec()
    streams = {} if spec is None else {s.name: torch.full((40, s.heads, page, s.width), 30.0, dtype=dtype, device=DEV) for s in spec.streams}
    table = torch.stack([torch.arange(25), torch.arange(25) + 15]).flip(1).to(torch.int32)     # 25 and 11 pages used
    table[1, 11:] = -1
    table[1, :11] = torch.arange(25, 36, dtype=torch.int32)
    status = kernels.new_status(DEV)
    for step in _steps(lens, cuts):
        starts = _starts(step)
        T = starts[-1]
        pos = _i32([p + i for _, p, n in step for i in range(n)])
        ctx = StepContext(n_tokens=T, positions=pos.view(T, 1), tok_pos=pos, tok_req=_i32([i for i, (_, _, n) in enumerate(step) for _ in range(n)]),
                          req_slot=_i32([r + 1 for r, _, _ in step]), req_start=_i32(starts), req_len_after=_i32([p + n for _, p, n in step]),
                          status=status, dtype=dtype, max_new_tokens_per_req=max(n for _, _, n in step),
                          max_len_after=max(p + n for _, p, n in step))
        cache = None if spec is None else LayerCache(streams=streams, page_size=page, block_table=table[[r for r, _, _ in step]].contiguous().to(DEV))
        x = torch.cat([xs[r][p: p + n] for r, p, n in step]).to(DEV)
        got = part.forward(x, ctx, cache, state)
        got = got.total() if isinstance(got, Addends) else got
        kernels.raise_on_status(status.cpu())
        for i, (r, p, n) in enumerate(step):
            # a norm over a state of one or two tokens may divide by little: the plain scale of the whole request counts
            err = float((got[starts[i]: starts[i + 1]].cpu() - want[r][p: p + n]).abs().max() / want[r].abs().max())
            assert err < (3e-5 if dtype == torch.float32 else 4e-2), (f"request {r}, tokens {p}:{p + n}", err)
    for t in state.values():
        assert float(t[0].min()) == 2.0 == float(t[0].max())


# ---- feed-forward, norms ---------------------------------------------------------------------------------------------
class _Ctx:
    def __init__(self):
        from quanta_b200 import kernels
        self.status = kernels.new_status(DEV)


@pytest.mark.parametrize("T,W,E,top,ff,shared,scale,dtype", [
    (9, 40, 5, 2, 24, 16, 1.7, torch.float32), (150, 64, 8, 1, 64, 128, 0.6, torch.bfloat16), (5, 48, 5, 1, 24, 16, 2.5, torch.float32),
    (1, 64, 4, 4, 16, None, 1.0, torch.bfloat16), (3, 24, 3, 3, 8, None, 0.4, torch.float32), (40, 128, 6, 3, 32, 40, 3.0, torch.bfloat16)])
def test_sigmoid_routed_ungated_experts(T, W, E, top, ff, shared, scale, dtype):
    """Choice, shares of the sum (one chosen expert has the whole share), the scale, the squared relu, the shared expert."""
    from quanta_b200 import matmul
    from quanta_b200.parts.base import make
    matmul.configure()
    g = torch.Generator().manual_seed(T + W)
    mlp = {"router": {"experts": E, "top": top, "scale": scale}, "expert": {"ff": ff}, "shared": None if shared is None else {"ff": shared}}
    w = {"router": torch.randn(E, W, generator=g) * 3 / math.sqrt(W)}
    for e in list(range(E)) + ([] if shared is None else ["shared"]):
        name, inner = (f"e{e}", ff) if isinstance(e, int) else (e, shared)
        w.update({name + ".up": torch.randn(inner, W, generator=g) * 2 / math.sqrt(W), name + ".down": torch.randn(W, inner, generator=g) / math.sqrt(inner)})
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    part = make("feed_forward", ("sigmoid_ungated_experts", dict(
        hidden_size=W, expert_size=ff, n_experts=E, top_k=top, scaling=scale, shared_size=shared or 0,
        names={"gate": "router", "up": "e{e}.up", "down": "e{e}.down", "shared_up": "shared.up", "shared_down": "shared.down"})))
    for p in [part, *part.children()]:
        kinds = {s.name: s.kind for s in p.tensor_specs()}
        p.load(lambda n: w[n].to(DEV, torch.float32 if kinds[n] == "f32" else dtype))
    x = torch.randn(T, W, generator=g).to(dtype)
    want, idx, margin = P.routed_ff(w, "", x.float(), mlp)
    clear = margin > (1e-5 if dtype == torch.float32 else 2e-2)
    part.trace = []
    got = part.forward(x.to(DEV), _Ctx()).total().cpu()
    assert bool((part.trace[0].cpu()[clear] == idx[clear]).all())
    part.trace = None                          # without a trace the small steps take one launch for routing and plan
    assert torch.equal(part.forward(x.to(DEV), _Ctx()).total().cpu(), got)
    _close(got[clear], want[clear], 3e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("W", [36, 64, 256])
def test_norms_stored_around_zero(W):
    """``h += (1 + w) rms(y)`` and the next norm in one launch, from gains that are stored minus one."""
    from quanta_b200.parts.base import NormedPending, make
    g = torch.Generator().manual_seed(W)
    h, y, a, b = torch.randn(7, W, generator=g) * 3, torch.randn(7, W, generator=g), torch.randn(W, generator=g), torch.randn(W, generator=g)
    after, before = (make("norm", ("rms_norm", dict(width=W, eps=1e-2, weight_name=n, around_zero=True))) for n in "ab")
    for part, t in ((after, a), (before, b)):
        part.load(lambda n: t.to(DEV))
    want_h = h + P.around_zero_norm(y, a, 1e-2)
    stream, out = h.to(DEV), torch.empty(7, W, device=DEV)
    before.forward(stream, NormedPending(y.to(DEV), after), out)
    _close(stream, want_h, 1e-6)
    _close(out, P.around_zero_norm(want_h, b, 1e-2), 2e-6)
