"""Every mechanism of the Lotilix decoder alone: the framework's kernel or part against the plain function of the same
mechanism (tests/plain/lotilix_plain.py), for prompts, portions and single tokens, on caches whose pages are shuffled
and partly given back and in state slots that were used before.  Where random numbers would hide a fault the inputs are
made so that it shows: one key whose score outweighs all others sits just inside or just outside a window's or a
chunk's edge, at a page's first and last place, at position 0 and far back among hundreds."""

import math

import pytest
import torch

from tests.plain import lotilix_plain as P

DEV = "cuda:0"
pytestmark = pytest.mark.gpu


def _close(got, want, tol, what=""):
    scale = float(want.abs().max()) or 1.0
    err = float((got.float().cpu() - want.float().cpu()).abs().max()) / scale
    assert err < tol, (what, err)


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


class Pages:
    """Pages of one or two streams in a shuffled order, stale numbers everywhere; ``forget(r, before)`` gives the pages
    back that hold only positions below ``before`` (their table entries become -1)."""

    def __init__(self, lengths, widths, heads, page, dtype, seed=0):
        from quanta_b200 import kernels
        per = [-(-n // page) for n in lengths]
        total = sum(per) + 3
        order = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
        self.page = page
        self.streams = [torch.full((total, heads, page, w), 37.0 - 80 * i, dtype=dtype, device=DEV) for i, w in enumerate(widths)]
        self.table = torch.full((len(lengths), max(per)), -1, dtype=torch.int32)
        for r in range(len(lengths)):
            for p in range(per[r]):
                self.table[r, p] = order.pop()
        self.dev_table = self.table.to(DEV)
        self.status = kernels.new_status(DEV)

    def forget(self, r, before):
        self.dev_table[r, : before // self.page] = -1


# ---- rotation, values that are the keys, cache write ---------------------------------------------------------
@pytest.mark.parametrize("nq,G,hd,dims,page,dtype", [
    (4, 2, 12, 8, 4, torch.float32), (6, 2, 16, 16, 8, torch.bfloat16), (5, 5, 10, 6, 3, torch.float32),
    (3, 1, 64, 32, 16, torch.bfloat16), (2, 2, 18, 18, 4, torch.bfloat16), (2, 1, 24, 0, 4, torch.float32)])
def test_neighbours_are_rotated_and_values_are_unrotated_keys(nq, G, hd, dims, page, dtype):
    from quanta_b200 import kernels
    g = torch.Generator().manual_seed(hd)
    n = 29
    qk = torch.randn(n, (nq + G) * hd + 3, generator=g)                      # rows wider than what counts
    rot = {"dims": dims, "base": 40.0}
    pos = torch.arange(n) + 5
    q0, k0 = qk[:, : nq * hd].view(n, nq, hd), qk[:, nq * hd: (nq + G) * hd].reshape(n, G, hd)
    want_q = P.rotate_neighbours(q0, pos, rot) if dims else q0
    want_k = P.rotate_neighbours(k0, pos, rot) if dims else k0
    cache = Pages([n + 5], [hd, hd], G, page, dtype, seed=1)
    q = torch.empty((n, nq, hd), dtype=dtype, device=DEV)
    freqs = torch.tensor(P.frequencies(rot), dtype=torch.float32, device=DEV)
    p32 = pos.to(DEV, torch.int32)
    kernels.qknorm_rope_write(qk.to(DEV), q, *cache.streams, None, None, kernels.NORM_NONE, 0.0, freqs, None, p32.view(n, 1),
                              p32, torch.zeros_like(p32), cache.dev_table, nq, G, hd, dims, page, cache.status,
                              interleaved=True, tied_values=True)
    assert int(cache.status[0]) == 0
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    _close(q, want_q, tol, "queries")
    for t in range(n):
        at = int(cache.table[0, int(pos[t]) // page]), slice(None), int(pos[t]) % page
        _close(cache.streams[0][at], want_k[t], tol, f"key {t}")
        _close(cache.streams[1][at], k0[t], 1e-9 if dtype == torch.float32 else 8e-3, f"value {t}")


# ---- attention inside chunks -------------------------------------------------------------------------------------
def _chunk_case(n, nq, G, hd, page, dtype, seed, q=None, k=None):
    g = torch.Generator().manual_seed(seed)
    q = torch.randn(n, nq, hd, generator=g) if q is None else q
    k = torch.randn(n, G, hd, generator=g) if k is None else k
    v = torch.randn(n, G, hd, generator=g)
    q, k, v = (t.to(dtype) for t in (q, k, v))
    cache = Pages([n], [hd, hd], G, page, dtype, seed=seed)
    for p in range(n):
        at = int(cache.table[0, p // page]), slice(None), p % page
        cache.streams[0][at], cache.streams[1][at] = k[p].to(DEV), v[p].to(DEV)
    return q, k, v, cache


def _attend_chunk(cache, q, p0, p1, scale, chunk, **opts):
    from quanta_b200 import kernels
    rows = q[p0:p1].contiguous().to(DEV)
    out = torch.empty_like(rows)
    kernels.window_attention(rows, *cache.streams, out, _i32(list(range(p0, p1))), _i32([0] * (p1 - p0)), cache.dev_table,
                             scale, 0, cache.status, chunk=chunk, **opts)
    assert int(cache.status[0]) == 0
    return out.float().cpu()


@pytest.mark.parametrize("nq,G,hd,page,chunk,dtype", [
    (4, 2, 12, 4, 10, torch.float32), (4, 2, 32, 16, 48, torch.bfloat16), (6, 3, 16, 8, 8, torch.float32),
    (2, 2, 64, 16, 100, torch.bfloat16), (3, 1, 10, 5, 1, torch.float32), (8, 1, 48, 16, 33, torch.bfloat16),
    (2, 1, 128, 16, 64, torch.bfloat16), (5, 5, 20, 4, 7, torch.bfloat16), (4, 2, 16, 8, 500, torch.float32)])
def test_chunk_attention_of_prompts_portions_and_single_tokens(nq, G, hd, page, chunk, dtype):
    n, scale = 170, 0.31
    q, k, v, cache = _chunk_case(n, nq, G, hd, page, dtype, seed=hd)
    want = P.attend(q.float(), k.float(), v.float(), scale, P.chunk_mask(n, chunk))
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    _close(_attend_chunk(cache, q, 0, n, scale, chunk, n_requests=1), want, tol, "prompt")
    if dtype == torch.float32:
        _close(_attend_chunk(cache, q, 0, n, scale, chunk, n_split=1), want, tol, "prompt, one range")
    # portions cut anywhere, the pages of finished chunks given back first; then single tokens, in ranges
    for p0, p1 in ((60, 62), (62, 99), (99, 100), (100, 150)):
        cache.forget(0, p0 // chunk * chunk)
        _close(_attend_chunk(cache, q, p0, p1, scale, chunk, n_requests=1), want[p0:p1], tol, f"portion {p0}:{p1}")
    for p, split in ((150, 1), (151, 2), (152, 7), (153, 64), (160, 5)):
        cache.forget(0, p // chunk * chunk)
        _close(_attend_chunk(cache, q, p, p + 1, scale, chunk, n_split=split), want[p:p + 1], tol, f"token {p}, {split} ranges")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("chunk,back", [(48, 0), (48, 1), (50, 0), (50, 1), (64, 0), (64, 1), (200, 0), (200, 1), (16, 1)])
def test_a_key_at_the_edge_of_a_chunk(chunk, back, dtype):
    """A key that stands out at a chunk's first place (``back`` 0: every later token of the chunk sees it) and at the
    last place of the chunk before (``back`` 1: no token of the chunk does)."""
    n, nq, G, hd, page = 420, 4, 2, 32, 16
    first = 2 * chunk
    g = torch.Generator().manual_seed(chunk + back)
    k = torch.randn(n, G, hd, generator=g) * 0.1
    q = torch.randn(n, nq, hd, generator=g) * 0.1
    k[first - back] = 0.0
    k[first - back, :, 3] = 6.0
    for p in range(first, n):
        q[p] = 0.0
        q[p, :, 3] = 6.0
    qb, kb, v, cache = _chunk_case(n, nq, G, hd, page, dtype, seed=back, q=q, k=k)
    want = P.attend(qb.float(), kb.float(), v.float(), 1.0, P.chunk_mask(n, chunk))
    own = v.float()[first - back].repeat_interleave(nq // G, 0)
    stands_out = float((want[min(n, first + chunk) - 1] - own).abs().max()) < 1e-3
    assert stands_out == (back == 0)
    tol = 1e-4 if dtype == torch.float32 else 2e-2
    _close(_attend_chunk(cache, qb, 0, n, 1.0, chunk, n_requests=1), want, tol, "prompt")
    for p in sorted({first, first + 1, min(first + chunk // 2, n - 1), min(n, first + chunk) - 1}):
        cache.forget(0, p // chunk * chunk)
        for split in (1, 4):
            _close(_attend_chunk(cache, qb, p, p + 1, 1.0, chunk, n_split=split), want[p:p + 1], tol, f"token {p}")


# ---- latent attention --------------------------------------------------------------------------------------------
def test_latent_rows_and_query_latents_are_written_in_one_launch():
    """Rows of a fused projection: the cache row (norm with gain; neighbours rotated, the rest unchanged), the queries'
    latent (norm with its gain), and each of the two alone."""
    from quanta_b200 import kernels
    for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
        C, R, Q, page, eps, T = 24, 12, 20, 4, 1e-3, 11
        g = torch.Generator().manual_seed(3)
        fused = torch.randn(T, Q + C + R + 5, generator=g).to(DEV)
        gain, q_gain = 1 + 0.3 * torch.randn(C, generator=g), 1 + 0.3 * torch.randn(Q, generator=g)
        pos = torch.arange(3, 3 + T)
        for rotated in (12, 8):
            rot = {"dims": rotated, "base": 30.0}
            freqs = torch.tensor(P.frequencies(rot), dtype=torch.float32, device=DEV)
            cache = Pages([14], [C + R], 1, page, dtype, seed=2)
            cq = torch.full((T, Q), 9.0, dtype=dtype, device=DEV)
            args = (gain.to(DEV), freqs, cache.streams[0], pos.to(DEV, torch.int32), _i32([0] * T), cache.dev_table, C, R, rotated,
                    page, eps, cache.status)
            kernels.latent_write(fused[:, Q: Q + C + R], *args, interleaved=True, q_down=fused[:, :Q], q_gain=q_gain.to(DEV), q_out=cq)
            rows = fused.cpu()
            want_q = P.rms(rows[:, :Q], eps) * q_gain
            want = torch.cat([P.rms(rows[:, Q: Q + C], eps) * gain, P.rotate_neighbours(rows[:, Q + C: Q + C + R], pos, rot)], -1)

            def check(what):
                for t in range(T):
                    p = int(pos[t])
                    _close(cache.streams[0][int(cache.table[0, p // page]), 0, p % page], want[t], tol, (what, t))
            check("both")
            _close(cq, want_q, tol, "queries")
            cache.streams[0].fill_(5.0)
            kernels.latent_write(fused[:, Q: Q + C + R].contiguous(), *args, interleaved=True)
            check("rows alone")
            cq.fill_(9.0)
            cache.streams[0].fill_(5.0)
            kernels.latent_write(None, *args, q_down=fused[:, :Q], q_gain=q_gain.to(DEV), q_out=cq)
            _close(cq, want_q, tol, "queries alone")
            assert float(cache.streams[0].float().min()) == 5.0 and int(cache.status[0]) == 0


def _latent_want(q_lat, q_rot, rows, scale, window, gate, positions):
    """[heads, T, C] of the queries at ``positions`` over the cached rows."""
    C = q_lat.shape[2]
    out = torch.zeros_like(q_lat)
    for t, p in enumerate(positions):
        lo = max(0, p - window + 1) if window else 0
        keys = rows[lo: p + 1]
        s = (q_lat[:, t] @ keys[:, :C].T + q_rot[t] @ keys[:, C:].T) * scale
        out[:, t] = torch.softmax(s, -1) @ keys[:, :C] * torch.sigmoid(gate[t])[:, None]
    return out


def _latent_run(cache, q_lat, q_rot, gate_rows, gate_off, positions, scale, window, n_ranges, dtype, tc, split=True):
    from quanta_b200 import kernels
    H, T, C = q_lat.shape
    out = torch.empty((H, T, C), dtype=dtype, device=DEV)
    kernels.latent_attend(q_lat.to(DEV), q_rot.to(DEV), cache.streams[0], None, out, _i32(positions), _i32([0] * T),
                          cache.dev_table, scale, n_ranges, cache.status, req_start=_i32([0, T]), tensor_cores=tc,
                          window=window, gate=gate_rows.to(DEV)[:, gate_off: gate_off + H], float32_weights=split)
    assert int(cache.status[0]) == 0
    return out.float().cpu()


LATENT_SHAPES = [(16, 64, 16), (5, 104, 24), (3, 40, 8), (6, 80, 16), (33, 136, 24), (2, 512, 64), (1, 200, 40), (4, 264, 8)]


@pytest.mark.parametrize("heads,C,R", LATENT_SHAPES)
@pytest.mark.parametrize("window", [0, 1, 40, 64, 150])
def test_windowed_latent_attention_with_gates(heads, C, R, window):
    """A portion in the middle of a sequence and single tokens, in one and in several ranges, on the tensor cores and on
    the CUDA cores (bfloat16 and float32 caches); pages wholly before the window are gone."""
    from quanta_b200 import kernels
    g = torch.Generator().manual_seed(heads + C + window)
    n, page, scale = 230, 16, 0.4
    gate_rows = torch.randn(40, heads + 4, generator=g) * 2
    for dtype in (torch.bfloat16, torch.float32):
        rows = (torch.randn(n, C + R, generator=g) * 0.5).to(dtype)
        cache = Pages([n], [C + R], 1, page, dtype, seed=C)
        for p in range(n):
            cache.streams[0][int(cache.table[0, p // page]), 0, p % page] = rows[p].to(DEV)
        on_tc = kernels.latent_attend_uses_tensor_cores(dtype, C, R)
        assert on_tc == (dtype == torch.bfloat16)
        for positions in (list(range(0, 5)), list(range(150, 190)), [229]):
            T = len(positions)
            q_lat = torch.randn(heads, T, C, generator=g) * (2.0 / math.sqrt(C))
            q_rot = torch.randn(T, heads, R, generator=g) * (1.0 / math.sqrt(R))
            if on_tc:       # the operands the tensor cores see
                q_lat, q_rot = ((t * scale).to(dtype).float() / scale for t in (q_lat, q_rot))
            if window:
                cache.forget(0, max(0, positions[0] - window + 1))
            want = _latent_want(q_lat, q_rot, rows.float(), scale, window, gate_rows[:T, 2: 2 + heads], positions)
            for n_ranges in (1, 3):
                for tc in ((True, False) if on_tc else (False,)):
                    got = _latent_run(cache, q_lat, q_rot, gate_rows[:T], 2, positions, scale, window, n_ranges, dtype, tc)
                    _close(got, want, 1e-2 if dtype == torch.bfloat16 else 2e-5, (dtype, positions[0], n_ranges, tc))


@pytest.mark.parametrize("window", [7, 64, 96, 100])
@pytest.mark.parametrize("back", [0, -1])
def test_a_key_at_the_edge_of_a_window(window, back):
    """Every query has one key that stands out, ``window - 1`` tokens back (the last one it sees) or ``window`` back (the
    first one it does not see); prompts and single tokens, both precisions."""
    g = torch.Generator().manual_seed(window)
    n, page, heads, C, R = 300, 16, 5, 64, 16
    for dtype in (torch.bfloat16, torch.float32):
        rows = (0.3 * torch.randn(n, C + R, generator=g)).to(dtype)
        cache = Pages([n], [C + R], 1, page, dtype, seed=window)
        for p in range(n):
            cache.streams[0][int(cache.table[0, p // page]), 0, p % page] = rows[p].to(DEV)
        gate = torch.zeros(n, heads)
        q_lat, q_rot = 0.1 * torch.randn(heads, n, C, generator=g), 0.1 * torch.randn(n, heads, R, generator=g)
        for p in range(n):
            key = rows.float()[max(0, p - window + 1 + back)]
            q_lat[:, p] += 14.0 * key[:C] / key[:C].norm() ** 2
        positions = list(range(n))
        want = _latent_want(q_lat, q_rot, rows.float(), 1.0, window, gate, positions)
        other = _latent_want(q_lat, q_rot, rows.float(), 1.0, window - 1 if back == 0 else window + 1, gate, positions)
        assert float((want - other).abs().max()) > 0.3 * float(want.abs().max())          # one token off would show
        tol = 3e-2 if dtype == torch.bfloat16 else 2e-5
        _close(_latent_run(cache, q_lat, q_rot, gate, 0, positions, 1.0, window, 1, dtype, None), want, tol, "prompt")
        for p in (0, window - 1, window, 143, 144, 255, 256, 299):
            cache.forget(0, max(0, p - window + 1))
            for n_ranges in (1, 2):
                got = _latent_run(cache, q_lat[:, p:p + 1].contiguous(), q_rot[p:p + 1].contiguous(), gate[p:p + 1], 0, [p], 1.0,
                                  window, n_ranges, dtype, None)
                _close(got, want[:, p:p + 1], tol, f"token {p}")


def test_softmax_weights_keep_their_bits_on_the_tensor_cores():
    """Two keys with nearly equal weights and opposite values: what is left of the sum lives in the weights' low bits."""
    C, R, page = 64, 16, 16
    cache = Pages([16], [C + R], 1, page, torch.bfloat16)
    rows = torch.zeros(2, C + R)
    rows[0, 0], rows[1, 0], rows[1, C] = 1.0, -1.0, 0.015625
    for p in (0, 1):
        cache.streams[0][int(cache.table[0, 0]), 0, p] = rows[p].to(DEV, torch.bfloat16)
    q_lat, q_rot, gate = torch.zeros(1, 1, C), torch.zeros(1, 1, R), torch.full((1, 1), 50.0)
    q_rot[0, 0, 0] = -0.125                                           # scores 0 and -2^-9
    want = math.tanh(2.0 ** -10)                                      # (1 - e^-d) / (1 + e^-d)
    got = float(_latent_run(cache, q_lat, q_rot, gate, 0, [1], 1.0, 0, 1, torch.bfloat16, True)[0, 0, 0])
    assert abs(got - want) < 0.02 * want
    rounded = float(_latent_run(cache, q_lat, q_rot, gate, 0, [1], 1.0, 0, 1, torch.bfloat16, True, split=False)[0, 0, 0])
    assert abs(rounded - want) > 0.5 * want                           # one bfloat16 part alone would lose it


def test_latent_part_against_the_plain_mixer():
    """The whole mixer: portions and single tokens of one sequence through the part, a window that slides over pages."""
    from quanta_b200 import kernels, matmul
    from quanta_b200.parts.base import LayerCache, StepContext, make
    matmul.configure()
    m = {"heads": 3, "dim": 10, "rot_dim": 6, "vdim": 14, "q_rank": 20, "kv_rank": 22, "scale": 0.4, "mask": {"size": 13},
         "rot": {"base": 25.0, "dims": 6}}
    cfg = {"vocab": 4, "width": 30, "token_side": {"dim": 2}, "layers": [{"type": "latent_attention", "mixer": m, "mlp": None}]}
    w = {k: v.float() for k, v in P.draw_weights(cfg, 5).items()}
    x = torch.randn(50, 30, generator=torch.Generator().manual_seed(1))
    want = P.latent_attention(w, "l0.mix.", x, m, 1e-4)
    q = "l0.mix."
    part = make("mixer", ("latent_attention", dict(
        hidden_size=30, n_heads=3, dim=10, rot_dim=6, value_dim=14, q_rank=20, kv_rank=22, scale=0.4, norm_eps=1e-4, sink=False,
        window=13, float32_weights=True, position=("partial_rotary", dict(head_dim=6, rotary_dim=6, theta=25.0, interleaved=True)),
        names={"dq": q + "dq", "dq_norm": q + "dq.norm", "uq": q + "uq", "dkv": q + "dkv", "dkv_norm": q + "dkv.norm", "uk": q + "uk",
               "uv": q + "uv", "g": q + "g", "o": q + "o"})))
    part.load(lambda n: w[n].to(DEV))
    cache = Pages([50], [28], 1, 4, torch.float32)
    p0 = 0
    for n in (7, 2, 1, 1, 20, 1, 5, 13):
        cache.forget(0, max(0, p0 - 12))
        pos = _i32(list(range(p0, p0 + n)))
        ctx = StepContext(n_tokens=n, positions=pos.view(n, 1), tok_pos=pos, tok_req=_i32([0] * n), req_slot=_i32([0]),
                          req_start=_i32([0, n]), req_len_after=_i32([p0 + n]), status=cache.status, dtype=torch.float32,
                          max_new_tokens_per_req=n, max_len_after=p0 + n)
        got = part.forward(x[p0: p0 + n].to(DEV), ctx, LayerCache(streams={"latent": cache.streams[0]}, page_size=4,
                                                                  block_table=cache.dev_table), {})
        kernels.raise_on_status(cache.status.cpu())
        _close(got, want[p0: p0 + n], 2e-5, f"tokens {p0}:{p0 + n}")
        p0 += n


# ---- the delta rule with a decay per key channel ----------------------------------------------------------------
@pytest.mark.parametrize("lens,cuts", [([37, 12], [[5, 1, 1, 2, 17, 1, 10], [1, 2, 9]]),
                                       ([131, 90], [[50, 33, 1, 47], [35, 2, 53]])])       # the second: blocks of four tokens
@pytest.mark.parametrize("H,G,D,DV", [(4, 2, 12, 20), (4, 4, 64, 32), (2, 1, 24, 8), (3, 3, 10, 14), (8, 2, 128, 64), (1, 1, 40, 130),
                                     (6, 3, 33, 5), (2, 2, 256, 16), (2, 1, 130, 70), (40, 20, 16, 64)])
def test_channel_delta_rule_in_portions(H, G, D, DV, lens, cuts):
    """Two sequences in unequal portions and single tokens, in slots that hold stale states, against the plain
    recurrence over the whole sequences; the state that is left equals the plain one.  The decays differ widely from
    channel to channel."""
    from quanta_b200 import kernels
    g = torch.Generator().manual_seed(H * D + DV)
    C = 2 * G * D + H * DV
    A_log, dt_bias = torch.rand(H, generator=g) * 2 - 1.5, torch.randn(H * D, generator=g) * 2
    seqs, want, want_S = [], [], []
    for n in lens:
        qkv, b = torch.randn(n, C + 5, generator=g), torch.randn(n, H + 3, generator=g) * 2
        a = torch.randn(n, H * D + 2, generator=g) * 2
        seqs.append((qkv, b, a))
        q, k = qkv[:, : G * D].view(n, G, D), qkv[:, G * D: 2 * G * D].view(n, G, D)
        v = qkv[:, 2 * G * D: C].view(n, H, DV)
        q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
        k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        step = torch.nn.functional.softplus(a[:, 1: 1 + H * D] + dt_bias).view(n, H, D)
        decay = torch.exp(-torch.exp(A_log)[None, :, None] * step)
        o, S = P.delta_recurrence(q.double(), k.double(), v.double(), decay.double(), torch.sigmoid(b[:, 2: 2 + H]).double())
        want.append(o.float())
        want_S.append(S.float())
    state = torch.full((3, H, D, DV), 3.0, device=DEV)
    slots = [1, 2]
    for s in slots:
        state[s].zero_()
    done, got = [0, 0], [[], []]
    for step in range(max(len(c) for c in cuts)):
        rows, start, slot, who = [[], [], []], [0], [], []
        for r in (0, 1):
            if step < len(cuts[r]):
                n = cuts[r][step]
                for i in range(3):
                    rows[i].append(seqs[r][i][done[r]: done[r] + n])
                start.append(start[-1] + n)
                slot.append(slots[r])
                who.append((r, n))
                done[r] += n
        qkv, b, a = (torch.cat(x).to(DEV) for x in rows)
        out = torch.empty((qkv.shape[0], H, DV), device=DEV)
        kernels.gated_delta(qkv, b, 0, 2, A_log.to(DEV), dt_bias.to(DEV), state, out, _i32(start), _i32(slot), H, G, D, DV,
                            D ** -0.5, 1e-6, channel_decay=a[:, 1: 1 + H * D])
        at = 0
        for r, n in who:
            got[r].append(out[at: at + n].cpu())
            at += n
    for r in (0, 1):
        _close(torch.cat(got[r]), want[r], 2e-5, f"sequence {r}")
        _close(state[slots[r]], want_S[r], 2e-5, f"state {r}")
    assert float(state[0].min()) == 3.0


def test_a_slow_channel_remembers_and_a_fast_one_forgets():
    """A value written at position 0 is read again 500 tokens later through a key channel that hardly decays, and is
    gone through one that does."""
    from quanta_b200 import kernels
    n, D, DV = 501, 8, 4
    qkv = torch.zeros(n, 2 * D + DV)
    qkv[0, D + 2], qkv[0, D + 5] = 1.0, 1.0                             # the first key: channels 2 and 5
    qkv[0, 2 * D:] = torch.tensor([1.0, -2.0, 3.0, 0.5])
    qkv[1:, D + 7] = 1.0                                                # the others write zeros through channel 7
    b = torch.full((n, 1), 30.0)                                        # beta = 1
    a = torch.full((n, D), -30.0)                                       # hardly any decay
    a[:, 5] = 0.0
    for ch in (2, 5):
        qkv[n - 1, :D] = 0.0
        qkv[n - 1, ch] = 1.0
        state, out = torch.zeros(1, 1, D, DV, device=DEV), torch.empty(n, 1, DV, device=DEV)
        kernels.gated_delta(qkv.to(DEV), b.to(DEV), 0, 0, torch.zeros(1, device=DEV), torch.zeros(D, device=DEV), state, out,
                            _i32([0, n]), _i32([0]), 1, 1, D, DV, 1.0, 1e-6, channel_decay=a.to(DEV))
        want = qkv[0, 2 * D:] / math.sqrt(2.0) if ch == 2 else torch.zeros(DV)
        assert torch.allclose(out[-1, 0].cpu(), want, atol=1e-5), ch


@pytest.mark.parametrize("H,G,D,V,taps,ranks", [(4, 2, 12, 20, 3, (5, 7)), (3, 3, 10, 6, 1, (4, 9)), (6, 2, 16, 24, 5, (16, 8))])
def test_channel_delta_part_against_the_plain_mixer(H, G, D, V, taps, ranks):
    """Projections, convolutions with their state, low-rank decay and gate, per-head norm: portions down to one token."""
    from quanta_b200 import matmul
    from quanta_b200.parts.base import StepContext, make
    matmul.configure()
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "conv": taps}
    cfg = {"vocab": 4, "width": 30, "token_side": {"dim": 2}, "layers": [{"type": "channel_delta", "mixer": m, "mlp": None}]}
    w = {k: v.float() for k, v in P.draw_weights(cfg, 9, ranks).items()}
    x = torch.randn(40, 30, generator=torch.Generator().manual_seed(2))
    want = P.channel_delta(w, "l0.mix.", x, m, 1e-4)
    names = {k: "l0.mix." + k for k in ("q", "k", "v", "b", "A_log", "dt_bias", "norm", "a1", "a2", "g1", "g2", "o")}
    names.update({f"{k}_conv": f"l0.mix.{k}.conv" for k in "qkv"})
    part = make("mixer", ("gated_delta_rule", dict(hidden_size=30, n_heads=H, n_groups=G, dim=D, value_dim=V, conv_taps=taps,
                                                   q_scale=D ** -0.5, unit_eps=1e-6, norm_eps=1e-4, decay_rank=ranks[0],
                                                   gate_rank=ranks[1], gate_activation="sigmoid", names=names)))
    part.load(lambda n: w[n].to(DEV))
    state = {n: torch.zeros((2, *shape), dtype=dt, device=DEV) for n, (shape, dt) in part.state_spec().items()}
    p0 = 0
    for n in (6, 2, 1, 1, 2, 17, 1, 10):
        pos = _i32(list(range(p0, p0 + n)))
        ctx = StepContext(n_tokens=n, positions=pos.view(n, 1), tok_pos=pos, tok_req=_i32([0] * n), req_slot=_i32([1]),
                          req_start=_i32([0, n]), req_len_after=_i32([p0 + n]), status=_i32([0, 0, 0, 0]), dtype=torch.float32)
        _close(part.forward(x[p0: p0 + n].to(DEV), ctx, None, state), want[p0: p0 + n], 3e-5, f"tokens {p0}:{p0 + n}")
        p0 += n


# ---- feed-forward, the token's own input, the parallel sum ---------------------------------------------------------
@pytest.mark.parametrize("I", [20, 64, 72])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_activations(I, dtype):
    """All three forms, sizes that move in 16-byte pieces and sizes that do not."""
    from quanta_b200 import kernels
    g = torch.Generator().manual_seed(I)
    gu, bias = (torch.randn(9, 2 * I, generator=g) * 3).to(dtype), torch.randn(2 * I, generator=g)
    a, b = gu.float()[:, :I], gu.float()[:, I:]
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    out = torch.empty((9, I), dtype=dtype, device=DEV)
    kernels.glu_act(gu.to(DEV), out, kind=kernels.GLU_GELU_TANH)
    _close(out, P.gelu_tanh(a) * b, tol, "gelu")
    kernels.glu_act(gu.to(DEV), out, bias=bias.to(DEV))
    _close(out, torch.nn.functional.silu(a + bias[:I]) * (b + bias[I:]), tol, "silu with biases")
    kernels.glu_act(gu.to(DEV), out, kind=kernels.GLU_CLAMPED, limit=0.9, alpha=1.702)
    ac, bc = torch.clamp(a, max=0.9), torch.clamp(b, -0.9, 0.9)
    _close(out, ac * torch.sigmoid(1.702 * ac) * (bc + 1), tol, "clamped")


@pytest.mark.parametrize("T,W,D,layers,index", [(1, 48, 5, 3, 1), (8, 64, 16, 2, 0), (9, 33, 7, 4, 3), (40, 72, 12, 3, 2), (3, 136, 24, 1, 0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_tokens_own_input(T, W, D, layers, index, dtype):
    """Gate, gather of the layer's part of the token's row, projection, norm and sum; the gate inside the launch and as a
    library product."""
    from quanta_b200 import kernels, matmul
    from quanta_b200.parts.base import StepContext, make
    matmul.configure()
    g = torch.Generator().manual_seed(W)
    V, eps = 19, 1e-3
    w = {"gate": torch.randn(D, W, generator=g) * 1.5 / math.sqrt(W), "proj": torch.randn(W, D, generator=g),
         "norm": torch.rand(W, generator=g) + 0.5, "table": torch.randn(V, D * layers, generator=g)}
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    x = torch.randn(T, W, generator=g).to(dtype).float()
    ids = torch.randint(0, V, (T,), generator=g)
    e = w["table"][ids, index * D: (index + 1) * D]
    want_g = P.gelu_tanh(x @ w["gate"].T) * e
    tol = 3e-6 if dtype == torch.float32 else 1e-2
    d = lambda t: t.to(DEV, dtype)  # noqa: E731
    status = kernels.new_status(DEV)
    for gate in (None, (x @ w["gate"].T).to(DEV)):
        out = torch.empty((T, D), dtype=dtype, device=DEV)
        kernels.token_input(d(x), d(w["gate"]), d(w["table"]), index * D, ids.to(DEV, torch.int32), out, status, gate=gate)
        _close(out, want_g, tol, "gate")
    part = make("token_input", ("gated_token_row", dict(
        hidden_size=W, vocab_size=V, dim=D, index=index, layers=layers, names={"table": "table", "gate": "gate", "proj": "proj"},
        norm=("rms_norm", dict(width=W, eps=eps, weight_name="norm")))))
    part.load(lambda n: d(w[n]))
    part.norm.load(lambda n: w[n].to(DEV))
    ctx = StepContext(n_tokens=T, positions=None, tok_pos=None, tok_req=None, req_slot=None, req_start=None, req_len_after=None,
                      status=status, dtype=dtype, token_ids=ids.to(DEV, torch.int32))
    h = x.to(DEV)
    normed = torch.empty((T, W), dtype=torch.float32, device=DEV)
    nxt = make("norm", ("rms_norm", dict(width=W, eps=eps, weight_name="norm")))
    nxt.load(lambda n: w[n].to(DEV))
    nxt.forward(h, part.forward(d(x), ctx), normed)
    want = x + P.token_input({"gate": w["gate"], "proj": w["proj"], "norm": w["norm"]}, "", x, e, eps)
    _close(h, want, tol, "stream")
    _close(normed, P.rms(want, eps) * w["norm"], tol, "next norm")
    # a token id outside the table is refused by the host's next read
    kernels.token_input(d(x), d(w["gate"]), d(w["table"]), index * D, _i32([V] * T), out, status)
    with pytest.raises(kernels.KernelError):
        kernels.raise_on_status(status.cpu())


@pytest.mark.parametrize("W", [40, 256, 66])
def test_two_sublayers_join_the_stream_together(W):
    """``Addends`` as a pending contribution: a norm that reads it adds both outputs; so does the plain copy."""
    from quanta_b200.parts.base import Addends, make
    g = torch.Generator().manual_seed(W)
    h, a, b, gain = (torch.randn(5, W, generator=g) for _ in range(4))
    gain = gain[0]
    x = h + a + b
    for norm, want in ((("rms_norm", dict(width=W, eps=1e-3, weight_name="w")), P.rms(x, 1e-3) * gain), (("none", dict(width=W)), x)):
        part = make("norm", norm)
        part.load(lambda n: gain.to(DEV))
        hd, out = h.clone().to(DEV), torch.empty((5, W), device=DEV)
        part.forward(hd, Addends(a.to(DEV), extra=b.to(DEV)), out)
        _close(hd, x, 1e-6, "stream")
        _close(out, want, 2e-6, norm[0])
