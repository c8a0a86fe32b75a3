"""Whole Lotilix models through the engine against the plain implementation: every cutting of the requests into steps,
both precisions, other orders of layers, long decoding, slots and pages that are given back and used again, generation
through the scheduler and the command line."""

from __future__ import annotations

import json
import math

import pytest
import torch

from tests import helpers as H
from tests.plain import lotilix_plain as P

pytestmark = pytest.mark.gpu


def _latent(heads, dim, rot, vdim, q_rank, kv_rank, window, base=50.0, scale=None, ff=None):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale or (dim + rot) ** -0.5, "mask": {"size": window}, "rot": {"base": base, "dims": rot}}}


def _delta(heads, groups, dim, vdim, conv, ff=None):
    return {"type": "channel_delta", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": groups, "dim": dim, "vdim": vdim, "conv": conv}}


def _attn(heads, kv, dim, chunk, dims, base=100.0, scaling=None, scale=None, ff=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5, "mask": {"size": chunk},
         "rot": {"dims": dims, "base": base}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _config(vocab, width, side, layers, eps=1e-5):
    return {"architecture": "Lotilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "token_side": {"dim": side},
            "layers": layers}


# Configurations that differ in every size and option: windows and chunks from one token to more than the sequence,
# smaller and larger than a page and across its border; one to several heads and groups; sizes that are no multiples of
# 8 or 16 and sizes that take the tensor-core kernels; whole, partial and no rotation; ladders that reach all three
# wavelength ranges; convolutions of one to five taps; layers with and without a feed-forward.
CONFIGS = {
    "A": _config(97, 44, 6, [
        _latent(3, 10, 6, 14, 20, 26, 13, ff=40), _delta(4, 2, 12, 20, 3, ff=24),
        _attn(4, 2, 12, 21, 12, scaling=(3.0, 1.0, 3.0, 40), ff=36), _latent(2, 8, 4, 6, 12, 18, 40)]),
    "B": _config(130, 96, 24, [
        _delta(6, 2, 16, 12, 1), _attn(6, 3, 24, 10, 8, base=5000.0, ff=72), _attn(8, 1, 16, 300, 16, base=30.0, scaling=(8.0, 0.5, 2.0, 64)),
        _latent(5, 24, 16, 40, 40, 48, 9, base=1e4, ff=64), _delta(2, 1, 40, 24, 5, ff=48)], eps=1e-6),
    "C": _config(61, 30, 5, [
        _attn(2, 1, 22, 1, 10, base=9.0), _latent(1, 16, 10, 8, 9, 30, 1, ff=20), _delta(3, 3, 18, 26, 2, ff=20),
        _attn(1, 1, 14, 5, 0, ff=12)], eps=1e-4),
    # shapes that the tensor-core kernels take in bfloat16
    "D": _config(111, 128, 32, [
        _latent(8, 32, 16, 16, 64, 112, 48, ff=96), _attn(8, 2, 64, 40, 32, base=1e4, scaling=(4.0, 1.0, 4.0, 128), ff=160),
        _delta(4, 2, 64, 32, 4, ff=96), _latent(4, 16, 32, 32, 48, 64, 72, base=1e5), _attn(2, 1, 128, 64, 128, ff=64)]),
}
RANKS = {"A": (5, 7), "B": (16, 8), "C": (3, 3), "D": (16, 24)}


def _folder(tmp_path_factory, name, cfg=None, seed=None, ranks=None):
    from quanta_b200.weights.safetensors_io import write_safetensors
    cfg = cfg or CONFIGS[name]
    d = tmp_path_factory.mktemp(f"lotilix_{name}")
    weights = P.draw_weights(cfg, seed=(700 + ord(name[0])) if seed is None else seed, inner_ranks=ranks or RANKS.get(name, (5, 7)))
    write_safetensors(d / "model.safetensors", weights)
    (d / "config.json").write_text(json.dumps(cfg))
    return d, weights, cfg


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return {name: _folder(tmp_path_factory, name) for name in CONFIGS}


def _engine(folder, dtype, steps=None, page_size=16, slots=4, num_pages=None):
    from quanta_b200.engine.model import load_model
    from quanta_b200.engine.step import Engine
    model, _ = load_model(folder, dtype=dtype)
    if num_pages is None:
        num_pages = H.tokens_in_flight(steps, page_size) // page_size
    return Engine(model, num_pages=num_pages, page_size=page_size, max_requests=slots)


def _want(weights, cfg, reqs):
    out = {}
    for rid, toks in reqs.items():
        lg = P.forward(weights, cfg, toks)
        for i in range(len(toks)):
            out[(rid, i)] = lg[i]
    return out


def _shake(weights, cfg, reqs, want):
    """Per position, what the plain model makes of a 2^-9 disturbance of what its sublayers read (the largest of three
    draws): where it turns a rounding into a large difference (a per-head norm of a state that is nearly zero after the
    first tokens, a token's own input whose gates are all nearly closed and that is normed afterwards), bfloat16 results
    say little about the engine."""
    worst: dict = {}
    for seed in (1, 2, 3):
        g = torch.Generator().manual_seed(seed)
        for rid, toks in reqs.items():
            lg = P.forward(weights, cfg, toks, disturb=lambda t: t * (1 + 2.0 ** -9 * torch.randn(t.shape, generator=g)))
            for (_, i), e in _errors({(rid, i): lg[i] for i in range(len(toks))}, want).items():
                worst[(rid, i)] = max(worst.get((rid, i), 0.0), e)
    return worst


def _errors(got, want):
    err = {}
    for key, row in got.items():
        d = row - want[key]
        e = float((d - d.mean()).pow(2).mean().sqrt() / want[key].std())
        err[key] = e if e == e else math.inf
    return err


def _worst(got, want, shake=None):
    err = _errors(got, want)
    if shake is not None:
        assert sum(1 for k in err if 6 * shake[k] < 0.2) >= 0.6 * len(err), "the model is unsteady nearly everywhere"
        err = {k: max(0.0, e - 6 * shake[k]) for k, e in err.items()}
    where = max(err, key=lambda k: err[k])
    return err[where], where


TOL = {"float32": 1e-4, "bfloat16": 0.08}


def _requests(vocab, lengths, seed):
    return {f"r{i}": H.random_tokens(n, vocab, seed + i) for i, n in enumerate(lengths)}


def _compare(folder, want, shake, steps, dtype, what, **engine_args):
    eng = _engine(folder, dtype, steps, **engine_args)
    got = H.replay(eng, steps)
    worst, where = _worst(got, want, shake if dtype == "bfloat16" else None)
    assert worst < TOL[dtype], f"{what} {dtype}: {worst} at {where}"
    assert len(got) == len(want)
    eng.manager.check_invariants()
    assert eng.manager.stats()["live_requests"] == 0
    return eng


@pytest.mark.parametrize("name", list(CONFIGS))
def test_cuttings_agree_with_plain(models, name):
    folder, weights, cfg = models[name]
    reqs = _requests(cfg["vocab"], [1, 2, 37, 70, 5, 110], seed=11)
    want = _want(weights, cfg, reqs)
    shake = _shake(weights, cfg, reqs, want)
    cuttings = {
        "whole": H.cut_whole(reqs),
        "decode": H.cut_tail_decode(reqs, tail=45),
        "portions": H.cut_portions(reqs, sizes=(7, 2, 13, 3, 1, 2, 29, 4, 16, 2)),
        "mixed": H.cut_mixed(reqs, max_live=3, seed=5, portion_sizes=(2, 3, 5, 8, 17, 33)),
    }
    for dtype in ("float32", "bfloat16"):
        for cut, steps in cuttings.items():
            # exactly the pages the cutting needs and three state slots: both are given back and used again
            _compare(folder, want, shake, steps, dtype, f"{name} {cut}", page_size=8 if name in "AC" else 16, slots=3)


ORDERS = {
    "latent_only": [_latent(2, 12, 8, 10, 16, 24, 7, ff=16)],
    "attention_only": [_attn(3, 3, 10, 6, 10, ff=16), _attn(4, 2, 8, 13, 4)],
    "delta_only": [_delta(2, 1, 8, 12, 2), _delta(4, 4, 16, 8, 4, ff=24)],
    "no_feed_forward": [_attn(2, 1, 16, 9, 8), _delta(2, 2, 8, 8, 3), _latent(2, 8, 4, 8, 8, 16, 11)],
    "delta_last": [_latent(4, 8, 8, 8, 24, 32, 30, ff=40), _attn(2, 2, 20, 33, 20, scaling=(16.0, 1.0, 2.0, 24), ff=8), _delta(1, 1, 24, 24, 4, ff=24)],
}


@pytest.mark.parametrize("order", list(ORDERS))
def test_other_orders_of_layers(tmp_path_factory, order):
    cfg = _config(67, 40, 9, ORDERS[order])
    folder, weights, cfg = _folder(tmp_path_factory, "A", cfg=cfg, seed=3, ranks=(4, 11))
    reqs = _requests(cfg["vocab"], [1, 40, 75], seed=1)
    want = _want(weights, cfg, reqs)
    shake = _shake(weights, cfg, reqs, want)
    steps = H.cut_mixed(reqs, max_live=3, seed=5, portion_sizes=(2, 3, 5, 8, 17))
    for dtype in ("float32", "bfloat16"):
        _compare(folder, want, shake, steps, dtype, order, slots=3)


def test_residual_stream_after_every_layer(models):
    from quanta_b200.engine.step import StepEntry
    for name in ("A", "B", "C"):
        folder, weights, cfg = models[name]
        toks = H.random_tokens(29, cfg["vocab"], 3)
        _, layers = P.forward(weights, cfg, toks, details=True)
        eng = _engine(folder, "float32", num_pages=8)
        eng.model.residual_trace = []
        eng.step([StepEntry("a", toks, (0,))], end=["a"])
        assert len(eng.model.residual_trace) == len(cfg["layers"])
        for i, got in enumerate(eng.model.residual_trace):
            want = layers[i]
            assert torch.allclose(got.cpu(), want, atol=1e-4 * float(want.abs().max()), rtol=1e-4), (name, i)


def test_token_by_token_equals_whole_prompt(models):
    for name in ("A", "B", "D"):
        folder, weights, cfg = models[name]
        reqs = _requests(cfg["vocab"], [90], seed=3)
        one, whole = H.cut_tail_decode(reqs, tail=1000), H.cut_whole(reqs)
        a = H.replay(_engine(folder, "float32", one, page_size=4), one)
        b = H.replay(_engine(folder, "float32", whole, page_size=4), whole)
        worst, where = _worst(a, b)
        assert worst < 3e-5, (name, worst, where)


def test_portions_of_two_tokens(models):
    """Portions shorter than the convolutions' reach, that begin and end at every place of a chunk and a window."""
    for name in ("A", "B"):
        folder, weights, cfg = models[name]
        reqs = _requests(cfg["vocab"], [67], seed=8)
        steps = H.cut_portions(reqs, sizes=(2, 2, 1, 2, 3, 2, 1, 1, 2))
        worst, where = _worst(H.replay(_engine(folder, "float32", steps, page_size=4), steps), _want(weights, cfg, reqs))
        assert worst < TOL["float32"], (name, worst, where)


def test_batch_does_not_change_a_request(models):
    folder, weights, cfg = models["D"]
    reqs = _requests(cfg["vocab"], [33, 3, 90, 64], seed=21)
    together = [{"entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in reqs.items()], "end": list(reqs)}]
    alone = H.cut_whole(reqs)
    for dtype, tol in (("float32", 2e-5), ("bfloat16", TOL["bfloat16"])):
        a, b = H.replay(_engine(folder, dtype, together), together), H.replay(_engine(folder, dtype, alone), alone)
        shake = None if dtype == "float32" else _shake(weights, cfg, reqs, _want(weights, cfg, reqs))
        worst, where = _worst(a, b, shake)
        assert worst < tol, (dtype, worst, where)


def test_long_decoding_through_captured_steps(models):
    """A short prompt and 180 single tokens (captured decode steps once the shape has been seen), for two requests side
    by side that cross page, window and chunk borders at different steps."""
    for name in ("A", "D"):
        folder, weights, cfg = models[name]
        reqs = _requests(cfg["vocab"], [187, 201], seed=4)
        steps = [{"entries": [{"id": "r0", "tokens": reqs["r0"][:7], "want": [6]}, {"id": "r1", "tokens": reqs["r1"][:21], "want": [20]}],
                  "end": []}]
        for i in range(180):
            steps.append({"entries": [{"id": "r0", "tokens": [reqs["r0"][7 + i]], "want": [0]},
                                      {"id": "r1", "tokens": [reqs["r1"][21 + i]], "want": [0]}], "end": []})
        want = _want(weights, cfg, reqs)
        shake = _shake(weights, cfg, reqs, want)
        for dtype in ("float32", "bfloat16"):
            eng = _engine(folder, dtype, num_pages=52, page_size=8)
            got = H.replay(eng, steps)
            assert eng.stats()["graph_replays"] > 120
            worst, where = _worst(got, {k: want[k] for k in got}, shake if dtype == "bfloat16" else None)
            assert worst < TOL[dtype], (name, dtype, worst, where)


def test_slots_and_pages_are_used_again(models):
    """One slot and the pages of one request: five requests one after the other, each starting from a zero state and
    empty convolution inputs although the slot and the pages still hold the last request's numbers."""
    folder, weights, cfg = models["A"]
    reqs = _requests(cfg["vocab"], [30, 30, 29, 31, 30], seed=9)
    steps = H.cut_portions(reqs, sizes=(9, 1, 20, 1))
    got = H.replay(_engine(folder, "float32", num_pages=8, page_size=4, slots=1), steps)
    worst, where = _worst(got, _want(weights, cfg, reqs))
    assert worst < TOL["float32"], (worst, where)


def test_a_request_longer_than_the_pool(models):
    """Pages for 64 positions and a request of 200 tokens: what the windows and chunks have passed is given back and
    written again, over and over."""
    folder, weights, cfg = models["A"]                    # the longest window is 40, the chunk 21
    reqs = _requests(cfg["vocab"], [200], seed=14)
    steps = H.cut_portions(reqs, sizes=(9, 2, 16, 1, 1, 1, 5))
    eng = _engine(folder, "float32", num_pages=16, page_size=4, slots=1)
    worst, where = _worst(H.replay(eng, steps), _want(weights, cfg, reqs))
    assert worst < TOL["float32"], (worst, where)
    assert all(g["allocations"] == 50 for g in eng.stats()["groups"])
    eng.manager.check_invariants()


def test_every_constant_counts(tmp_path_factory):
    """The engine agrees with the plain implementation on a model whose constants are all far from neutral, and a plain
    model with ONE constant or tensor changed is far off: none of them is a detail that this test could not see."""
    layers = [_latent(3, 12, 8, 10, 18, 28, 12, base=20.0, scale=0.5, ff=24), _delta(4, 2, 10, 14, 3, ff=20),
              _attn(4, 2, 16, 17, 12, base=40.0, scaling=(4.0, 1.0, 4.0, 24), scale=0.6, ff=28)]
    cfg = _config(50, 42, 6, layers, eps=1e-3)
    folder, weights, cfg = _folder(tmp_path_factory, "A", cfg=cfg, seed=77)
    reqs = _requests(cfg["vocab"], [61], seed=2)
    steps = H.cut_portions(reqs, sizes=(2, 3, 1, 2, 4, 6, 1, 1, 1, 5, 3, 12))
    got = H.replay(_engine(folder, "float32", steps, page_size=4), steps)
    worst, where = _worst(got, _want(weights, cfg, reqs))
    assert worst < TOL["float32"], (worst, where)

    def other(edit, w=None):
        c = json.loads(json.dumps(cfg))
        if edit is not None:
            edit(c)
        return _worst(got, _want(w or weights, c, reqs))[0]

    def setter(layer, path, value):
        def edit(c):
            m = c["layers"][layer]["mixer"]
            for key in path[:-1]:
                m = m[key]
            m[path[-1]] = value
        return edit

    ones = lambda name: dict(weights, **{name: torch.ones_like(weights[name])})  # noqa: E731
    zeros = lambda name: dict(weights, **{name: torch.zeros_like(weights[name])})  # noqa: E731

    def newest_tap(name):
        t = torch.zeros_like(weights[name])
        t[:, -1] = weights[name][:, -1]
        return dict(weights, **{name: t})

    def mean_decay():                       # one decay a head instead of one a channel
        t = weights["l1.mix.dt_bias"].float().view(4, 10).mean(1, keepdim=True).expand(4, 10).reshape(-1)
        a2 = weights["l1.mix.a2"].float().view(4, 10, -1).mean(1, keepdim=True).expand(4, 10, -1).reshape(40, -1)
        return dict(weights, **{"l1.mix.dt_bias": t, "l1.mix.a2": a2})

    swapped = weights["side.embed"].clone()
    swapped[:, :6], swapped[:, 6:12] = weights["side.embed"][:, 6:12], weights["side.embed"][:, :6]
    changed = {
        "window one longer": other(setter(0, ("mask", "size"), 13)),
        "window one shorter": other(setter(0, ("mask", "size"), 11)),
        "latent scale": other(setter(0, ("scale",), 0.7)),
        "latent rotation base": other(setter(0, ("rot", "base"), 80.0)),
        "latent gates": other(None, zeros("l0.mix.g")),
        "query latent gain": other(None, ones("l0.mix.dq.norm")),
        "latent gain": other(None, ones("l0.mix.dkv.norm")),
        "chunk one longer": other(setter(2, ("mask", "size"), 18)),
        "chunk one shorter": other(setter(2, ("mask", "size"), 16)),
        "attention scale": other(setter(2, ("scale",), 0.4)),
        "rotated part": other(setter(2, ("rot", "dims"), 16)),
        "rotation base": other(setter(2, ("rot", "base"), 4.0)),
        "no frequency scaling": other(lambda c: c["layers"][2]["mixer"]["rot"].pop("scaling")),
        "scaling factor": other(setter(2, ("rot", "scaling", "factor"), 8.0)),
        "scaling low": other(setter(2, ("rot", "scaling", "low"), 0.25)),
        "scaling original": other(setter(2, ("rot", "scaling", "original"), 64)),
        "eps": other(lambda c: c["norm"].update(eps=0.5)),
        "decay per channel": other(None, mean_decay()),
        "decay rate": other(None, zeros("l1.mix.A_log")),
        "decay bias": other(None, zeros("l1.mix.dt_bias")),
        "output gate": other(None, zeros("l1.mix.g2")),
        "per-head gain": other(None, ones("l1.mix.norm")),
        "q convolution": other(None, newest_tap("l1.mix.q.conv")),
        "k convolution": other(None, newest_tap("l1.mix.k.conv")),
        "v convolution": other(None, newest_tap("l1.mix.v.conv")),
        "write strength": other(None, zeros("l1.mix.b")),
        "which part of the token's row": other(None, dict(weights, **{"side.embed": swapped})),
        "gain of the token's input": other(None, ones("l2.side.norm")),
        "no token input in a layer": other(None, zeros("l1.side.norm")),
        "layer norm": other(None, ones("l2.norm1")),
        "feed-forward": other(None, zeros("l0.mlp.down")),
    }
    for what, far in changed.items():
        assert far > 30 * TOL["float32"], (what, far)


def test_greedy_generation_through_the_scheduler(models):
    from quanta_b200 import generate
    from quanta_b200.engine.generate import LLM
    for name in ("A", "C"):
        folder, weights, cfg = models[name]
        prompts = [H.random_tokens(n, cfg["vocab"], 40 + n) for n in (9, 23, 4, 31)]
        llm = LLM(str(folder), dtype="float32", page_size=4, num_pages=40, max_requests=2, max_step_tokens=16, prefill_chunk=6)
        got = generate(llm, prompts, max_new_tokens=14, eos_id=[])
        for p, g in zip(prompts, got):
            assert g == P.generate(weights, cfg, p, 14)
        assert llm.last_stats["cache"]["live_requests"] == 0


def test_command_line_and_random_weights(tmp_path):
    """``python -m quanta_b200 random-weights`` writes a folder for this architecture and ``generate`` runs it."""
    import subprocess
    import sys
    cfg = json.loads(json.dumps(CONFIGS["A"]))
    cfg["layers"][1]["mixer"].update(decay_rank=6, gate_rank=10)
    (tmp_path / "c.json").write_text(json.dumps(cfg))
    out = tmp_path / "model"
    root = str(H.__file__).rsplit("/tests/", 1)[0]
    subprocess.run([sys.executable, "-m", "quanta_b200", "random-weights", "--config", str(tmp_path / "c.json"), "--seed", "3",
                    "--out", str(out)], check=True, cwd=root)
    r = subprocess.run([sys.executable, "-m", "quanta_b200", "generate", "--model", str(out), "--prompt-ids", "1,2,3,4,5",
                        "--max-new-tokens", "5", "--dtype", "float32", "--eos-id", "60"], check=True, capture_output=True,
                       text=True, cwd=root)
    ids = [int(x) for x in r.stdout.strip().split(",")]
    from safetensors.torch import load_file
    want = P.generate(load_file(str(out / "model.safetensors")), json.loads((out / "config.json").read_text()), [1, 2, 3, 4, 5], 5)
    if 60 in want:
        want = want[: want.index(60)]
    assert ids == want


def test_trace_program_replays_a_schedule(models, tmp_path):
    import subprocess
    import sys
    import numpy as np
    folder, weights, cfg = models["B"]
    reqs = _requests(cfg["vocab"], [40, 9, 66], seed=31)
    steps = H.cut_mixed(reqs, max_live=3, seed=2, portion_sizes=(2, 5, 17))
    lines = "".join(json.dumps({"step": n, "entries": s["entries"], "end": s["end"]}) + "\n" for n, s in enumerate(steps))
    root = str(H.__file__).rsplit("/tests/", 1)[0]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, root + "/bin/trace_run", "--model", str(folder), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", str(H.tokens_in_flight(steps))], input=lines, capture_output=True, text=True, cwd=root)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {n}" for n in range(len(steps))]
    want = _want(weights, cfg, reqs)
    got, pos = {}, {}
    for n, s in enumerate(steps):
        rows = np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        row = 0
        for e in s["entries"]:
            base = pos.get(e["id"], 0)
            for w in e["want"]:
                got[(e["id"], base + w)] = torch.from_numpy(rows[row].copy())
                row += 1
            pos[e["id"]] = base + len(e["tokens"])
    assert len(got) == sum(len(t) for t in reqs.values())
    worst, where = _worst(got, want)
    assert worst < TOL["float32"], (worst, where)
