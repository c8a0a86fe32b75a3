"""Gate: the Lotilix decoder through the entry point gives the plain implementation's tokens and logits.

A small model (windowed latent attention with gates, a delta rule with a decay per key channel, chunked attention whose
values are its keys, a second latent attention without a feed-forward; a row of the token's own in every layer): greedy
tokens of three prompts fed in portions of 6 beside decoded tokens, pages of 4, two state slots that are used again;
then the logits of one prompt through the step function, whole and token by token."""
# parity-gate: gpu

from __future__ import annotations

import json
import tempfile
from pathlib import Path

from parity._gates import Checks


def _latent(window, mlp):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": 3, "dim": 10, "rot_dim": 6, "vdim": 14, "q_rank": 20, "kv_rank": 26, "scale": 0.3,
                      "mask": {"size": window}, "rot": {"base": 100.0, "dims": 6}}}


CONFIG = {"architecture": "Lotilix", "vocab": 90, "width": 48, "norm": {"eps": 1e-5}, "token_side": {"dim": 10}, "layers": [
    _latent(9, {"kind": "dense", "ff": 40}),
    {"type": "channel_delta", "mlp": {"kind": "dense", "ff": 32},
     "mixer": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 12, "conv": 4}},
    {"type": "attention", "mlp": {"kind": "dense", "ff": 24},
     "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 12, "scale": 0.3, "mask": {"size": 7},
               "rot": {"dims": 8, "base": 100.0, "scaling": {"factor": 3.0, "low": 1.0, "high": 3.0, "original": 40}}}},
    _latent(20, None)]}


def run() -> int:
    import torch

    from quanta_b200 import generate
    from quanta_b200.engine.generate import LLM
    from quanta_b200.weights.safetensors_io import write_safetensors
    from tests import helpers as H
    from tests.plain import lotilix_plain as P

    c = Checks("lotilix_generate_test")
    with tempfile.TemporaryDirectory() as d:
        weights = P.draw_weights(CONFIG, seed=5)
        write_safetensors(Path(d) / "model.safetensors", weights)
        (Path(d) / "config.json").write_text(json.dumps(CONFIG))
        llm = LLM(d, dtype="float32", page_size=4, num_pages=40, max_requests=2, max_step_tokens=12, prefill_chunk=6)
        prompts = [H.random_tokens(n, CONFIG["vocab"], 40 + i) for i, n in enumerate((5, 11, 16))]
        got = generate(llm, prompts, max_new_tokens=8, eos_id=[])
        for p, g in zip(prompts, got):
            c.ok(g == P.generate(weights, CONFIG, p, 8), f"greedy tokens of a prompt of {len(p)}")
        c.ok(llm.engine.manager.stats()["live_requests"] == 0, "all slots released")
        reqs = {"a": H.random_tokens(33, CONFIG["vocab"], 7)}
        want = P.forward(weights, CONFIG, reqs["a"])
        for name, steps in (("whole", H.cut_whole(reqs)), ("token by token", H.cut_tail_decode(reqs, tail=1000))):
            rows = H.replay(llm.engine, steps)
            worst = max(float((rows[("a", i)] - want[i]).abs().max()) for i in range(33))
            c.ok(worst < 2e-4 * float(want.abs().max()), f"logits, {name}: {worst}")
        c.ok(torch.isfinite(want).all().item(), "finite logits")
    c.done()
    return 0


if __name__ == "__main__":
    raise SystemExit(run())
