"""Gate: the Gedelorn decoder through the entry point gives the plain implementation's tokens and logits.

A small model (a state-space recurrence with routed experts, windowed attention with capped scores beside constant-decay
linear attention, a matrix memory with a dense feed-forward, a second state-space layer without one): greedy tokens of
three prompts fed in portions of 6 beside decoded tokens, pages of 4, two state slots that are used again; then the logits
of one prompt through the step function, whole and token by token."""
# parity-gate: gpu

from __future__ import annotations

import json
import tempfile
from pathlib import Path

from parity._gates import Checks

CONFIG = {"architecture": "Gedelorn", "vocab": 90, "width": 48, "norm": {"eps": 1e-5}, "layers": [
    {"type": "mamba2", "mixer": {"heads": 4, "vdim": 10, "state": 12, "groups": 2, "conv": 3, "norm_groups": 2},
     "mlp": {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 5, "top": 2, "scale": 1.3}, "shared": {"ff": 24}}},
    {"type": "parallel", "mlp": {"kind": "dense", "ff": 40},
     "mixer": {"left": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 12, "scale": 0.3, "softcap": 4.0, "mask": {"size": 9},
                        "rot": {"dims": 8, "base": 100.0}},
               "right": {"heads": 3, "dim": 8, "vdim": 10, "decay": [0.6, 0.9, 0.99]}, "left_scale": 0.8, "right_scale": 1.1}},
    {"type": "mlstm", "mixer": {"heads": 2, "dim": 14, "vdim": 18, "gate_cap": 6.0}, "mlp": {"kind": "dense", "ff": 32}},
    {"type": "mamba2", "mixer": {"heads": 2, "vdim": 16, "state": 8, "groups": 1, "conv": 4, "norm_groups": 1}, "mlp": None}]}


def run() -> int:
    import torch

    from quanta_b200 import generate
    from quanta_b200.engine.generate import LLM
    from quanta_b200.weights.safetensors_io import write_safetensors
    from tests import helpers as H
    from tests.plain import gedelorn_plain as P

    c = Checks("gedelorn_generate_test")
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
