"""Bibalix models of random sizes, layer orders, windows, kept tokens and constants through the engine
under two ways of cutting the work, against the plain implementation: float32 row by row; bfloat16 by
the root mean square over all rows (a single row may rest on a close call of a router)."""

import json
import os
import random

import pytest
import torch

from somi_inference_b200.weights.safetensors_io import save_safetensors
from tests import replay
from tests.bibalix_tiny import (dense, latent, layer, moe, random_tokens, random_weights, stored_values,
                                two_maps)
from tests.plain import bibalix_plain as plain

pytestmark = pytest.mark.gpu


def random_config(rng: random.Random) -> dict:
    width = rng.choice([64, 96, 160, 192, 320, 104, 90])

    def mixer(kind):
        base = rng.choice([1e4, 5e5, 100.0, 2500.0])
        window = rng.choice([None, 1, 7, 33, 100, 64])
        if kind == "attention":
            heads = rng.choice([2, 4, 6, 8, 3, 1])
            kv = rng.choice([g for g in (1, 2, 3, 4, heads) if heads % g == 0])
            d = rng.choice([8, 16, 32, 32, 48, 64, 64, 24, 10])
            dv = rng.choice([2 * d, 2 * d, 2 * d, 16, 33, 96])
            dims = rng.choice([d, d // 2, 8, 0])
            return two_maps(heads, kv, d, dv, 0.6 * d ** -0.5, rng.uniform(0.05, 0.6), window,
                            None if window is None else rng.choice([None, 0, 1, 4, 16, 17, 40]), dims - dims % 2, base)
        scaling = None
        if rng.random() < 0.8:
            scaling = (rng.choice([2.0, 8.0, 32.0]), rng.choice([32, 512, 4096]), rng.choice([32.0, 8.0]), rng.choice([1.0, 2.0]))
        return latent(rng.choice([1, 3, 5, 8]), rng.choice([16, 32, 40, 1]), rng.choice([2, 8, 16, 24, 6]),
                      rng.choice([16, 32, 24, 7]), rng.choice([16, 40, 64, 136, 200, 36]), rng.choice([0.1, 0.2]),
                      window, base, scaling)

    def feed_forward():
        pick = rng.random()
        if pick < 0.15:
            return None
        if pick < 0.4:
            return dense(rng.choice([16, 64, 96, 200, 20]))
        experts = rng.choice([1, 2, 5, 8, 12])
        shared = None if rng.random() < 0.2 else (rng.choice([16, 40, 96, 9]), rng.choice([0.5, 1.0, 3.0]))
        return moe(experts, rng.randint(1, min(5, experts)), rng.choice([16, 64, 96, 20]), rng.choice([0.5, 1.0, 4.0]),
                   rng.choice([None, 0.5, 1.0, 2.5]), shared)

    layers = [layer(kind, mixer(kind), feed_forward())
              for kind in (rng.choice(["attention", "latent_attention"]) for _ in range(rng.choice([3, 4, 6])))]
    return dict(architecture="Bibalix", vocab=rng.choice([100, 513, 333]), width=width,
                norm={"eps": rng.choice([1e-6, 1e-5])}, layers=layers)


@pytest.mark.parametrize("seed", range(8))
def test_random_models_in_portions_and_mixed_batches(tmp_path, seed):
    from somi_inference_b200.engine import Engine
    raw = random_config(random.Random(300 + seed))
    reqs = {f"r{i}": random_tokens(n, raw["vocab"], 50 + i) for i, n in enumerate([330, 37, 70, 1, 64, 5])}
    for dt, dtype in ((torch.float32, "float32"), (torch.bfloat16, "bfloat16")):
        d = str(tmp_path / dtype)
        os.makedirs(d)
        w = random_weights(raw, seed, dt)
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(raw, f)
        save_safetensors(w, os.path.join(d, "model.safetensors"))
        ref = {rid: plain.forward(raw, stored_values(w), toks) for rid, toks in reqs.items()}
        scale = max(v.abs().max().item() for v in ref.values())
        for cut in (replay.portions, replay.mixed):
            steps, max_tokens = cut(reqs)
            eng = Engine(d, dtype=dtype, page_size=16, max_tokens=max_tokens, max_requests=4)
            got = replay.run_steps(eng, steps)
            eng.ops.check_errors()
            assert len(got) >= 100
            diffs = {k: (row.double() - ref[k[0]][k[1]]) for k, row in got.items()}
            if dtype == "float32":
                worst = max((v.abs().max().item(), k) for k, v in diffs.items())
                assert worst[0] < 2e-4 * scale, (json.dumps(raw), worst)
            else:
                rms = (sum((v ** 2).mean().item() for v in diffs.values()) / len(diffs)) ** 0.5
                assert rms < 3e-2 * scale, (json.dumps(raw), rms)
            assert all(f == eng.num_pages for f in eng.cache.free_pages()), "pages were lost"
