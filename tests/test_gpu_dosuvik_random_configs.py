"""Dosuvik models of random sizes, layer orders, windows and constants through the engine under two
ways of cutting the work, against the plain implementation: float32 row by row; bfloat16 by the root
mean square over all rows (a single row may rest on a close call of a router, or on the sign of one
retention head's q.k at a sequence's first positions, which the norm per head turns into the sign
of that head's whole output)."""

import json
import os
import random

import pytest
import torch

from somi_inference_b200.weights.safetensors_io import save_safetensors
from tests import replay
from tests.dosuvik_tiny import (dense, latent, layer, moe, random_tokens, random_weights, retention,
                                stored_values, windowed)
from tests.plain import dosuvik_plain as plain

pytestmark = pytest.mark.gpu


def random_config(rng: random.Random) -> dict:
    width = rng.choice([64, 96, 160, 192, 320, 104, 90])

    def mixer(kind):
        base = rng.choice([1e4, 5e5, 100.0, 2500.0])
        if kind == "attention":
            heads = rng.choice([2, 4, 6, 8, 3])
            kv = rng.choice([g for g in (1, 2, 3, 4, heads) if heads % g == 0])
            d = rng.choice([16, 32, 48, 64, 96, 128, 24])
            dv = rng.choice([d, d, 16, 32, 64, 128])
            dims = rng.choice([d, d // 2, 8])
            return windowed(heads, kv, d, dv, 0.5 * d ** -0.5, rng.choice([None, 1, 7, 33, 100, 64]),
                            dims - dims % 2, base)
        if kind == "latent_attention":
            return latent(rng.choice([1, 3, 5, 8]), rng.choice([16, 32, 40]), rng.choice([2, 8, 16, 24, 6]),
                          rng.choice([16, 32, 24]), rng.choice([16, 40, 64, 136, 200, 36]),
                          rng.choice([0.1, 0.07]), base)
        heads = rng.choice([2, 3, 5, 8])
        d = rng.choice([8, 40, 64, 128, 20])
        dims = rng.choice([d, d // 2, 2, 0])
        return retention(d, rng.choice([8, 64, 96, 20, 32]), [1.0 - 2.0 ** -rng.uniform(1, 12) for _ in range(heads)],
                         dims - dims % 2, base)

    def feed_forward():
        pick = rng.random()
        if pick < 0.15:
            return None
        if pick < 0.4:
            return dense(rng.choice([16, 64, 96, 200, 20]), rng.choice([0.5, 1.0, 3.0]))
        count = rng.choice([1, 2, 3, 4])
        size = rng.choice([2, 3, 4, 1])
        keep = rng.randint(1, count)
        top = rng.randint(1, min(6, keep * size))
        return moe(count * size, top, rng.choice([16, 64, 96, 20]), (count, keep) if count > 1 or rng.random() < 0.5 else None)

    layers = [layer(kind, mixer(kind), feed_forward())
              for kind in (rng.choice(["attention", "latent_attention", "retention"]) for _ in range(rng.choice([3, 4, 6])))]
    return dict(architecture="Dosuvik", vocab=rng.choice([100, 513, 333]), width=width,
                norm={"eps": rng.choice([1e-6, 1e-5])}, layers=layers)


@pytest.mark.parametrize("seed", range(8))
def test_random_models_in_portions_and_mixed_batches(tmp_path, seed):
    from somi_inference_b200.engine import Engine
    raw = random_config(random.Random(200 + seed))
    reqs = {f"r{i}": random_tokens(n, raw["vocab"], 50 + i) for i, n in enumerate([120, 37, 70, 1, 64, 5])}
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
