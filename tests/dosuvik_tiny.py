"""Small Dosuvik configurations for the tests, with random weights that make faults show.

A: every kind of layer, grouped heads, values wider and narrower than keys, rotation on part of
   the head, windows (9, 21) that are no multiple of the page (8), a layer without a feed-forward,
   a dense feed-forward whose limit cuts, groups of experts of which some are dropped.
B: an odd width, one head, widths that are no multiple of 4 or 8, a window of one (a token sees only
   itself) beside an attention without a window, no rotation of keys, a router without groups whose
   tokens take every expert, groups of one expert each.
C: keys and values of equal width, a window of 64 over pages of 16, several retention heads, a latent
   wider than the model, tokens that take one expert.
D: head sizes of 64 and 128, key widths of 128 in the recurrence, windows (48, 200) that are no
   multiple of a key tile, a page or a query tile, a latent of 256 with 32 rotated elements.
"""

from __future__ import annotations

import torch

from somi_inference_b200.config import DosuvikConfig
from somi_inference_b200.parts import declared_tensors


def windowed(heads, kv_heads, dim, vdim, scale, window, dims, base):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot={"dims": dims, "base": base})
    if window is not None:
        m["mask"] = {"size": window}
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
                rot={"dims": rot_dim, "base": base})


def retention(dim, vdim, decay, dims, base):
    return dict(heads=len(decay), dim=dim, vdim=vdim, decay=list(decay), rot={"dims": dims, "base": base})


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, groups=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


TINY_A = dict(architecture="Dosuvik", vocab=127, width=48, norm={"eps": 1e-5},
              layers=[layer("retention", retention(10, 6, (0.9, 0.99, 0.5), 8, 100.0), dense(40, 0.8)),
                      layer("attention", windowed(4, 2, 12, 20, 0.4, 9, 8, 500.0), moe(8, 3, 24, (4, 2))),
                      layer("latent_attention", latent(3, 8, 6, 12, 16, 0.3, 300.0), None),
                      layer("attention", windowed(3, 1, 16, 8, 0.35, 21, 16, 1e4), moe(6, 2, 16, (2, 1))),
                      layer("retention", retention(16, 24, (0.97, 0.8), 4, 1e4), moe(9, 4, 20, (3, 2)))])
TINY_B = dict(architecture="Dosuvik", vocab=67, width=45, norm={"eps": 1e-4},
              layers=[layer("attention", windowed(1, 1, 5, 6, 0.8, 1, 0, 50.0), moe(3, 3, 9)),
                      layer("latent_attention", latent(1, 7, 2, 3, 5, 0.5, 20.0), dense(33, 2.5)),
                      layer("attention", windowed(3, 3, 10, 2, 0.5, None, 6, 80.0), moe(4, 2, 21, (4, 3))),
                      layer("retention", retention(3, 5, (0.75,), 2, 10.0), None)])
TINY_C = dict(architecture="Dosuvik", vocab=257, width=96, norm={"eps": 1e-6},
              layers=[layer("latent_attention", latent(4, 24, 8, 24, 104, 0.2, 1e4), dense(64, 1.0)),
                      layer("attention", windowed(4, 2, 32, 32, 0.25, 64, 32, 1e6), dense(72, 1.5)),
                      layer("retention", retention(8, 8, (0.5, 0.9, 0.95, 0.98, 0.99, 0.999), 8, 2e4),
                            moe(8, 5, 24, (2, 2))),
                      layer("latent_attention", latent(5, 16, 16, 8, 40, 0.25, 5e4), dense(56, 0.7)),
                      layer("attention", windowed(6, 6, 16, 16, 0.3, 30, 8, 100.0), moe(10, 1, 40, (5, 2)))])
TINY_D = dict(architecture="Dosuvik", vocab=300, width=128, norm={"eps": 1e-6},
              layers=[layer("attention", windowed(4, 2, 64, 64, 0.15, 48, 48, 1e4), dense(96, 1.2)),
                      layer("retention", retention(128, 32, (0.96, 0.9995), 64, 1e5), moe(8, 2, 64, (4, 2))),
                      layer("latent_attention", latent(4, 32, 32, 64, 256, 0.15, 3e4), moe(6, 3, 64, (2, 1))),
                      layer("attention", windowed(2, 1, 128, 128, 0.1, 200, 128, 1e4), moe(3, 2, 48))])
TINY = {"A": TINY_A, "B": TINY_B, "C": TINY_C, "D": TINY_D}
PAGE_SIZES = {"A": 8, "B": 4, "C": 16, "D": 16}


def random_weights(raw: dict, seed: int, dtype=torch.float32) -> dict[str, torch.Tensor]:
    """Tensors for `raw`, by name: query and key matrices spread widely enough that attention is
    peaked; sinks of a score's own size; norm weights spread around zero (around one for the plain
    ones); every earlier result takes part in the averages over depth; routers and their corrections
    spread the choice scores without saturating the sigmoids.  The layers' norms are small on
    average, so that a branch moves the stream by a fraction of its size and the rounding of
    bfloat16 is not multiplied from layer to layer; a retention's keys resemble its queries, so that a
    token's own q.k, which the norm per head turns into a sign at a sequence's first positions, stays
    away from zero."""
    g = torch.Generator().manual_seed(seed)
    cfg = DosuvikConfig.from_dict(raw)
    retentions = {f"l{i}.mix.k" for i, l in enumerate(cfg.layers) if l.type == "retention"}
    out = {}
    for name, decl in declared_tensors(cfg.to_model_spec()).items():
        shape = tuple(decl.shape)
        last = name.split(".")[-1]
        noise = torch.randn(shape, generator=g)
        if last in ("norm1", "norm2"):
            t = -0.4 + 0.2 * noise
        elif name == "final.norm":
            t = 0.2 * noise
        elif last == "norm":
            t = 1.0 + 0.2 * noise
        elif last == "sink":
            t = 1.5 * noise
        elif last == "dwa":
            t = 0.25 * noise
            t[-1] += 0.8
        elif last == "correction":
            t = 0.7 * noise
        elif last == "router":
            t = noise * (3.0 / shape[1] ** 0.5)
        elif name == "embed":
            t = noise
        elif last in ("q", "k"):
            t = noise * (1.8 / shape[1] ** 0.5)
            if name in retentions:
                t = 0.8 * out[name[:-1] + "q"].float() + 0.6 * t
        else:
            t = noise * (1.2 / shape[1] ** 0.5)
        out[name] = t.to(dtype)
    return out


def stored_values(weights: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
    """The weights as float64, exactly the values that were stored."""
    return {k: v.double() for k, v in weights.items()}


def random_tokens(n: int, vocab: int, seed: int) -> list[int]:
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
