"""Small Bibalix configurations for the tests, with random weights that make faults show.

A: every kind of layer, grouped heads, values wider than both keys together and narrower, rotation on
   part of a key, windows (9, 21) that are no multiple of the page (8), kept first tokens that are no
   multiple of it either, a layer without a feed-forward, experts whose limits cut.
B: an odd width, one head, widths that are no multiple of 4 or 8, attention without a window, a window
   of one beside kept tokens, a router whose tokens take every expert, no shared expert, no scaling.
C: the two keys of a head together as wide as a value (one cache tensor) at sizes the tensor-core
   kernels refuse, a window of 40 beside more kept tokens than a page of 16 holds, every head with
   keys of its own, a latent wider than the model, experts of which a token takes one.
D: keys of 64 and 32 under values of 128 and 64 (the tensor-core kernels), windows (48, 200, 90) that
   are no multiple of a key tile, a page or a query tile, kept tokens within a page and beyond a key
   tile, sequences long enough that whole key tiles lie between the kept ones and the window's.
"""

from __future__ import annotations

import torch

from somi_inference_b200.config import BibalixConfig
from somi_inference_b200.parts import declared_tensors


def two_maps(heads, kv_heads, dim, vdim, scale, diff, window, keep, dims, base):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff,
             rot={"dims": dims, "base": base})
    if window is not None:
        m["mask"] = {"size": window} if keep is None else {"size": window, "keep_first": keep}
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, window, base, scaling=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
             rot={"dims": rot_dim, "base": base})
    if window is not None:
        m["mask"] = {"size": window}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling, strict=True))
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, scale=None, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if scale is not None:
        out["router"]["scale"] = scale
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


TINY_A = dict(architecture="Bibalix", vocab=131, width=48, norm={"eps": 1e-5},
              layers=[layer("attention", two_maps(4, 2, 12, 28, 0.4, 0.3, 9, 3, 8, 500.0), dense(40)),
                      layer("latent_attention", latent(3, 8, 6, 12, 16, 0.3, 21, 300.0, (4.0, 64, 8.0, 1.0)),
                            moe(7, 3, 24, 0.7, 1.6, (20, 0.5))),
                      layer("attention", two_maps(3, 1, 10, 8, 0.5, 0.6, 21, 13, 10, 1e3), None),
                      layer("latent_attention", latent(4, 6, 8, 10, 20, 0.35, 9, 1e4, (8.0, 200, 16.0, 2.0)),
                            moe(5, 2, 16, 1.2, 0.8, (28, 0.9)))])
TINY_B = dict(architecture="Bibalix", vocab=71, width=45, norm={"eps": 1e-4},
              layers=[layer("attention", two_maps(1, 1, 5, 3, 0.8, 0.2, None, None, 4, 50.0), moe(3, 3, 9, 0.8)),
                      layer("latent_attention", latent(1, 7, 2, 3, 5, 0.5, None, 20.0), dense(33)),
                      layer("attention", two_maps(3, 3, 6, 7, 0.6, 0.5, 1, 5, 0, 80.0), moe(4, 2, 21, 2.5, 1.0)),
                      layer("latent_attention", latent(2, 3, 4, 6, 9, 0.6, 2, 10.0), None)])
TINY_C = dict(architecture="Bibalix", vocab=263, width=96, norm={"eps": 1e-6},
              layers=[layer("latent_attention", latent(4, 24, 8, 24, 104, 0.2, 64, 1e4, (16.0, 128, 32.0, 1.0)), dense(64)),
                      layer("attention", two_maps(4, 4, 20, 40, 0.25, 0.45, 40, 20, 16, 1e6), moe(9, 1, 40, 0.6, 3.0, (16, 1.5))),
                      layer("attention", two_maps(6, 2, 8, 16, 0.4, 0.1, 30, None, 8, 100.0), dense(72)),
                      layer("latent_attention", latent(5, 16, 16, 8, 40, 0.25, 33, 5e4, (2.0, 4096, 32.0, 1.0)),
                            moe(8, 5, 24, 1.0, 1.3, (48, 0.7)))])
TINY_D = dict(architecture="Bibalix", vocab=300, width=128, norm={"eps": 1e-6},
              layers=[layer("attention", two_maps(4, 2, 64, 128, 0.12, 0.35, 48, 5, 64, 1e4), dense(96)),
                      layer("latent_attention", latent(4, 32, 32, 64, 256, 0.12, 90, 3e4, (8.0, 512, 32.0, 1.0)),
                            moe(6, 2, 64, 1.0, 1.5, (64, 1.2))),
                      layer("attention", two_maps(3, 1, 32, 64, 0.18, 0.55, 90, 131, 16, 1e5), moe(5, 2, 48, 0.8, 2.0, (40, 0.8))),
                      layer("attention", two_maps(2, 2, 64, 128, 0.12, 0.25, 200, 17, 32, 1e4), dense(80))])
TINY = {"A": TINY_A, "B": TINY_B, "C": TINY_C, "D": TINY_D}
PAGE_SIZES = {"A": 8, "B": 4, "C": 16, "D": 16}


def random_weights(raw: dict, seed: int, dtype=torch.float32) -> dict[str, torch.Tensor]:
    """Tensors for `raw`, by name: query and key matrices spread widely enough that attention is
    peaked; biases of the projections' own size; vectors that move the second map's factor without
    bringing it near one (where the two maps of a first token would cancel); routers that spread the
    scores; norm weights around one and biases around zero."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, decl in declared_tensors(BibalixConfig.from_dict(raw).to_model_spec()).items():
        if decl.ignored:
            continue
        shape = tuple(decl.shape)
        parts = name.split(".")
        last = parts[-1]
        noise = torch.randn(shape, generator=g)
        if last == "b":
            t = noise * (0.2 if "norm" in name else 0.4)
        elif "norm" in name:
            t = 1.0 + 0.2 * noise
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = noise * (0.35 / shape[0] ** 0.25)
        elif last == "router":
            t = noise * (2.5 / shape[1] ** 0.5)
        elif last == "sg":
            t = noise * (1.5 / shape[1] ** 0.5)
        elif name == "embed":
            t = 0.4 * noise         # (the head is tied to it: large rows would name their own token)
        elif last in ("q", "k") or last == "dkv":
            t = noise * (1.8 / shape[1] ** 0.5)
        elif last in ("o", "down"):
            t = noise * (0.9 / shape[1] ** 0.5)
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
