"""Bibalix's mechanisms one at a time: each kernel and each part against the plain function of the
same mechanism.

Attention cases plant dominating keys (a key and one query are scaled so that its score stands out),
another one for each map of a token: on either side of the window's edge, on either side of the last
kept token, at page borders, the very first, the token itself; in prompt portions and in single-token
steps, through every kernel that takes the sizes.  Pages that no request holds are filled with
not-a-number, so a value read from one shows."""

import math

import pytest
import torch

from somi_inference_b200.config import BibalixConfig
from somi_inference_b200.parts import FEED_FORWARDS, MIXERS, NORMS, BuildContext, declared_tensors
from somi_inference_b200.parts.base import PagedKVNeeds
from somi_inference_b200.parts.position import rotary_frequencies
from tests.bibalix_tiny import dense, latent, layer, moe, random_weights, two_maps
from tests.gpu_util import Steps, gather_cache
from tests.plain import bibalix_plain as plain

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
STEPS = ({"a": 9, "b": 1}, {"a": 1, "b": 1, "c": 30}, {"c": 1, "a": 2, "b": 40}, {"a": 1, "c": 1},
         {"a": 17, "b": 2, "c": 8})


@pytest.fixture(scope="module")
def ops():
    from somi_inference_b200.ops import cuda_ops
    return cuda_ops()


def tol(dtype, f32=2e-5, bf16=2e-2):
    return f32 if dtype == torch.float32 else bf16


def one_layer_model(kind, mixer, mlp, width=40, eps=1e-5):
    return dict(architecture="Bibalix", vocab=11, width=width, norm={"eps": eps},
                layers=[layer(kind, mixer, mlp)])


def build_parts(raw, ops, dtype, seed):
    """(mixer, feed-forward or None, weights by name as float64) of the only layer of `raw`."""
    w = random_weights(raw, seed, dtype)
    model = BibalixConfig.from_dict(raw).to_model_spec()
    spec, decl = model.layers[0], declared_tensors(model)
    ctx = BuildContext(dtype=dtype, device=torch.device("cuda"), ops=ops)
    placed = {k: ctx.place(v, matrix=decl[k].matrix) for k, v in w.items()}
    mixer = MIXERS.build(spec.mixer, placed, ctx)
    ff = None if spec.feed_forward is None else FEED_FORWARDS.build(spec.feed_forward, placed, ctx)
    return mixer, ff, {k: v.double() for k, v in w.items()}


def summed(t):
    return t.double().sum(0) if t.dim() == 3 else t.double()


LATENT = ("latent_attention", latent(1, 4, 2, 4, 4, 0.5, None, 10.0))


# ------------------------------------------------------------------------ norms
@pytest.mark.parametrize("width, tokens", [(48, 9), (256, 3), (1030, 5), (37, 9), (4104, 2), (1536, 300)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_layer_norm_with_a_bias(ops, dtype, width, tokens):
    g = torch.Generator().manual_seed(width)
    T, H, eps = tokens, width, 1e-3
    rnd = lambda *s: torch.randn(s, generator=g)
    w, b = (1 + 0.3 * rnd(H)).to(dtype).cuda(), (0.5 * rnd(H)).to(dtype).cuda()
    ctx = BuildContext(dtype=dtype, device=torch.device("cuda"), ops=ops)
    norm = NORMS.get("layernorm")({"size": H, "eps": eps, "names": {"weight": "w", "bias": "b"}}, {"w": w, "b": b}, ctx)
    res = (rnd(T, H) * 2 + 1.5).cuda()
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32, device="cuda")
    for delta in (None, rnd(T, H).to(dtype).cuda(), rnd(3, T, H).cuda(), rnd(T, H).cuda()):
        want = res.double() if delta is None else res.double() + summed(delta)
        x = res.clone()
        got = norm.forward(x, delta)
        ref = plain.layer_norm(want, w.double(), b.double(), eps)
        assert (x.double() - want).abs().max().item() < 1e-5
        assert (got.double() - ref).abs().max().item() < tol(dtype, 2e-5, 3e-2)
        y = res.clone()
        got = norm.forward(y, delta, rows)
        assert torch.equal(y, res)
        assert (got.double() - ref[rows.long()]).abs().max().item() < tol(dtype, 2e-5, 3e-2)


# ------------------------------------------------------------- rotation, norms and cache rows
@pytest.mark.parametrize("case", [
    # (heads, kv heads, key width, value width, rotated, normed, scaling factor, columns behind)
    (4, 2, 12, 28, 8, True, None, 0), (1, 1, 5, 3, 4, True, 8.0, 3), (3, 1, 10, 8, 10, True, None, 1),
    (6, 2, 64, 128, 32, True, None, 8), (2, 2, 32, 64, 0, True, None, 0), (8, 1, 16, 32, 16, False, 2.0, 0),
    (30, 5, 64, 128, 48, True, 4.0, 40), (1, 1, 128, 256, 128, True, None, 8), (2, 1, 256, 8, 16, True, 8.0, 8),
    (9, 3, 32, 24, 16, False, None, 0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_two_queries_and_two_keys_a_head(ops, dtype, case):
    H, G, d, dv, rot, normed, factor, pad = case
    g = torch.Generator().manual_seed(d + dv)
    steps = Steps(ops, 2, paged=PagedKVNeeds(G, 2 * d, None, dv if dv != 2 * d else None), dtype=dtype, page_size=4)
    steps.step({"a": 30})
    batch, where = steps.step({"a": 5, "b": 7} if H < 30 else {"a": 300, "b": 1})
    wide = torch.randn((batch.num_tokens, 2 * (H + G) * d + G * dv + pad), generator=g).to(dtype).cuda()
    qkv = wide.clone()
    qw = (1 + 0.3 * torch.randn(d, generator=g)).to(dtype).cuda() if normed else None
    kw = (1 + 0.3 * torch.randn(d, generator=g)).to(dtype).cuda() if normed else None
    eps = 1e-3
    rot_cfg = {"dims": rot, "base": 700.0}
    if factor is not None:
        rot_cfg["scaling"] = dict(factor=factor, original=64, fast=8.0, slow=1.0)
    freq, mag = rotary_frequencies({**rot_cfg, "scaling": {"kind": "ramp", **rot_cfg["scaling"]}} if factor else rot_cfg)
    view = steps.mgr.view(0).paged
    ops.headnorm_rotary_store(qkv, batch.positions, freq.cuda(), 2 * H, 2 * G, d, dv, rot, qw, kw, eps,
                              batch.groups[0].slot_map, view.keys, view.values, magnitude=mag, maps=2)
    table = batch.groups[0].block_table.cpu()
    bound = tol(dtype, 1e-5, 3e-2)
    for j, r in enumerate(batch.host.requests):
        first, q, c = where[r]
        x = wide[first:first + q].double().cpu()
        qs, ks = x[:, :2 * H * d].reshape(q, 2 * H, d), x[:, 2 * H * d:2 * (H + G) * d].reshape(q, 2 * G, d)
        if normed:
            qs, ks = plain.rms_norm(qs, qw.double().cpu(), eps), plain.rms_norm(ks, kw.double().cpu(), eps)
        qs, ks = plain.rotate_halves(qs, rot_cfg, first=c), plain.rotate_halves(ks, rot_cfg, first=c)
        keys, values = gather_cache(view, table[j], c + q, 4)
        assert (qkv[first:first + q, :2 * H * d].double().cpu().reshape(q, 2 * H, d) - qs).abs().max() < bound
        assert (keys[c:].reshape(q, 2 * G, d) - ks).abs().max() < bound
        assert torch.equal(values[c:].reshape(q, G * dv), x[:, 2 * (H + G) * d:2 * (H + G) * d + G * dv])
    if pad:
        assert torch.equal(qkv[:, -pad:], wide[:, -pad:])


@pytest.mark.parametrize("case", [
    # (heads, query width, rotated, latent, scaling factor)
    (3, 8, 6, 16, 4.0), (1, 7, 2, 5, None), (5, 16, 16, 40, 8.0), (4, 32, 32, 256, 32.0), (2, 12, 4, 24, 2.0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_rows_with_a_scaled_rotation(ops, dtype, case):
    H, qd, rot, rank, factor = case
    g = torch.Generator().manual_seed(rank)
    W = rank + rot
    steps = Steps(ops, 2, paged=PagedKVNeeds(1, W, None, value_dim=0), dtype=dtype, page_size=4)
    steps.step({"a": 30})
    batch, where = steps.step({"a": 5, "b": 7})
    T, c_at = batch.num_tokens, H * (qd + rot)
    x = torch.randn((T, c_at + W + 2 + (c_at + W) % 2), generator=g).to(dtype).cuda()
    w = (1 + 0.3 * torch.randn(rank, generator=g)).to(dtype).cuda()
    rot_cfg = {"dims": rot, "base": 40.0}
    if factor is not None:
        rot_cfg["scaling"] = dict(factor=factor, original=30, fast=3.0, slow=0.5)
    freq, mag = rotary_frequencies({**rot_cfg, "scaling": {"kind": "ramp", **rot_cfg["scaling"]}} if factor else rot_cfg)
    assert (mag > 1.05) == (factor is not None)
    view = steps.mgr.view(0).paged
    qa = torch.full((H, T, W), 7.0, dtype=dtype, device="cuda")
    ops.latent_rotary_store(x, 0, H, qd, rot, c_at, rank, batch.positions, freq.cuda(), False, w, 1e-3,
                            batch.groups[0].slot_map, view.keys, qa, magnitude=mag)
    assert (qa[:, :, :rank] == 7.0).all()
    table = batch.groups[0].block_table.cpu()
    bound = tol(dtype, 1e-5, 3e-2)
    for j, r in enumerate(batch.host.requests):
        first, q, c = where[r]
        rows = x[first:first + q].double().cpu()
        cache = torch.stack([view.keys[int(table[j, p // 4]), 0, p % 4] for p in range(c, c + q)]).double().cpu()
        assert (cache[:, :rank] - plain.rms_norm(rows[:, c_at:c_at + rank], w.double().cpu(), 1e-3)).abs().max() < bound
        want = plain.rotate_halves(rows[:, None, c_at + rank:c_at + W], rot_cfg, first=c)[:, 0]
        assert (cache[:, rank:] - want).abs().max() < bound
        tails = rows[:, :c_at].reshape(q, H, qd + rot)[..., qd:]
        got = qa[:, first:first + q, rank:].double().cpu().transpose(0, 1)
        assert (got - plain.rotate_halves(tails, rot_cfg, first=c)).abs().max() < bound


# ------------------------------------------------------------- two maps, kept tokens, planted keys
@pytest.mark.parametrize("case", [
    # (heads, kv heads, key width, value width, window, kept, page size)
    (4, 2, 12, 28, 9, 3, 8), (2, 1, 16, 32, 21, 21, 4), (3, 3, 5, 3, 1, 7, 4), (2, 2, 24, 16, 64, 0, 16),
    (1, 1, 20, 40, None, 0, 16), (4, 1, 130, 8, 33, 40, 16),
    (6, 3, 32, 64, 36, 5, 16), (4, 2, 64, 128, 130, 17, 16), (2, 1, 64, 128, 20, 129, 8), (8, 1, 64, 128, None, 0, 16),
    (3, 3, 32, 64, 129, 128, 32), (2, 2, 64, 128, 1, 1, 64), (7, 1, 64, 128, 300, 40, 16), (2, 2, 32, 64, 5, 0, 16)])
@pytest.mark.parametrize("gated", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
def test_two_map_attention_with_planted_keys(ops, dtype, case, gated):
    H, G, d, dv, window, keep, ps = case
    g = torch.Generator().manual_seed(10 * (window or 7) + keep)
    reach = window or 10 ** 6
    steps = Steps(ops, 7, paged=PagedKVNeeds(G, 2 * d, window, dv if dv != 2 * d else None, keep), dtype=dtype,
                  page_size=ps, max_len=700)
    steps.step({"a": 130, "b": 2 * reach + 3 if reach < 100 else 77, "c": 1, "d": min(reach, 300), "g": 610})
    batch, where = steps.step({"a": 19, "b": 1, "c": 2, "d": 1, "e": 37, "f": 450, "g": 1})
    view = steps.mgr.view(0).paged
    for t in (view.keys, view.values):
        t.copy_(torch.randn(t.shape, generator=g).to(dtype))
    held = torch.zeros(view.keys.shape[0], dtype=torch.bool)
    for r in where:
        held[steps.mgr.held_pages(r, 0)] = True
    view.keys[~held] = float("nan")
    view.values[~held] = float("nan")
    width = 2 * (H + G) * d + G * dv
    gate_at = width + (-width % 8)
    qkv = torch.randn((batch.num_tokens, gate_at + 16), generator=g).to(dtype)
    table = batch.groups[0].block_table.cpu()
    planted = 0
    for j, r in enumerate(batch.host.requests):
        first, q, c = where[r]
        for i in range(q):
            p = c + i
            oldest = max(0, p - reach + 1)
            targets = [oldest, oldest - 1, keep - 1, keep, p - p % ps - 1, 0, p]
            for n in (0, 1):
                target = targets[(i + j + 3 * n) % 7]
                page = int(table[j, target // ps]) if 0 <= target <= p else -1
                if page < 0:      # given back: it is out of sight and must not be read anyway
                    continue
                sign = torch.where(torch.randn(d, generator=g) > 0, 1.0, -1.0)
                key = view.keys[page, :, target % ps]
                key[:, n * d:(n + 1) * d] = (min(6.0, 20.0 / (0.4 * d)) * sign).to(dtype).cuda()
                qkv[first + i, :2 * H * d].view(H, 2, d)[:, n] = sign.to(dtype)
                planted += 1
    assert planted > 20
    qkv = qkv.cuda()
    gate = qkv[:, gate_at:gate_at + H] if gated else None
    factor, eps, gain, scale = 0.4, 1e-5, 0.65, 0.4
    mask = None if window is None else {"size": window, "keep_first": keep}
    wants = {}
    for j, r in enumerate(batch.host.requests):
        first, q, c = where[r]
        keys, values = gather_cache(view, table[j], c + q, ps)
        seen = plain.visible(c + q, mask)[c:]
        rows = qkv[first:first + q].double().cpu()
        qs = rows[:, :2 * H * d].reshape(q, H, 2, d)
        want = torch.zeros((q, H, dv), dtype=torch.float64)
        for h in range(H):
            kh = h // (H // G)
            a = [plain.softmax_attention(qs[:, h, n], keys[:, kh, n * d:(n + 1) * d], values[:, kh], scale, seen)
                 for n in (0, 1)]
            want[:, h] = plain.difference_of_maps(a[0], a[1], factor, 1.0 - gain, eps)
            if gated:
                want[:, h] *= plain.sigmoid(rows[:, gate_at + h])[:, None]
        wants[r] = want.reshape(q, H * dv)
    kernels = [(True, True, 0)]
    if dtype == torch.bfloat16 and dv == 2 * d and dv in (64, 128):
        # tensor cores with one chunk of keys a CTA and with several; the kernel for any size
        kernels = [(True, True, 1), (True, True, 2), (True, True, 5), (False, False, 0), (True, False, 0)]
    saved = ops.use_pp_prefill, ops.use_tma_decode
    for choice in kernels:
        out = torch.full((batch.num_tokens, H * dv), float("nan"), dtype=dtype, device="cuda")
        ops.use_pp_prefill, ops.use_tma_decode = choice[:2]
        ops.set_decode_ring_chunks(choice[2])
        try:
            ops.two_map_attention(qkv, view.keys, view.values, batch, batch.groups[0], H, G, d, dv, scale, window,
                                  keep, factor, eps, gain, gate, out, storage=view.storage)
        finally:
            ops.use_pp_prefill, ops.use_tma_decode = saved
            ops.set_decode_ring_chunks(0)
        ops.check_errors()
        for r, (first, q, c) in where.items():
            err = (out[first:first + q].double().cpu() - wants[r]).abs().max().item()
            assert err < tol(dtype, 1e-4, 5e-2), (r, c, q, err, choice)


@pytest.mark.parametrize("case", [
    # (heads, latent, tail, page size, window)
    (3, 16, 6, 8, 1), (5, 40, 16, 4, 23), (4, 64, 16, 16, 64), (70, 128, 64, 16, 129), (4, 256, 32, 16, 100),
    (2, 512, 64, 16, 70), (1, 512, 8, 16, 200)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_window_with_planted_keys(ops, dtype, case):
    """Queries that point at one cached row each, through its latent or through its rotated tail:
    just inside and just outside the window, at page borders, the token itself."""
    H, R, tail, ps, window = case
    g = torch.Generator().manual_seed(R + tail)
    W = R + tail
    steps = Steps(ops, 5, paged=PagedKVNeeds(1, W, window, value_dim=0), dtype=dtype, page_size=ps, max_len=400)
    steps.step({"a": 300, "b": 77, "c": 1, "d": 129})
    batch, where = steps.step({"a": 1, "b": 19, "c": 2, "d": 1, "e": 200})
    view = steps.mgr.view(0).paged
    view.keys.copy_(torch.randn(view.keys.shape, generator=g).to(dtype))
    qa = torch.randn((H, batch.num_tokens, W), generator=g).to(dtype) * 0.3
    table = batch.groups[0].block_table.cpu()
    for j, r in enumerate(batch.host.requests):
        first, q, c = where[r]
        for i in range(q):
            p = c + i
            oldest = max(0, p - window + 1)
            target = [oldest, oldest - 1, p - p % ps - 1, p][(i + j) % 4]
            page = int(table[j, target // ps]) if target >= 0 else -1
            if page < 0:
                continue
            lo, hi = (R, W) if (i + j) % 2 else (0, R)
            sign = torch.where(torch.randn(hi - lo, generator=g) > 0, 1.0, -1.0)
            big = (16.0 / (0.5 * (hi - lo))) ** 0.5
            view.keys[page, 0, target % ps, lo:hi] = (big * sign).to(dtype).cuda()
            qa[:, first + i] = 0.0
            qa[:, first + i, lo:hi] = (big * sign).to(dtype)
    qa = qa.cuda()
    out = torch.empty((H, batch.num_tokens, R), dtype=dtype, device="cuda")
    ops.latent_attention(qa, view.keys, batch, batch.groups[0], H, R, 0.5, window, None, out, tail=tail)
    for j, r in enumerate(batch.host.requests):
        first, q, c = where[r]
        rows = torch.zeros((c + q, W), dtype=torch.float64)
        for p in range(c + q):
            page = int(table[j, p // ps])
            if page >= 0:
                rows[p] = view.keys[page, 0, p % ps].double().cpu()
        seen = plain.visible(c + q, {"size": window})[c:]
        for h in range(0, H, 1 + H // 6):
            want = plain.softmax_attention(qa[h, first:first + q].double().cpu(), rows, rows[:, :R], 0.5, seen)
            err = (out[h, first:first + q].double().cpu() - want).abs().max().item()
            assert err < tol(dtype, 4e-5, 4e-2), (r, c, q, h, err)


# ------------------------------------------------------------------ router, experts, dense
@pytest.mark.parametrize("n, top, factor, behind", [(9, 4, 1.5, 7), (5, 1, 0.25, 0), (3, 3, 1.0, 1), (64, 6, 2.0, 8)])
def test_router_softmax_over_all_times_a_factor(ops, n, top, factor, behind):
    """Weights are the chosen scores of a softmax over all experts, times the factor; columns behind
    the experts' (another product's outputs) take no part."""
    g = torch.Generator().manual_seed(n)
    logits = torch.randn((61, n + behind), generator=g).cuda() * 2
    if behind:
        logits[:, n:] += 30.0
    chosen, weight = ops.moe_router_select(logits, None, 1, 1, top, outputs=n, factor=factor)
    z = logits[:, :n].double().cpu()
    idx, wt = plain.choose_experts(z, {"top": top, "scale": factor})
    assert torch.equal(chosen.cpu().long(), idx)
    assert (weight.double().cpu() - wt).abs().max().item() < 1e-6
    # the same from partial sums, and the column behind the outputs summed beside it
    parts = torch.randn((5, *logits.shape), generator=g).cuda()
    parts[-1] += logits - parts.sum(0)
    again, w2, *behind_sum = ops.moe_router_select(parts, None, 1, 1, top, outputs=n, factor=factor, tail=behind > 0)
    z = parts.double().sum(0).cpu()
    clear = plain.choice_margin(z[:, :n], {"top": top}) > 1e-4
    assert torch.equal(again.cpu().long()[clear], idx[clear]) and clear.sum() > 50
    assert (w2.double().cpu() - wt)[clear].abs().max().item() < 1e-5
    if behind:
        assert (behind_sum[0].double().cpu() - z[:, n]).abs().max().item() < 1e-4


@pytest.mark.parametrize("tokens", [1, 5, 16, 40, 130])
@pytest.mark.parametrize("experts, top, ff, limit, scale, shared", [
    (8, 3, 24, 0.5, 1.7, (40, 0.8)), (3, 1, 20, 1.5, None, None), (2, 2, 9, 0.7, 0.5, (7, 2.0)),
    (6, 3, 64, 1.0, 2.5, (24, 0.4)), (1, 1, 16, 0.9, 1.0, (16, 0.9))])
@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_beside_a_gated_shared_expert(ops, dtype, tokens, experts, top, ff, limit, scale, shared):
    """One token to many (every way through the experts), against the plain mixture; rows whose
    choice is a close call in bfloat16 are left out."""
    raw = one_layer_model(*LATENT, moe(experts, top, ff, limit, scale, shared))
    _, part, w = build_parts(raw, ops, dtype, experts)
    steps = Steps(ops, 1, dtype=dtype, max_len=256)
    batch, _ = steps.step({"a": tokens})
    x = (1.5 * torch.randn((tokens, 40), generator=torch.Generator().manual_seed(tokens))).to(dtype)
    got = summed(part.forward(x.cuda(), batch)).cpu()
    ops.check_errors()
    margins = []
    mlp = raw["layers"][0]["mlp"]
    want = plain.expert_mixture(x.double(), w, "l0.mlp.", mlp, margins)
    keep = margins[0] > (2e-2 if dtype == torch.bfloat16 else 1e-5)
    assert keep.sum().item() * 2 >= tokens
    assert (x.double() @ w["l0.mlp.e0.gate"].T > limit).any()
    err = (got - want)[keep].abs().max().item()
    assert err < tol(dtype, 3e-5, 4e-2) * max(1.0, want.abs().max().item())
    if shared is not None:       # the gate and the shared expert are large enough to be seen missing
        alone = plain.expert(x.double(), w, "l0.mlp.shared.", shared[1])
        assert (want - (want - plain.sigmoid(x.double() @ w["l0.mlp.shared.sg"].T) * alone)).abs().max() > 0.05


@pytest.mark.parametrize("tokens", [1, 7, 16, 40, 200])
@pytest.mark.parametrize("width, ff", [(40, 24), (37, 33), (64, 72), (2048, 96)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_gelu_gated_feed_forward(ops, dtype, tokens, width, ff):
    """In the decode product's epilogue (few tokens) and as a kernel of its own; gates from far below
    zero to far above."""
    raw = one_layer_model(*LATENT, dense(ff), width=width)
    _, part, w = build_parts(raw, ops, dtype, 5)
    steps = Steps(ops, 1, dtype=dtype, max_len=256)
    batch, _ = steps.step({"a": tokens})
    x = (2.0 * torch.randn((tokens, width), generator=torch.Generator().manual_seed(tokens))).to(dtype)
    x[0] *= 8.0
    got = summed(part.forward(x.cuda(), batch)).cpu()
    ops.check_errors()
    want = plain.gelu_dense(x.double(), w, "l0.mlp.")
    assert (x.double() @ w["l0.mlp.gate"].T).abs().max() > 10
    assert torch.isfinite(got).all()
    assert (got - want).abs().max().item() < tol(dtype, 3e-5, 2e-2) * max(1.0, want.abs().max().item())


# ------------------------------------------------------------------ whole mixers over steps
MIXER_CASES = {
    "attention": ("attention", two_maps(4, 2, 12, 28, 0.5, 0.3, 9, 5, 8, 500.0)),
    "attention_no_window": ("attention", two_maps(6, 3, 10, 20, 0.4, 0.6, None, None, 10, 300.0)),
    "attention_32": ("attention", two_maps(4, 2, 32, 64, 0.25, 0.4, 21, 11, 16, 1e4)),
    "attention_64": ("attention", two_maps(3, 1, 64, 128, 0.18, 0.2, 14, 3, 64, 1e4)),
    "attention_odd": ("attention", two_maps(3, 3, 9, 7, 0.4, 0.5, 1, 2, 4, 30.0)),
    "latent": ("latent_attention", latent(3, 8, 6, 12, 16, 0.3, 9, 300.0, (4.0, 32, 4.0, 1.0))),
    "latent_wide": ("latent_attention", latent(2, 32, 24, 48, 72, 0.2, 17, 1e4, (8.0, 256, 32.0, 1.0))),
    "latent_no_window": ("latent_attention", latent(4, 16, 8, 16, 32, 0.3, None, 1e4)),
    "latent_odd": ("latent_attention", latent(1, 5, 2, 3, 7, 0.5, 1, 20.0)),
}


@pytest.mark.parametrize("case", list(MIXER_CASES))
@pytest.mark.parametrize("dtype", DTYPES)
def test_mixers_alone_over_steps(ops, dtype, case):
    """Each mixer by itself, three requests in five steps of unequal portions and single tokens,
    against the plain mixer on whole sequences."""
    kind, m = MIXER_CASES[case]
    raw = one_layer_model(kind, m, None)
    mixer, _, w = build_parts(raw, ops, dtype, 7)
    if kind == "attention":
        assert mixer.factor == pytest.approx(float(plain.second_map_factor(w, "l0.mix.", m["diff"])), abs=1e-6)
    needs = mixer.cache_needs()
    steps = Steps(ops, 3, paged=needs.paged, state=needs.state, dtype=dtype, page_size=8)
    g = torch.Generator().manual_seed(3)
    seqs = {r: torch.randn((60, 40), generator=g).to(dtype) for r in "abc"}
    view = steps.mgr.view(0)
    got = {r: [] for r in seqs}
    for counts in STEPS:
        batch, where = steps.step(counts)
        rows = torch.zeros((batch.num_tokens, 40), dtype=dtype)
        for r, (first, q, c) in where.items():
            rows[first:first + q] = seqs[r][c:c + q]
        y = summed(mixer.forward(rows.cuda(), batch, view, True)).cpu()
        for r, (first, q, c) in where.items():
            got[r].append(y[first:first + q])
    ops.check_errors()
    for r in seqs:
        have = torch.cat(got[r])
        want = plain.mixer(kind, seqs[r].double(), w, "l0.mix.", m, 1e-5)[:len(have)]
        err = (have - want).abs().max().item()
        assert err < tol(dtype, 5e-5, 8e-2) * max(1.0, want.abs().max().item()), (r, err)


def test_angles_far_along_a_sequence(ops):
    """Positions up to a million: float32 results stay within a rounding of the exact rotation."""
    d, T = 16, 6
    pos = torch.tensor([0, 1, 4097, 65535, 300001, 1048575], dtype=torch.int32, device="cuda")
    qkv = torch.randn((T, 4 * d + 8), generator=torch.Generator().manual_seed(0)).cuda()
    got = qkv.clone()
    rot = {"dims": d, "base": 1e4, "scaling": dict(factor=4.0, original=2048, fast=32.0, slow=1.0)}
    freq, mag = rotary_frequencies({**rot, "scaling": {"kind": "ramp", **rot["scaling"]}})
    ops.headnorm_rotary_store(got, pos, freq.cuda(), 2, 2, d, 8, d, None, None, 0.0, None, None, None,
                              magnitude=mag, maps=2)
    for i, p in enumerate(pos.tolist()):
        want = plain.rotate_halves(qkv[i:i + 1, :2 * d].double().cpu().reshape(1, 2, d), rot, first=p)
        assert (got[i, :2 * d].double().cpu().reshape(2, d) - want[0]).abs().max() < 3e-6
    assert mag == pytest.approx(0.1 * math.log(4.0) + 1)
