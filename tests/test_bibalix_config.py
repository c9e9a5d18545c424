"""Bibalix: reading config.json, what it refuses, the model spec it produces (parts, tensor names, the
tied head); the plain implementation's mechanisms against cases written out by hand; pages of kept
first tokens in the cache manager and the scheduler's bounds."""

import copy
import json
import math
import random

import pytest
import torch

from somi_inference_b200.cache import FREED, CacheManager
from somi_inference_b200.config import BibalixConfig, ConfigError, load_config
from somi_inference_b200.engine.scheduler import Request, Scheduler
from somi_inference_b200.parts import declared_tensors
from somi_inference_b200.parts.base import CacheNeeds, PagedKVNeeds
from somi_inference_b200.parts.feedforward import GATED_FORMS, gated_form
from somi_inference_b200.parts.position import rotary_frequencies
from somi_inference_b200.sampling import SamplingParams
from somi_inference_b200.weights.random_init import random_tensors
from tests.bibalix_tiny import TINY, TINY_A, TINY_B, TINY_C, random_tokens, random_weights, stored_values
from tests.plain import bibalix_plain as plain

F64 = torch.float64


# ------------------------------------------------------------------------ config
def test_round_trip_and_registry(tmp_path):
    for raw in TINY.values():
        cfg = BibalixConfig.from_dict(raw)
        assert BibalixConfig.from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == raw
    (tmp_path / "config.json").write_text(json.dumps(TINY_A))
    cfg = load_config(str(tmp_path))
    assert isinstance(cfg, BibalixConfig) and cfg.vocab_size == 131
    assert cfg.hidden_size == 48 and cfg.norm_eps == 1e-5


def test_spec_parts_and_names():
    spec = BibalixConfig.from_dict(TINY_A).to_model_spec()
    assert [r.layer for r in spec.schedule] == [0, 1, 2, 3]
    assert all(r.cache_of is None and r.average is None for r in spec.schedule)
    assert [l.mixer.kind for l in spec.layers] == ["differential_attention", "latent_attention"] * 2
    assert [None if l.feed_forward is None else l.feed_forward.kind for l in spec.layers] == \
        ["clamped_glu", "routed_moe", None, "routed_moe"]
    for i, l in enumerate(spec.layers):
        assert l.arrangement == "pre_norm" and l.norms["mixer"].params["names"]["bias"] == f"l{i}.norm1.b"
        assert ("feed_forward" in l.norms) == (l.feed_forward is not None)
    a = spec.layers[0].mixer.params
    assert a["mask"] == {"kind": "window", "size": 9, "keep_first": 3} and a["start"] == 0.3
    assert a["qkv_bias"] and a["head_norm"] and a["head_gate"] and a["rotary"] == {"dims": 8, "base": 500.0}
    z = spec.layers[1].mixer.params
    assert z["window"] == 21 and z["gate"] == "head" and z["q_rank"] is None
    assert z["rotary"]["scaling"] == {"kind": "ramp", "factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 1.0}
    ff = spec.layers[1].feed_forward.params
    assert ff["factor"] == 1.6 and ff["gated"] == {"limit": 0.7, "alpha": 1.702, "shift": 1.0}
    assert ff["shared"]["ff"] == 20 and ff["shared"]["gated"]["limit"] == 0.5 and ff["shared"]["token_gate"]
    assert spec.layers[0].feed_forward.params["activation"] == "gelu_tanh"
    assert spec.head.params["tied"] and spec.head.params["names"]["tied_to"] == "embed"
    names = {n: d.shape for n, d in declared_tensors(spec).items() if not d.ignored}
    assert "head" not in names and names["final.norm.b"] == (48,)
    assert names["l0.mix.q"] == (96, 48) and names["l0.mix.q.b"] == (96,) and names["l0.mix.q.norm"] == (12,)
    assert names["l0.mix.k"] == (48, 48) and names["l0.mix.v"] == (56, 48) and names["l0.mix.v.b"] == (56,)
    assert names["l0.mix.lq1"] == names["l0.mix.lk2"] == (12,) and names["l0.mix.g"] == (4, 48)
    assert names["l0.mix.o"] == (48, 112) and "l0.mix.o.b" not in names
    assert names["l1.mix.q"] == (42, 48) and names["l1.mix.dkv"] == (22, 48) and names["l1.mix.g"] == (3, 48)
    assert names["l1.mix.uk"] == (24, 16) and names["l1.mix.uv"] == (36, 16) and "l1.mix.q.b" not in names
    assert names["l1.mlp.router"] == (7, 48) and names["l1.mlp.e6.down"] == (48, 24)
    assert names["l1.mlp.shared.sg"] == (1, 48) and names["l1.mlp.shared.down"] == (48, 20)
    assert "l2.norm2" not in names and "l2.mlp.gate" not in names
    b = BibalixConfig.from_dict(TINY_B).to_model_spec()
    assert b.layers[0].mixer.params["mask"] is None and b.layers[1].mixer.params["window"] is None
    assert b.layers[0].feed_forward.params["shared"] is None and b.layers[0].feed_forward.params["factor"] == 1.0
    assert "scaling" not in b.layers[1].mixer.params["rotary"]


def test_random_tensors_cover_every_declared_name():
    cfg = BibalixConfig.from_dict(TINY_C)
    w = random_tensors(cfg, 5)
    assert set(w) == {n for n, d in declared_tensors(cfg.to_model_spec()).items() if not d.ignored}
    assert w["l0.norm1.b"].abs().max() == 0 and w["l0.mix.dkv.norm"].min() == 1


@pytest.mark.parametrize("change, what", [
    (lambda d: d.pop("width"), "lacks"),
    (lambda d: d["layers"][0].update(type="mamba"), "not a mixer"),
    (lambda d: d["layers"][0]["mixer"].update(heads=3), "multiple of kv_heads"),
    (lambda d: d["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=14), "even"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda d: d["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=4), "rot_dim"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), "positive"),
    (lambda d: d["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda d: d["layers"][1]["mlp"]["expert"].update(limit=0), "limit"),
    (lambda d: d["layers"][1]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=8), "exceeds"),
    (lambda d: d["layers"][1]["mlp"].update(kind="other"), "kind"),
    (lambda d: d["norm"].update(eps=0), "eps"),
])
def test_what_is_refused(change, what):
    d = copy.deepcopy(TINY_A)
    change(d)
    with pytest.raises(ConfigError, match=what):
        BibalixConfig.from_dict(d)


# ---------------------------------------------------------- the plain mechanisms by hand
def test_visible_keys_by_hand():
    seen = plain.visible(7, {"size": 2, "keep_first": 3})
    assert [[j for j in range(7) if seen[i, j]] for i in range(7)] == \
        [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [0, 1, 2, 3, 4], [0, 1, 2, 4, 5], [0, 1, 2, 5, 6]]
    assert plain.visible(4, {"size": 1}).equal(torch.eye(4, dtype=torch.bool))
    assert plain.visible(4, None).sum() == 10


def test_layer_norm_and_gelu_by_hand():
    x = torch.tensor([[1.0, 3.0]], dtype=F64)
    y = plain.layer_norm(x, torch.tensor([2.0, 5.0]), torch.tensor([0.5, -1.0]), 0.0)
    assert torch.allclose(y, torch.tensor([[-1.5, 4.0]], dtype=F64))
    z = torch.linspace(-6, 6, 41, dtype=F64)
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    # the product's form of it: z sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3))
    limit, alpha, shift, cubic = gated_form({"activation": "gelu_tanh"})
    assert torch.allclose(z * plain.sigmoid(alpha * (z + cubic * z ** 3)), plain.gelu_tanh(z)) and shift == 0
    assert limit == math.inf and GATED_FORMS["silu"] == (math.inf, 1.0, 0.0, 0.0)
    with pytest.raises(ValueError, match="unknown gated"):
        gated_form({"activation": "tanh"})
    with pytest.raises(ValueError, match="positive"):
        gated_form({"limit": 0, "alpha": 1.0, "shift": 0.0})


def test_scaled_frequencies_by_hand():
    rot = {"dims": 8, "base": 10000.0, "scaling": dict(factor=4.0, original=2048, fast=32.0, slow=1.0)}
    place = lambda t: 8 * math.log(2048 / (2 * math.pi * t)) / (2 * math.log(10000.0))
    lo, hi = math.floor(place(32)), math.ceil(place(1))
    assert (lo, hi) == (1, 3)
    f = [10000.0 ** (-2 * i / 8) for i in range(4)]
    freq, mag = plain.turn_frequencies(rot)
    want = [f[0], f[1], f[2] / 4 * 0.5 + f[2] * 0.5, f[3] / 4]
    assert freq == pytest.approx(want) and mag == pytest.approx(0.1 * math.log(4.0) + 1.0)
    got, m2 = rotary_frequencies({"dims": 8, "base": 10000.0, "scaling": {"kind": "ramp", **rot["scaling"]}})
    assert got.tolist() == pytest.approx(freq) and m2 == pytest.approx(mag)
    # both cut-offs on one pair: the ramp's width is held above zero
    tight = {"dims": 4, "base": 100.0, "scaling": dict(factor=2.0, original=7, fast=1.0, slow=1.0)}
    got, _ = rotary_frequencies({**tight, "scaling": {"kind": "ramp", **tight["scaling"]}})
    assert got.tolist() == pytest.approx(plain.turn_frequencies(tight)[0])
    x = torch.tensor([[[1.0, 0.0, 0.0, 0.0, 0.0, 0.0, 0.0, 0.0, 9.0]]], dtype=F64)
    y = plain.rotate_halves(x, rot, first=5)[0, 0]
    assert y[0] == pytest.approx(math.cos(5.0) * mag) and y[4] == pytest.approx(math.sin(5.0) * mag)
    assert y[8] == 9.0


def test_difference_of_maps_by_hand():
    a1, a2 = torch.tensor([[3.0, 1.0]], dtype=F64), torch.tensor([[2.0, 4.0]], dtype=F64)
    y = plain.difference_of_maps(a1, a2, 0.5, 0.2, 0.0)           # (2, -1) over sqrt(2.5), times 0.8
    assert y[0].tolist() == pytest.approx([2 / math.sqrt(2.5) * 0.8, -1 / math.sqrt(2.5) * 0.8])
    w = {n: torch.tensor(v, dtype=F64) for n, v in
         dict(lq1=[1.0, 0.5], lk1=[0.2, 0.4], lq2=[0.0, 1.0], lk2=[5.0, -0.3]).items()}
    assert float(plain.second_map_factor(w, "", 0.3)) == pytest.approx(math.exp(0.4) - math.exp(-0.3) + 0.3)


def test_two_map_attention_of_one_token_is_its_value():
    """The first token sees itself only: both maps give its value, whose direction the norm keeps."""
    raw = TINY_A
    w = stored_values(random_weights(raw, 1))
    m = raw["layers"][0]["mixer"]
    h = torch.randn((1, 48), generator=torch.Generator().manual_seed(2), dtype=F64)
    v = (h @ w["l0.mix.v"].T + w["l0.mix.v.b"]).reshape(2, 28)
    d = v * (1 - plain.second_map_factor(w, "l0.mix.", 0.3))
    d = d / torch.sqrt((d * d).mean(1, keepdim=True) + 1e-5) * 0.7
    gate = plain.sigmoid(h @ w["l0.mix.g"].T)[0]
    heads = torch.cat([d[i // 2] * gate[i] for i in range(4)])
    assert torch.allclose(plain.two_map_attention(h, w, "l0.mix.", m, 1e-5)[0], heads @ w["l0.mix.o"].T)


def test_choice_of_experts_by_hand():
    z = torch.tensor([[0.0, 2.0, 1.0, -1.0]], dtype=F64)
    idx, wt = plain.choose_experts(z, {"top": 2, "scale": 1.5})
    total = sum(math.exp(v) for v in (0.0, 2.0, 1.0, -1.0))
    assert idx.tolist() == [[1, 2]]
    assert wt[0].tolist() == pytest.approx([1.5 * math.exp(2) / total, 1.5 * math.exp(1) / total])
    assert plain.choice_margin(z, {"top": 2})[0] == 1.0 and plain.choice_margin(z, {"top": 4})[0] == math.inf


def test_expert_by_hand():
    h = torch.tensor([[1.0]], dtype=F64)
    w = {"gate": torch.tensor([[3.0], [-4.0]], dtype=F64), "up": torch.tensor([[5.0], [-5.0]], dtype=F64),
         "down": torch.eye(2, dtype=F64)}
    s = lambda z: 1 / (1 + math.exp(-1.702 * z))
    y = plain.expert(h, w, "", 2.0)
    assert y[0].tolist() == pytest.approx([2 * s(2) * 3.0, -4 * s(-4) * -1.0])   # the gate has no lower limit


@pytest.mark.parametrize("name", list(TINY))
def test_the_prefix_property_and_every_tensor_counts(name):
    """Logits of a position do not change when tokens follow it, and no tensor is read without effect
    (experts may go unchosen)."""
    raw = TINY[name]
    w = stored_values(random_weights(raw, 3))
    toks = random_tokens(24, raw["vocab"], 4)
    full = plain.forward(raw, w, toks)
    assert torch.allclose(plain.forward(raw, w, toks[:15]), full[:15], atol=1e-9)
    for n in w:
        if ".mlp.e" in n:
            continue
        w2 = dict(w)
        w2[n] = w[n] * 1.2 + 0.05
        assert not torch.allclose(plain.forward(raw, w2, toks), full, atol=1e-6), n


# ------------------------------------------------------- kept tokens in cache and scheduler
def kept_manager(window, keep, num_pages, page_size=4, requests=3):
    return CacheManager([CacheNeeds(paged=PagedKVNeeds(1, 8, window, None, keep))], [None],
                        num_pages=num_pages, page_size=page_size, max_requests=requests,
                        max_positions=400, dtype=torch.float32, device="cpu")


@pytest.mark.parametrize("window, keep", [(6, 0), (6, 1), (6, 4), (9, 5), (3, 13), (1, 8), (40, 21)])
def test_pages_of_kept_tokens_stay(window, keep):
    """After every step a request holds exactly the pages that a later token may read, and they are
    the pages it took."""
    rng = random.Random(window * 100 + keep)
    m = kept_manager(window, keep, 40)
    m.register("a")
    table, n, taken = m.groups[0].tables[m.slot("a")], 0, {}
    while n < 150:
        c = rng.choice([1, 1, 2, 5, 11])
        m.reserve("a", c)
        for b in range(-(-(n + c) // 4)):
            if table[b] != FREED:
                assert taken.setdefault(b, int(table[b])) == int(table[b])
        m.commit("a")
        n += c
        readable = {j // 4 for j in range(n) if j < keep or j > n - window}
        held = {b for b in range(-(-n // 4)) if table[b] != FREED}
        # (a page of kept tokens is held from its first token on, even where the last is not yet in)
        assert held >= readable and held - readable <= {(n - 1) // 4} | set(range(-(-keep // 4)))
        assert sorted(m.held_pages("a", 0)) == sorted(int(table[b]) for b in held)
        m.check_consistency()
    m.release("a")
    assert m.free_pages() == [40]


def test_release_and_cancel_before_the_kept_tokens_are_full():
    m = kept_manager(4, 30, 20)
    for n in (1, 9, 30):
        m.register(n)
        m.reserve(n, n)
        m.cancel(n)
        assert m.free_pages() == [20]
        m.reserve(n, n)
        m.commit(n)
        m.reserve(n, 3)
        m.cancel(n)
        m.check_consistency()
        assert len(m.held_pages(n, 0)) == -(-n // 4)
        m.release(n)
        assert m.free_pages() == [20]


def test_requests_share_a_small_pool_by_window_and_kept_tokens():
    """Groups that differ in their kept tokens only are groups of their own; requests that come and
    go never lose a page."""
    needs = [CacheNeeds(paged=PagedKVNeeds(1, 8, 6, None, k)) for k in (0, 5, 5)]
    m = CacheManager(needs, [None] * 3, num_pages=30, page_size=4, max_requests=4, max_positions=400,
                     dtype=torch.float32, device="cpu")
    assert [len(g.runs) for g in m.groups] == [1, 2] and [g.kept for g in m.groups] == [0, 2]
    rng = random.Random(3)
    live = {}
    for step in range(600):
        if len(live) < 4 and rng.random() < 0.3:
            m.register(step)
            live[step] = 0
        for r in list(live):
            c = rng.choice([1, 1, 3, 7])
            m.reserve(r, c)
            if rng.random() < 0.2:
                m.cancel(r)
                continue
            m.commit(r)
            live[r] += c
            if live[r] > 60:
                m.release(r)
                del live[r]
        m.check_consistency()


@pytest.mark.parametrize("policy", ["preempt", "reserve"])
def test_scheduler_counts_the_kept_tokens(policy):
    """A long request is admitted when window, portion and kept tokens fit, refused one page short."""
    for pages, fits in ((8, True), (7, False)):          # ceil((8 + 4) / 4) + 1 + ceil(13 / 4)
        cache = kept_manager(8, 13, pages)
        s = Scheduler(cache, max_concurrent=1, max_num_batched_tokens=8, chunk_size=4, max_positions=300, policy=policy)
        req = Request("r", list(range(100)), 100, SamplingParams(temperature=0.0))
        if fits:
            s.add_request(req)
        else:
            with pytest.raises(ValueError, match="8 pages"):
                s.add_request(req)
