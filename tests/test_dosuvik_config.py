"""Dosuvik: reading config.json, what it refuses, the model spec it produces (norms behind the
branches only, the average over depth behind every run, parts, tensor names); the plain
implementation's mechanisms against cases written out by hand."""

import copy
import json
import math

import pytest
import torch

from somi_inference_b200.config import (ConfigError, DosuvikConfig, ModelSpec, PartSpec, RunSpec,
                                        load_config)
from somi_inference_b200.parts import declared_tensors
from somi_inference_b200.parts.position import rotary_frequencies
from somi_inference_b200.weights.random_init import random_tensors
from tests.dosuvik_tiny import TINY, TINY_A, TINY_B, TINY_C, random_tokens, random_weights, stored_values
from tests.plain import dosuvik_plain as plain

F64 = torch.float64


def test_round_trip_and_registry(tmp_path):
    for raw in TINY.values():
        cfg = DosuvikConfig.from_dict(raw)
        assert DosuvikConfig.from_dict(cfg.to_dict()) == cfg
    (tmp_path / "config.json").write_text(json.dumps(TINY_A))
    cfg = load_config(str(tmp_path))
    assert isinstance(cfg, DosuvikConfig) and cfg.vocab_size == 127
    assert cfg.hidden_size == 48 and cfg.norm_eps == 1e-5


def test_spec_parts_and_names():
    spec = DosuvikConfig.from_dict(TINY_A).to_model_spec()
    assert [r.layer for r in spec.schedule] == [0, 1, 2, 3, 4]
    assert [r.average for r in spec.schedule] == [f"depth{i}" for i in range(5)]
    assert all(r.cache_of is None and r.remix is None and not r.add_embedding for r in spec.schedule)
    assert [l.mixer.kind for l in spec.layers] == ["retention", "normed_attention", "latent_attention",
                                                    "normed_attention", "retention"]
    assert [None if l.feed_forward is None else l.feed_forward.kind for l in spec.layers] == \
        ["clamped_glu", "routed_moe", None, "routed_moe", "routed_moe"]
    for l in spec.layers:
        assert l.arrangement == "sandwich_norm" and l.norms["mixer"].kind == "none"
        assert l.norms["mixer_post"].params["offset"] == 1.0
        assert ("feed_forward_post" in l.norms) == (l.feed_forward is not None)
    assert spec.final_norm.params["offset"] == 1.0
    a = spec.layers[1].mixer.params
    assert a["row_norm"] and a["turn_values"] and a["sink"] == "learned"
    assert a["mask"] == {"kind": "window", "size": 9} and a["rotary"] == {"dims": 8, "base": 500.0}
    z = spec.layers[2].mixer.params
    assert z["q_rank"] is None and z["rot_dim"] == 6 and z["rotary"]["neighbours"] and z["gate"]
    r = spec.layers[0].mixer.params
    assert r["decay"] == [0.9, 0.99, 0.5] and r["k_scale"] == 10 ** -0.5
    ff = spec.layers[1].feed_forward.params
    assert ff["scores"] == "sigmoid" and ff["correction"] and ff["groups"] == {"count": 4, "keep": 2, "best": 2}
    assert spec.layers[0].feed_forward.params["alpha"] == 1.702
    names = declared_tensors(spec)
    assert names["l1.mix.q"].shape == (48, 48) and names["l1.mix.v"].shape == (40, 48)
    assert names["l1.mix.q.norm"].shape == (48,) and names["l1.mix.k.norm"].shape == (24,)
    assert names["l1.mix.sink"].shape == (4,) and names["l1.mix.o"].shape == (48, 80)
    assert names["l2.mix.q"].shape == (42, 48) and names["l2.mix.dkv"].shape == (22, 48)
    assert names["l2.mix.dkv.norm"].shape == (16,) and names["l2.mix.uk"].shape == (24, 16)
    assert names["l2.mix.uv"].shape == (36, 16) and names["l2.mix.g"].shape == (36, 48)
    assert names["l0.mix.k"].shape == (30, 48) and names["l0.mix.g"].shape == (18, 48)
    assert "l0.mix.norm" not in names and "l2.norm2" not in names and "l2.mlp.router" not in names
    assert names["l0.mlp.gate"].shape == (40, 48) and names["l0.mlp.down"].shape == (48, 40)
    assert names["l1.mlp.router"].shape == (8, 48) and names["l1.mlp.correction"].shape == (8,)
    assert names["l1.mlp.e7.down"].shape == (48, 24) and "l1.mlp.e8.down" not in names
    assert [names[f"l{i}.dwa"].shape for i in range(5)] == [(i + 2,) for i in range(5)]
    b = DosuvikConfig.from_dict(TINY_B).to_model_spec()
    assert b.layers[2].mixer.params["mask"] is None and b.layers[0].feed_forward.params["groups"] is None


def test_averages_over_depth_are_for_every_run_or_none():
    spec = DosuvikConfig.from_dict(TINY_A).to_model_spec()

    def with_schedule(schedule):
        s = {k: getattr(spec, k) for k in spec.__dataclass_fields__}
        ModelSpec(**{**s, "schedule": tuple(schedule)}).validate()

    with_schedule(spec.schedule)
    with pytest.raises(ValueError, match="every run or behind none"):
        with_schedule([RunSpec(0), *spec.schedule[1:]])
    with pytest.raises(ValueError, match="none of the"):
        with_schedule([RunSpec(0, average="nothing")])
    with pytest.raises(ValueError, match="neither re-mixes"):
        with_schedule([spec.schedule[0], RunSpec(1, average="depth1", add_embedding=True)])
    assert isinstance(spec.stream_parts["depth0"], PartSpec)


def test_random_tensors_cover_every_declared_name():
    cfg = DosuvikConfig.from_dict(TINY_C)
    w = random_tensors(cfg, 5)
    assert set(w) == set(declared_tensors(cfg.to_model_spec()))
    assert w["l0.norm1"].abs().max() == 0 and w["l0.mix.dkv.norm"].min() == 1


@pytest.mark.parametrize("change, what", [
    (lambda d: d.pop("width"), "lacks"),
    (lambda d: d["layers"][0].update(type="mamba"), "not a mixer"),
    (lambda d: d["layers"][1]["mixer"].update(heads=3), "multiple of kv_heads"),
    (lambda d: d["layers"][1]["mixer"].update(vdim=7), "even"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"].update(decay=[0.5]), "decay"),
    (lambda d: d["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda d: d["layers"][2]["mixer"]["rot"].update(dims=4), "rot_dim"),
    (lambda d: d["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda d: d["layers"][0]["mlp"].update(limit=0), "limit"),
    (lambda d: d["layers"][1]["mlp"].update(kind="other"), "kind"),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=5), "exceeds"),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(count=3), "divide"),
    (lambda d: d["norm"].update(eps=0.0), "eps"),
])
def test_refusals(change, what):
    raw = copy.deepcopy(TINY_A)
    change(raw)
    with pytest.raises(ConfigError, match=what):
        DosuvikConfig.from_dict(raw)


# --------------------------------------------------------------- plain mechanisms by hand
def test_norms_by_hand():
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    w = torch.tensor([0.5, -1.0], dtype=F64)
    r = math.sqrt(12.5 + 0.1)
    assert torch.allclose(plain.shifted_norm(x, w, 0.1), torch.tensor([[4.5 / r, 0.0]], dtype=F64))
    assert torch.allclose(plain.rms_norm(x, w, 0.1), torch.tensor([[1.5 / r, -4.0 / r]], dtype=F64))


def test_rotations_by_hand():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F64).repeat(3, 1, 1)
    y, z = plain.rotate_halves(x, 4, 100.0), plain.rotate_neighbours(x, 4, 100.0)
    for p in range(3):
        for m, f in enumerate((1.0, 0.1)):
            c, s = math.cos(p * f), math.sin(p * f)
            for got, a, b in ((y, m, m + 2), (z, 2 * m, 2 * m + 1)):
                assert abs(got[p, 0, a] - (x[p, 0, a] * c - x[p, 0, b] * s)) < 1e-12
                assert abs(got[p, 0, b] - (x[p, 0, b] * c + x[p, 0, a] * s)) < 1e-12
        assert y[p, 0, 4] == z[p, 0, 4] == 5.0
    assert torch.allclose(plain.rotate_halves(y, 4, 100.0, sign=-1.0), x)
    got, mag = rotary_frequencies({"dims": 6, "base": 50.0})
    assert got.tolist() == pytest.approx([50.0 ** (-2 * m / 6) for m in range(3)], rel=1e-15) and mag == 1.0


def test_attention_window_sink_and_groups_by_hand():
    q = torch.ones((4, 1, 1), dtype=F64)
    k = torch.tensor([2.0, 0.0, 1.0, 3.0], dtype=F64).reshape(4, 1, 1)
    v = torch.tensor([1.0, 10.0, 100.0, 1000.0], dtype=F64).reshape(4, 1, 1)
    e = math.exp
    o = plain.masked_attention(q, k, v, 1.0, window=2, sink=torch.tensor([0.7], dtype=F64))
    assert abs(o[2, 0, 0] - (e(0) * 10 + e(1) * 100) / (e(0.7) + e(0) + e(1))) < 1e-12   # key 0 is out
    assert abs(o[0, 0, 0] - e(2) / (e(0.7) + e(2))) < 1e-12
    o = plain.masked_attention(q, k, v, 0.5)
    want = sum(e(0.5 * a) * b for a, b in zip((2.0, 0.0, 1.0, 3.0), (1.0, 10.0, 100.0, 1000.0)))
    assert abs(o[3, 0, 0] - want / sum(e(0.5 * a) for a in (2.0, 0.0, 1.0, 3.0))) < 1e-9
    g = torch.Generator().manual_seed(0)
    q4, k2, v2 = (torch.randn(s, generator=g, dtype=F64) for s in ((5, 4, 3), (5, 2, 3), (5, 2, 2)))
    o = plain.masked_attention(q4, k2, v2, 0.5)
    assert torch.allclose(o[:, 2:3], plain.masked_attention(q4[:, 2:3], k2[:, 1:2], v2[:, 1:2], 0.5))


def test_turned_values_depend_on_the_distance_only():
    """With one key in sight the output is the value, turned by (key position - query position)."""
    w = {"q": torch.zeros((2, 3)), "k": torch.zeros((2, 3)), "v": torch.eye(2, 3), "o": torch.eye(2),
         "q.norm": torch.ones(2), "k.norm": torch.ones(2), "sink": torch.full((1,), -1e9)}
    w = {n: t.to(F64) for n, t in w.items()}
    m = dict(heads=1, kv_heads=1, dim=2, vdim=2, scale=1.0, rot={"dims": 2, "base": 10.0}, mask={"size": 1})
    h = torch.randn((6, 3), generator=torch.Generator().manual_seed(1), dtype=F64)
    assert torch.allclose(plain.window_attention(h, w, "", m, 1e-6), h[:, :2])       # each sees itself
    m["mask"]["size"] = 2
    y = plain.window_attention(h, w, "", m, 1e-6)
    back = plain.rotate_halves(h[:5, None, :2], 2, 10.0, first=-1)[0]              # turned by -1
    u, v = h[0, :2]
    c, s = math.cos(-1.0), math.sin(-1.0)
    one_before = torch.stack([u * c - v * s, v * c + u * s])
    assert torch.allclose(back[0], one_before)
    assert torch.allclose(y[1], 0.5 * (h[1, :2] + one_before))


def test_decayed_sum_by_hand():
    q = torch.ones((3, 1, 2), dtype=F64)
    k = torch.tensor([[1.0, 0.0], [0.0, 1.0], [1.0, 1.0]], dtype=F64).reshape(3, 1, 2)
    v = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64).reshape(3, 1, 1)
    o = plain.decayed_sum(q, k, v, torch.tensor([0.5], dtype=F64))
    assert o.flatten().tolist() == [1.0, 10.5, 205.25]


def test_choice_of_experts_by_hand():
    s = torch.tensor([[0.9, 0.15, 0.6, 0.5, 0.8, 0.2]], dtype=F64)
    z = torch.log(s / (1 - s))
    none = torch.zeros(6, dtype=F64)
    idx, wt = plain.choose_experts(z, none, {"top": 2})
    assert idx.tolist() == [[0, 4]] and torch.allclose(wt, torch.tensor([[0.9, 0.8]], dtype=F64))
    # groups (0.9, 0.15), (0.6, 0.5), (0.8, 0.2): sums 1.05, 1.1, 1.0
    router = {"top": 2, "groups": {"count": 3, "keep": 1}}
    assert plain.choose_experts(z, none, router)[0].tolist() == [[2, 3]]
    router["groups"]["keep"] = 2
    assert plain.choose_experts(z, none, router)[0].tolist() == [[0, 2]]
    # a correction moves the choice and not the weights; choice scores may be negative
    corr = torch.tensor([-2.0, 0.0, -2.0, -2.0, -1.9, -2.0], dtype=F64)
    idx, wt = plain.choose_experts(z, corr, {"top": 2, "groups": {"count": 3, "keep": 1}})
    assert idx.tolist() == [[1, 0]] and torch.allclose(wt, torch.tensor([[0.15, 0.9]], dtype=F64))
    assert plain.choice_margin(z, none, {"top": 6})[0] == float("inf")
    assert plain.choice_margin(z, none, {"top": 2})[0] == pytest.approx(0.2)
    # groups of one member are ranked by it
    idx, _ = plain.choose_experts(z, none, {"top": 3, "groups": {"count": 6, "keep": 3}})
    assert idx.tolist() == [[0, 4, 2]]


def test_clamped_dense_by_hand():
    h = torch.tensor([[1.0]], dtype=F64)
    w = {"gate": torch.tensor([[3.0], [-4.0]], dtype=F64), "up": torch.tensor([[5.0], [-5.0]], dtype=F64),
         "down": torch.eye(2, dtype=F64)}
    y = plain.clamped_dense(h, w, "", {"kind": "dense", "limit": 2.0})
    s = lambda z: 1 / (1 + math.exp(-1.702 * z))
    assert y[0].tolist() == pytest.approx([2 * s(2) * 3.0, -4 * s(-4) * -1.0])   # the gate has no lower limit


def test_the_prefix_property_and_the_depth_average():
    """Logits of a position do not change when tokens follow it; every coefficient matters."""
    w = stored_values(random_weights(TINY_A, 3))
    toks = random_tokens(30, 127, 4)
    full = plain.forward(TINY_A, w, toks)
    assert torch.allclose(plain.forward(TINY_A, w, toks[:17]), full[:17], atol=1e-10)
    streams = []
    plain.forward(TINY_A, w, toks, streams=streams)
    assert len(streams) == 5
    for i in range(5):
        for j in range(i + 2):
            w2 = dict(w)
            w2[f"l{i}.dwa"] = w[f"l{i}.dwa"].clone()
            w2[f"l{i}.dwa"][j] += 0.3
            assert not torch.allclose(plain.forward(TINY_A, w2, toks), full, atol=1e-3), (i, j)
    assert torch.equal(plain.depth_average([torch.ones(2), torch.full((2,), 3.0)], torch.tensor([2.0, -1.0])),
                       torch.tensor([-1.0, -1.0]))
