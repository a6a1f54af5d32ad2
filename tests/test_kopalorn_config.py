"""The Kopalorn configuration on the CPU: read, written back, described as data; the repeated run of layers as schedule steps with a
cache or state of their own every time and a step of its own ahead of each; constants reaching the parts; rejections that name the
key; and the plain implementation against elementary identities."""
import copy
import math

import pytest
import torch

import citlali_b200 as cb
import plain_kopalorn as plain
from citlali_b200.cache import KVRequirement, StateRequirement
from citlali_b200.engine.model import DecoderModel, cache_requirements_of
from citlali_b200.parts.base import BuildContext
from kopalorn_models import CONFIGS, config, make_weights

KINDS = {"attention": "differential_attention", "mlstm": "linear_memory", "parallel": "parallel"}


def test_round_trip_and_spec_as_data():
    for name, d in CONFIGS.items():
        cfg = config(name)
        assert cfg.to_dict() == d and cb.config_from_dict(cfg.to_dict()).to_dict() == d
        spec = cfg.to_model_spec()
        assert spec.architecture == "Kopalorn" and spec.tie_head_to_embedding is False and spec.embedding_scale is None
        assert len(spec.layers) == len(d["layers"]) + (1 if "loop" in d else 0)
        for layer, described in zip(spec.layers, d["layers"]):
            names = {"mixer_norm", "mixer", "mixer_out_norm"}
            if described["mlp"]:
                names |= {"feed_forward_norm", "feed_forward", "feed_forward_out_norm"}
            assert layer.block == "sandwich_norm" and set(layer.parts) == names
            assert layer.parts["mixer"].kind == KINDS[described["type"]]
            for n in names - {"mixer", "feed_forward"}:
                assert layer.parts[n].params["scale"] == (d["residual_mult"] if n.endswith("out_norm") else 1.0)
        names = [t.name for t in cb.expected_tensors(spec)]
        assert len(names) == len(set(names)) and {"embed", "head", "final.norm", "final.norm.b"} <= set(names)
        assert ("loop.step" in names) == ("loop" in d)


def test_the_repeated_run_and_what_a_sequence_keeps():
    order = lambda name: [s.layer for s in config(name).to_model_spec().schedule]
    assert order("A") == [0, 4, 1, 2, 4, 1, 2, 3] and order("B") == [0, 1, 2] and order("C") == [3, 0, 1, 2, 3, 0, 1, 2]
    assert order("D") == [0, 3, 1, 2, 3, 1, 2, 3, 1, 2] and order("E") == [1, 0] and order("F") == [3, 0, 3, 0, 1, 2]
    for name, d in CONFIGS.items():
        spec = config(name).to_model_spec()
        assert [i for i, _ in plain.schedule(d)] == [i for i in order(name) if i < len(d["layers"])]
        assert all(s.cache_of is None for s in spec.schedule)
        for req, i in zip(cache_requirements_of(spec), order(name)):
            if i == len(d["layers"]):
                assert req is None
                continue
            m, kind = d["layers"][i]["mixer"], d["layers"][i]["type"]
            if kind == "attention":
                assert req == (KVRequirement(m["kv_heads"], 2 * m["dim"], m["mask"]["size"] if "mask" in m else None, value_dim=m["vdim"]),)
            elif kind == "mlstm":
                h, k, v = m["heads"], m["dim"], m["vdim"]
                assert req == StateRequirement((h * k * v + h * k + h,), torch.float32)
            else:
                l, r = m["left"], m["right"]
                assert req == ((KVRequirement(l["kv_heads"], l["dim"], None, value_dim=l["vdim"]),),
                               StateRequirement((r["heads"] * r["dim"] * r["vdim"],), torch.float32))


def test_constants_reach_the_parts():
    spec = config("A").to_model_spec()
    a, m, p, last = (l.parts["mixer"].params for l in spec.layers[:4])
    assert (a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], a["diff"], a["window"], a["eps"]) == (4, 2, 16, 24, 0.3, 0.4, 9, 1e-5)
    assert (a["rot_dims"], a["rot_base"], a["rot_layout"], a["gate"]) == (8, 100.0, "pairs", "heads") and last["window"] == 1
    assert (m["heads"], m["dim"], m["vdim"], m["gate_cap"], m["norm_over"], m["act"], m["norm_eps"]) == (3, 24, 16, 6.0, "head", None, 1e-5)
    assert m["q_scale"] == 24 ** -0.5 and "decay" not in m
    l, r = p["left"].params, p["right"].params
    assert (l["heads"], l["kv_heads"], l["dim"], l["vdim"], l["scale"], l["window"], l["rot_dims"], l["biases"], l["gate"]) == (
        6, 3, 16, 8, 0.25, None, 0, True, "elements")
    assert (r["heads"], r["dim"], r["vdim"], r["decay"], r["act"], r["norm_over"]) == (3, 16, 24, [0.5, 0.9, 0.99], "silu", "row")
    assert (p["left_scale"], p["right_scale"], p["out_norms"]) == (0.5, 0.5, {"size": 64, "eps": 1e-5, "left": "l2.mix.left.out",
                                                                              "right": "l2.mix.right.out"})
    ff = spec.layers[0].parts["feed_forward"].params
    assert (ff["experts"], ff["top"], ff["intermediate_size"], ff["groups"], ff["keep_groups"], ff["weight_scale"]) == (6, 2, 32, 2, 1, 1.7)
    assert (ff["score"], ff["correction"], ff["renormalise"], ff["group_score"], ff["activation"]) == ("sigmoid", True, True, "top2_sum", "relu_squared")
    assert ff["shared"] == {"intermediate_size": 24, "weight": "sigmoid"} and spec.layers[1].parts["feed_forward"].params["shared"] is None
    shapes = {t.name: tuple(t.shape) for t in cb.expected_tensors(spec)}
    assert shapes["l0.mix.q"] == (128, 64) and shapes["l0.mix.k"] == (64, 64) and shapes["l0.mix.v"] == (48, 64) and shapes["l0.mix.g"] == (4, 64)
    assert shapes["l0.mix.o"] == (64, 96) and shapes["l0.mix.lq1"] == (16,) and shapes["l1.mix.i"] == (3, 64) and shapes["l1.mix.norm"] == (48,)
    assert shapes["l2.mix.left.q.b"] == (96,) and shapes["l2.mix.left.g"] == (48, 64) and shapes["l2.mix.right.norm"] == (72,)
    assert shapes["l2.mix.right.out"] == (64,) and shapes["l0.mlp.e5.up"] == (32, 64) and shapes["l0.mlp.correction"] == (6,)
    assert shapes["l0.mlp.shared.sg"] == (1, 64) and shapes["loop.step"] == (2, 64) and shapes["l3.norm2b.b"] == (64,)
    assert not ({"l2.norm2", "l0.mix.q.b", "l2.mix.right.q.b", "l0.mlp.e0.gate", "l1.mlp.shared.up", "l2.mlp.router"} & set(shapes))
    plain_routers = [l.parts["feed_forward"].params for l in config("F").to_model_spec().layers if "feed_forward" in l.parts]
    assert plain_routers[-1]["groups"] is None and plain_routers[-1]["weight_scale"] == 0.8 and plain_routers[0]["weight_scale"] is None


def test_sizes_that_may_be_left_out():
    d = copy.deepcopy(CONFIGS["A"])
    del d["layers"][0]["mixer"]["kv_heads"], d["layers"][0]["mixer"]["vdim"], d["layers"][1]["mixer"]["vdim"], d["residual_mult"]
    spec = cb.config_from_dict(d).to_model_spec()
    shapes = {t.name: tuple(t.shape) for t in cb.expected_tensors(spec)}
    assert shapes["l0.mix.k"] == (128, 64) and shapes["l0.mix.v"] == (64, 64) and shapes["l1.mix.v"] == (72, 64)
    assert spec.layers[0].parts["mixer_out_norm"].params["scale"] == 1.0


def test_models_name_their_kernel_sources():
    named = {dt: set(DecoderModel(config("C").to_model_spec(), BuildContext(torch.device("cpu"), dt)).kernel_sources())
             for dt in (torch.float32, torch.bfloat16)}
    assert {"linear_memory", "differential", "heads_prepare", "sublayer", "moe", "activations"} <= named[torch.float32] & named[torch.bfloat16]
    assert "attention_prefill_tc" in named[torch.bfloat16] and "window_attention" in named[torch.float32]
    assert "delta_rule" not in named[torch.float32] | named[torch.bfloat16]


@pytest.mark.parametrize("edit,match", [
    (lambda d: d.pop("vocab"), "vocab"),
    (lambda d: d.pop("norm"), "eps"),
    (lambda d: d.update(layers=[]), "layers"),
    (lambda d: d["layers"][0].update(type="conv"), "type 'conv'"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda d: d["layers"][1]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda d: d["layers"][1]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=1), "key a head"),
    (lambda d: d["layers"][2]["mixer"].pop("left"), "left"),
    (lambda d: d["layers"][2]["mixer"]["left"].pop("scale"), "scale"),
    (lambda d: d["layers"][2]["mixer"]["right"].update(decay=[0.5, 0.5]), "decay"),
    (lambda d: d["layers"][2]["mixer"]["right"].update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=4), "top"),
    (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=3), "keep"),
    (lambda d: d["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda d: d["loop"].update(stop=5), "loop"),
    (lambda d: d["loop"].update(times=0), "times"),
])
def test_rejections_name_the_key(edit, match):
    d = copy.deepcopy(CONFIGS["A"])
    edit(d)
    with pytest.raises(cb.CitlaliError, match=match):
        cb.config_from_dict(d)


# ---- the plain implementation against elementary identities ---------------------------------------------------------------

def test_plain_norms_rotations_and_windows():
    x = torch.randn(5, 12, dtype=torch.float64)
    y = plain.layer_norm(x, torch.ones(12), torch.full((12,), 3.0), 0.0)
    assert torch.allclose(y.mean(-1), torch.full((5,), 3.0, dtype=torch.float64)) and torch.allclose(y.var(-1, unbiased=False), torch.ones(5, dtype=torch.float64))
    r = plain.rotate_pairs(x.view(5, 1, 12), range(5), 8, 100.0)[:, 0]
    assert torch.allclose(r[:, 8:], x[:, 8:]) and torch.allclose(r[0], x[0]) and torch.allclose((r ** 2).sum(-1), (x ** 2).sum(-1))
    a = 100.0 ** -0.25                                                      # pair 1 at position 1
    assert abs(float(r[1, 2]) - (float(x[1, 2]) * math.cos(a) - float(x[1, 3]) * math.sin(a))) < 1e-12
    see = plain.visible(4, 3)
    assert bool(see[3, 1]) and not bool(see[3, 0]) and not bool(see[1, 2])


def test_plain_memories():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(9, n, generator=g, dtype=torch.float64) for n in (4, 4, 3))
    one = plain.decayed_sums(q, k, v, 0.5)
    want = torch.stack([sum(0.5 ** (t - s) * float(q[t] @ k[s]) * v[s] for s in range(t + 1)) for t in range(9)])
    assert torch.allclose(one, want)
    # the running maximum changes nothing but the floor: without it the same ratio in logs
    i, f = torch.randn(9, generator=g, dtype=torch.float64) + 3.0, -torch.rand(9, generator=g, dtype=torch.float64)
    got = plain.stabilised_memory(q, k, v, i, f)
    for t in range(9):
        w = [math.exp(float(i[s] + f[s + 1:t + 1].sum())) for s in range(t + 1)]
        num = sum(w[s] * float(q[t] @ k[s]) * v[s] for s in range(t + 1))
        den = max(abs(sum(w[s] * float(q[t] @ k[s]) for s in range(t + 1))), 1.0)      # exp(-m) times exp(m)
        assert torch.allclose(got[t], num / den, rtol=1e-4)


def test_plain_router_and_causality():
    z = torch.tensor([4.0, -3.0, 0.5, 0.4, 3.0, -4.0], dtype=torch.float64)
    none = torch.zeros(6)
    # the second group's two best sum to more than any other's, though the best single expert is in the first
    picked = plain.route_row(z, none, {"top": 2, "groups": {"count": 3, "keep": 1}, "scale": 2.0})
    assert set(picked) == {2, 3} and abs(sum(picked.values()) - 2.0) < 1e-12
    assert set(plain.route_row(z, none, {"top": 2})) == {0, 4}
    # all choice scores below zero: a closed group is still never chosen
    low = torch.full((6,), -5.0)
    low[2] = -1.0
    assert set(plain.route_row(z, low, {"top": 2, "groups": {"count": 3, "keep": 1}})) == {2, 3}
    cfg, w = CONFIGS["A"], make_weights(config("A"), 3)
    toks = [5, 9, 100, 3, 77, 8, 1, 150, 60, 2, 31, 44, 12, 199, 0, 6]
    full = plain.forward(cfg, w, toks)
    assert torch.allclose(plain.forward(cfg, w, toks[:9]), full[:9], atol=1e-9)
