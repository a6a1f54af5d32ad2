"""The Nomutar configuration on the CPU: read, written back, described as data; the repeated run of layers as schedule steps
with a cache of their own every time; constants reaching the parts; the residual kept divided by its multiplier; scaled
frequencies; rejections that name the key; and the plain implementation against elementary identities."""
import copy
import math

import pytest
import torch

import citlali_b200 as cb
import plain_nomutar as plain
from citlali_b200.cache import KVRequirement, StateRequirement
from citlali_b200.engine.model import cache_requirements_of
from citlali_b200.parts.rotary import rotation_table
from nomutar_models import CONFIGS, config, make_weights


def test_round_trip_and_spec_as_data():
    for name, d in CONFIGS.items():
        cfg = config(name)
        assert cb.config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
        spec = cfg.to_model_spec()
        assert spec.architecture == "Nomutar" and spec.tie_head_to_embedding is False and spec.logit_softcap == d.get("logit_softcap")
        assert len(spec.layers) == len(d["layers"])
        for layer, described in zip(spec.layers, d["layers"]):
            assert layer.block == "parallel_residual"
            assert set(layer.parts) == {"norm", "mixer"} | ({"feed_forward"} if described["mlp"] else set()) | ({"mixer_input"} if "canon" in d else set())
            assert layer.parts["mixer"].kind == "window_attention" and layer.parts["norm"].kind == "grouped_rms_norm"
            assert layer.parts["norm"].params["groups"] == d["norm"]["groups"]
        names = [t.name for t in cb.expected_tensors(spec)]
        assert len(names) == len(set(names)) and {"embed", "head", "final.norm"} <= set(names)
        assert ("bigram" in names) == ("bigram" in d["embedding"]) and ("l0.canon1" in names) == ("canon" in d)


def test_the_repeated_run_and_what_a_sequence_keeps():
    order = lambda name: [s.layer for s in config(name).to_model_spec().schedule]
    assert order("P") == [0, 1, 2, 1, 2, 3] and order("Q") == [0, 1, 2] and order("R") == [0, 1, 2, 0, 1, 2]
    assert order("S") == [0, 1, 2, 1, 2, 1, 2] and order("U") == [0, 0, 1]
    for name, d in CONFIGS.items():
        spec = config(name).to_model_spec()
        assert plain.run_order(d) == order(name) and all(s.cache_of is None for s in spec.schedule)
        reqs = cache_requirements_of(spec)
        assert len(reqs) == len(order(name)) + (1 if "bigram" in d["embedding"] else 0)
        for req, i in zip(reqs, order(name)):
            m = d["layers"][i]["mixer"]
            kv = KVRequirement(m["kv_heads"], m["dim"], m["mask"]["size"] if "mask" in m else None, value_dim=m["vdim"])
            if "canon" not in d:
                assert req == (kv,)
                continue
            taps = d["canon"]["taps"]
            assert req == ((kv,), StateRequirement(((taps - 1) * d["width"],), torch.float32) if taps > 1 else None)
        if "bigram" in d["embedding"]:
            assert reqs[-1] == StateRequirement((1,), torch.int32)


def test_constants_reach_the_parts():
    spec = config("P").to_model_spec()
    a, b, c, last = (l.parts["mixer"].params for l in spec.layers)
    assert (a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], a["softcap"], a["window"]) == (4, 2, 16, 24, 0.25, 3.0, 9)
    assert (a["rot_dims"], a["rot_base"], a["rot_layout"], a["value_rot_base"], a["sink"], a["biases"]) == (8, 100.0, "halves", 100.0, "heads", False)
    assert a["rot_scaling"] == {"kind": "wavelength", "factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}
    assert (a["qk_norm_eps"], a["qk_norm_over"], a["names"]) == (1e-5, "projection", {"q_norm": "l0.mix.q.norm", "k_norm": "l0.mix.k.norm"})
    assert (b["qk_norm_eps"], b["rot_layout"], b["value_rot_base"], b["sink"], b["biases"], b["window"]) == (None, "pairs", None, 0.0, True, 65)
    assert b["rot_scaling"] == {"kind": "ramp", "factor": 4.0, "original": 128, "fast": 8.0, "slow": 1.0}
    assert (c["qk_norm_eps"], c["rot_layout"], c["value_rot_base"], c["sink"], c["biases"], c["window"], c["softcap"], c["rot_scaling"]) == (
        1e-5, "halves", None, None, False, None, None, None)
    assert last["window"] == 1 and last["rot_scaling"] is None
    ff = spec.layers[0].parts["feed_forward"]
    assert ff.kind == "routed_experts" and (ff.params["experts"], ff.params["top"], ff.params["intermediate_size"]) == (6, 2, 32)
    assert (ff.params["score"], ff.params["router_bias"], ff.params["shared"]) == ("softmax_chosen", True, {"intermediate_size": 24, "weight": "sigmoid"})
    assert spec.layers[3].parts["feed_forward"].params["shared"] is None
    assert spec.layers[0].parts["mixer_input"].params == {"hidden_size": 64, "taps": 4}
    shapes = {t.name: tuple(t.shape) for t in cb.expected_tensors(spec)}
    assert shapes["bigram"] == (62, 64) and shapes["l0.canon1"] == (64, 4) and shapes["l0.mix.q.norm"] == (64,) and shapes["l0.mix.k.norm"] == (32,)
    assert shapes["l0.mix.sink"] == (4,) and shapes["l1.mix.v.b"] == (8,) and shapes["l2.mix.o"] == (64, 240) and shapes["l0.mlp.shared.sg"] == (1, 64)
    assert not ({"l1.mix.sink", "l1.mix.q.norm", "l0.mix.q.b", "l2.mlp.gate", "l3.mlp.shared.gate", "l0.mix.o.b"} & set(shapes))


def test_the_residual_is_kept_divided_by_its_multiplier():
    """With y = x / m the sums need no factor: the norms take eps / m^2, the embedding's two rows enter divided by m."""
    for name, d in CONFIGS.items():
        m, spec = d["residual_mult"], config(name).to_model_spec()
        assert spec.embedding_scale == d["embedding"]["scale"] / m
        for p in [spec.final_norm] + [l.parts["norm"] for l in spec.layers]:
            assert p.params["eps"] == d["norm"]["eps"] / m ** 2
        if spec.embedding_addition is not None:
            assert spec.embedding_addition.params["pair_scale"] == 1.0 / m
        x = torch.randn(3, d["width"], dtype=torch.float64) * 0.01            # small rows: eps matters
        g = torch.ones(d["width"])
        assert torch.allclose(plain.group_norm(x / m, g, d["norm"]["groups"], d["norm"]["eps"] / m ** 2),
                              plain.group_norm(x, g, d["norm"]["groups"], d["norm"]["eps"]), rtol=1e-12)


@pytest.mark.parametrize("dims,base,scaling", [
    (32, 10000.0, dict(kind="wavelength", factor=8.0, low=1.0, high=4.0, original=128)),
    (48, 500000.0, dict(kind="wavelength", factor=4.0, low=0.5, high=32.0, original=1024)),
    (10, 7.0, dict(kind="wavelength", factor=2.0, low=1.0, high=2.0, original=4)),
    (64, 10000.0, dict(kind="ramp", factor=4.0, original=256, fast=32.0, slow=1.0)),
    (24, 100.0, dict(kind="ramp", factor=16.0, original=4096, fast=32.0, slow=1.0)),
    (6, 50.0, dict(kind="ramp", factor=2.0, original=16, fast=64.0, slow=0.01)),
    (128, 150000.0, dict(kind="ramp", factor=40.0, original=8192, fast=16.0, slow=2.0)),
])
def test_scaled_frequencies(dims, base, scaling):
    got, amplitude = rotation_table(dims, base, scaling)
    args = {k: v for k, v in scaling.items() if k != "kind"}
    plain_f = plain.base_frequencies(dims, base)
    if scaling["kind"] == "wavelength":
        want, amp = plain.llama3_frequencies(plain_f, **args), 1.0
    else:
        want, amp = plain.yarn_frequencies(plain_f, dims, base, **args)
    assert got.dtype == torch.float32 and torch.allclose(got.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6, atol=0.0)
    assert amplitude == amp
    # the ends of the stretch: nothing is raised, nothing falls below f / factor
    ratio = got.double() / torch.tensor(plain_f, dtype=torch.float64)
    assert float(ratio.max()) <= 1.0 + 1e-6 and float(ratio.min()) >= 1.0 / scaling["factor"] - 1e-6
    assert rotation_table(dims, base)[1] == 1.0


@pytest.mark.parametrize("edit,match", [
    (lambda d: d.pop("vocab"), "vocab"),
    (lambda d: d.pop("norm"), "eps"),
    (lambda d: d["norm"].update(groups=3), "groups"),
    (lambda d: d.update(residual_mult=0.0), "residual_mult"),
    (lambda d: d["embedding"]["bigram"].pop("buckets"), "buckets"),
    (lambda d: d["embedding"]["bigram"].update(mul_cur=-1), "mul_cur"),
    (lambda d: d["canon"].update(taps=0), "taps"),
    (lambda d: d["canon"].update(taps=17), "taps"),
    (lambda d: d["layers"][0].update(type="conv"), "type 'conv'"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"].pop("rot"), "dims"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"].update(vdim=23), "vdim"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][0]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("low"), "low"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(high=1.0), "high"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda d: d["layers"][2]["mixer"]["rot"].update(scaling={"factor": 2.0}), "attention_3"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda d: d["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda d: d["layers"][1]["mlp"].update(kind="sparse"), "kind"),
    (lambda d: d["loop"].update(stop=5), "loop"),
    (lambda d: d["loop"].update(times=0), "times"),
    (lambda d: d.update(logit_softcap=0.0), "logit_softcap"),
])
def test_rejections_name_the_key(edit, match):
    d = copy.deepcopy(CONFIGS["P"])
    edit(d)
    with pytest.raises(cb.CitlaliError, match=match):
        cb.config_from_dict(d)


# ---- the plain implementation against elementary identities ---------------------------------------------------------------

def test_plain_norms_convolution_and_pairs():
    x = torch.randn(5, 12, dtype=torch.float64)
    y = plain.group_norm(x, torch.ones(12), 3, 0.0)
    assert torch.allclose((y.view(5, 3, 4) ** 2).mean(-1), torch.ones(5, 3, dtype=torch.float64))
    assert torch.allclose(plain.group_norm(x, torch.full((12,), 2.0), 1, 0.0), 2.0 * plain.rms(x, 0.0))
    w = torch.zeros(12, 3)
    w[:, 2], w[:, 0] = 1.0, 10.0                                        # the token itself, and ten times the one two back
    c = plain.causal_conv(x, w)
    assert torch.allclose(c[:2], x[:2]) and torch.allclose(c[2:], x[2:] + 10.0 * x[:-2])
    assert plain.bigram_rows([5, 7, 7], 3, 10, 11) == [11, (15 + 70) % 11, (21 + 70) % 11]
    assert abs(float(plain.soft_cap(torch.tensor(1e6, dtype=torch.float64), 7.0)) - 7.0) < 1e-9


def test_plain_rotations_and_sinks():
    x = torch.randn(6, 3, 10, dtype=torch.float64)
    f = plain.base_frequencies(8, 100.0)
    for layout, a, b in (("halves", 1, 5), ("pairs", 2, 3)):
        r = plain.rotate(x, range(6), f, layout)
        assert torch.allclose(r[..., 8:], x[..., 8:]) and torch.allclose(r[0], x[0])
        assert torch.allclose((r[..., :8] ** 2).sum(-1), (x[..., :8] ** 2).sum(-1))
        ang = 100.0 ** (-0.25)                                          # pair 1 at position 1
        assert abs(float(r[1, 0, a]) - (float(x[1, 0, a]) * math.cos(ang) - float(x[1, 0, b]) * math.sin(ang))) < 1e-12
        assert torch.allclose(plain.rotate(r, range(6), f, layout, sign=-1.0), x)
        assert torch.allclose(plain.rotate(x, range(6), f, layout, amplitude=2.0)[..., :8], 2.0 * r[..., :8])
    s = torch.randn(4, 4, dtype=torch.float64)
    see = plain.visible(4, 3)
    assert bool(see[3, 1]) and not bool(see[3, 0]) and not bool(see[1, 2])
    p = plain.weights_with_sink(s, see, 0.0)
    e = torch.exp(s) * see
    assert torch.allclose(p, e / (1.0 + e.sum(-1, keepdim=True)))
    assert torch.allclose(plain.weights_with_sink(s, see, None).sum(-1), torch.ones(4, dtype=torch.float64))


def test_plain_router_and_causality():
    cfg, w = CONFIGS["P"], make_weights(config("P"), 3)
    h = torch.randn(7, 64, dtype=torch.float64)
    weights, chosen, margin = plain.route(h, w, "l0.mlp", cfg["layers"][0]["mlp"]["router"])
    assert bool(((weights > 0).sum(-1) == 2).all()) and torch.allclose(weights.sum(-1), torch.ones(7, dtype=torch.float64)) and bool((margin >= 0).all())
    toks = [5, 9, 100, 3, 77, 8, 1, 150, 60, 2, 31, 44, 12, 199, 0, 6]
    full = plain.forward(cfg, w, toks)
    assert torch.allclose(plain.forward(cfg, w, toks[:9]), full[:9], atol=1e-9)
    assert bool((full.abs() < cfg["logit_softcap"]).all())
