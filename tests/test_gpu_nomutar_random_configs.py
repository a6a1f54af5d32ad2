"""Nomutar configurations drawn at random (fixed seed): layer counts and orders of the three mixers, a repeated run of layers
anywhere (or none) that runs one to three times, head counts and groupings, key and value sizes equal or not, odd ones and
sizes the tensor cores like, rotations of all or part of a head with and without scaled frequencies, windows from 1 to 300 or
none, caps from 2 to 50 or none, norms over one to many parts, convolutions of one to five taps or none, pair tables, residual
multipliers, dense and routed feed-forwards with and without an expert for every token, top from 1 to all experts, layers
without a feed-forward; both dtypes.  Each is run whole, with its tail decoded and in a batch of two with unequal lengths,
against the plain implementation."""
import json
import os
import random

import pytest

import citlali_b200 as cb
import plain_nomutar as plain
import replay
from helpers import random_tokens
from nomutar_models import dense, make_weights, mixer, model, moe, ramp, wavelength

pytestmark = pytest.mark.gpu


def draw(i):
    rng = random.Random(9300 + i)
    width = rng.choice([40, 64, 72, 128])

    def mlp():
        kind = rng.random()
        if kind < 0.15:
            return None
        if kind < 0.5:
            return dense(rng.choice([24, 100, 128, 200]))
        experts = rng.choice([2, 3, 4, 8, 12, 16])
        return moe(experts, rng.randint(1, min(experts, 4)) if rng.random() < 0.8 else experts, rng.choice([16, 24, 40, 64]),
                   rng.choice([None, 16, 20, 48]))

    layers = []
    for _ in range(rng.randint(2, 5)):
        kind = rng.choice(["attention", "attention", "attention_2", "attention_2", "attention_3"])
        kv = rng.randint(1, 3)
        dim = rng.choice([8, 12, 16, 32, 48, 64, 80, 128])
        vdim = dim if rng.random() < 0.5 else rng.choice([8, 20, 24, 64, 104])
        dims = dim if rng.random() < 0.5 else rng.choice([2, 4, 8])
        base = rng.choice([10.0, 100.0, 10000.0, 500000.0])
        scaling = None
        if kind == "attention" and rng.random() < 0.7:
            low = rng.choice([0.5, 1.0, 2.0])
            scaling = wavelength(rng.choice([2.0, 8.0]), low, low * rng.choice([2.0, 4.0]), rng.choice([16, 64, 8192]))
        if kind == "attention_2" and rng.random() < 0.7:
            scaling = ramp(rng.choice([2.0, 16.0]), rng.choice([32, 256, 4096]), rng.choice([8.0, 32.0]), rng.choice([0.5, 1.0]))
        capped = kind != "attention_3"
        layers.append(mixer(kind, kv * rng.choice([1, 1, 2, 3, 4]), kv, dim, vdim, rng.choice([0.1, 0.2, dim ** -0.5]), (dims, base), mlp(),
                            softcap=rng.choice([None, 2.0, 5.0, 20.0, 50.0]) if capped else None,
                            window=rng.choice([None, 1, 7, 64, 65, 100, 300]) if capped else None, scaling=scaling))
    loop = None
    if rng.random() < 0.8:
        start = rng.randrange(len(layers))
        loop = (start, rng.randint(start + 1, len(layers)), rng.randint(1, 3))
    groups = rng.choice([1, 2, 4, 8])
    bigram = None if rng.random() < 0.2 else (rng.choice([5, 64, 701]), rng.randrange(2000), rng.randrange(1, 2000))
    return model(rng.choice([130, 256, 500]), width, rng.choice([1e-5, 1e-6]), groups, rng.choice([0.25, 0.6, 1.0, 1.4]), rng.choice([1.0, 4.0]),
                 bigram, rng.choice([None, 1, 2, 3, 4, 5]), rng.choice([None, 10.0, 30.0]), loop, layers)


@pytest.mark.parametrize("i", range(12))
def test_random_configuration(i, tmp_path):
    d = draw(i)
    cfg = cb.config_from_dict(json.loads(json.dumps(d)))
    w = make_weights(cfg, 900 + i)
    path = str(tmp_path / "m")
    os.makedirs(path)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg.to_dict(), f)
    cb.write_safetensors(os.path.join(path, "model.safetensors"), lambda: iter(w.items()), metadata={"format": "pt"})
    reqs = [("a", random_tokens(d["vocab"], 150, 3 * i + 1)), ("b", random_tokens(d["vocab"], 47, 3 * i + 2))]
    want = {rid: plain.forward(cfg.to_dict(), w, toks) for rid, toks in reqs}
    # 32-bit: every position within rounding of the exact evaluation.  bfloat16: a router's close call may fall the other
    # way, and every position behind it in the sequence then differs: most positions must agree and the median error must be
    # small; each bfloat16 kernel is held strictly where it is tested alone
    for dtype, tol, most in (("float32", 2e-5, 1.0), ("bfloat16", 5e-2, 0.6)):
        s = cb.InferenceSession().load_model(path, max_context=256, dtype=dtype, max_batch=2)
        for what, steps in (("whole", replay.whole(reqs)), ("tail", replay.tail(reqs, last=40)),
                            ("batched", replay.batched(reqs, [100, 20], 2))):
            got = replay.run_in_process(s, steps)
            good, errs = 0, []
            for (rid, pos), row in got.items():
                ref = want[rid][pos]
                diff = row.double() - ref
                # root mean square over the vocabulary, means taken off, relative to the logits' own spread
                err = float((diff - diff.mean()).pow(2).mean().sqrt() / (ref - ref.mean()).pow(2).mean().sqrt())
                errs.append(err)
                if err <= tol:
                    good += 1
                else:
                    assert dtype != "float32", f"configuration {i} {what}: {rid} position {pos}: {err:.3e}"
            assert good >= most * len(got), f"configuration {i} {dtype} {what}: only {good} of {len(got)} positions agree"
            assert sorted(errs)[len(errs) // 2] <= 0.6 * tol, f"configuration {i} {dtype} {what}: median error {sorted(errs)[len(errs) // 2]:.3e}"
