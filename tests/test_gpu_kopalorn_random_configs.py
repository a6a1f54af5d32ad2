"""Kopalorn configurations drawn at random (fixed seed): layer counts and orders of the three mixers, a repeated run of layers anywhere
(or none) that runs one to three times, head counts and groupings, key and value sizes equal or not, odd ones and sizes the tensor
cores like, rotations of all or part of a map or none, windows from 1 to 300 or none, decays from zero to one, caps from 1 to 30,
routers with one to five groups of which one to all are kept or without groups, scales, top from 1 to all that can be chosen, with
and without an expert for every token, layers without a feed-forward, residual multipliers; both dtypes.  Each is run whole, with its
tail decoded and in a batch of two with unequal lengths, against the plain implementation."""
import json
import os
import random

import pytest

import citlali_b200 as cb
import plain_kopalorn as plain
import replay
from helpers import random_tokens
from kopalorn_models import attention, make_weights, mlstm, model, moe, parallel
from test_gpu_kopalorn_replay import row_error

pytestmark = pytest.mark.gpu


def draw(i):
    rng = random.Random(7100 + i)
    width = rng.choice([40, 64, 72, 100, 128])
    size = lambda: rng.choice([8, 10, 12, 16, 24, 32, 40, 64])

    def mlp():
        if rng.random() < 0.15:
            return None
        count = rng.choice([None, 1, 2, 3, 5])
        per = rng.choice([2, 3, 4])
        experts = per * (count or rng.choice([1, 2, 3]))
        groups = None if count is None else (count, rng.randint(1, count))
        reach = experts if groups is None else groups[1] * per
        return moe(experts, rng.randint(1, min(reach, 4)) if rng.random() < 0.8 else reach, rng.choice([16, 24, 40, 30]), rng.choice([None, 16, 20, 48]),
                   groups, rng.choice([None, 0.5, 1.0, 2.5]))

    layers = []
    for _ in range(rng.randint(2, 5)):
        kind = rng.choice(["attention", "mlstm", "parallel"])
        kv = rng.randint(1, 3)
        if kind == "attention":
            dim = rng.choice([8, 10, 16, 32, 48, 64])
            rot = rng.choice([None, (dim, rng.choice([10.0, 1e4])), (2, 100.0), (dim // 4 * 2, 5e5)])
            layers.append(attention(kv * rng.choice([1, 2, 3, 4]), kv, dim, 2 * dim if rng.random() < 0.5 else size(), rng.choice([0.15, 0.3, dim ** -0.5]),
                                    rng.choice([0.0, 0.2, 0.5, 0.8]), rot, rng.choice([None, 1, 7, 64, 65, 100, 300]), mlp()))
        elif kind == "mlstm":
            layers.append(mlstm(rng.randint(1, 5), size(), rng.choice([6, 16, 24, 33, 64]), rng.choice([1.0, 5.0, 15.0, 30.0]), mlp()))
        else:
            layers.append(parallel((kv * rng.choice([1, 2, 4]), kv, size(), size(), rng.choice([0.2, 0.3])),
                                   (size(), size(), [rng.choice([0.0, 0.3, 0.6, 0.9, 0.97, 0.999, 1.0]) for _ in range(rng.randint(1, 5))]), mlp()))
    loop = None
    if rng.random() < 0.8:
        start = rng.randrange(len(layers))
        loop = (start, rng.randint(start + 1, len(layers)), rng.randint(1, 3))
    return model(rng.choice([130, 256, 501]), width, rng.choice([1e-5, 1e-6]), rng.choice([0.25, 0.6, 1.0, 1.4]), loop, layers)


@pytest.mark.parametrize("i", range(14))
def test_random_configuration(i, tmp_path):
    d = draw(i)
    cfg = cb.config_from_dict(json.loads(json.dumps(d)))
    w = make_weights(cfg, 800 + i)
    path = str(tmp_path / "m")
    os.makedirs(path)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg.to_dict(), f)
    cb.write_safetensors(os.path.join(path, "model.safetensors"), lambda: iter(w.items()), metadata={"format": "pt"})
    reqs = [("a", random_tokens(d["vocab"], 150, 3 * i + 1)), ("b", random_tokens(d["vocab"], 47, 3 * i + 2))]
    want = {rid: plain.forward(cfg.to_dict(), w, toks) for rid, toks in reqs}
    # 32-bit: every position within rounding of the exact evaluation (98 % tightly: a head of a matrix memory whose result nearly
    # cancels is blown up, rounding and all, by the norm behind it).  bfloat16: a router's close call may fall the other way, and
    # every position behind it in the sequence then differs: most positions must agree and the median error must be small; each
    # bfloat16 kernel is held strictly where it is tested alone
    for dtype, tol, most in (("float32", 5e-5, 0.98), ("bfloat16", 5e-2, 0.6)):
        s = cb.InferenceSession().load_model(path, max_context=256, dtype=dtype, max_batch=2)
        for what, steps in (("whole", replay.whole(reqs)), ("tail", replay.tail(reqs, last=40)),
                            ("batched", replay.batched(reqs, [100, 20], 2))):
            got = replay.run_in_process(s, steps)
            errs = []
            for (rid, pos), row in got.items():
                errs.append(row_error(row, want[rid][pos]))
                assert errs[-1] <= 20 * tol or dtype != "float32", f"configuration {i} {what}: {rid} position {pos}: {errs[-1]:.3e}"
            good = sum(e <= tol for e in errs)
            assert good >= most * len(errs), f"configuration {i} {dtype} {what}: only {good} of {len(errs)} positions agree"
            assert sorted(errs)[len(errs) // 2] <= 0.6 * tol, f"configuration {i} {dtype} {what}: median error {sorted(errs)[len(errs) // 2]:.3e}"
