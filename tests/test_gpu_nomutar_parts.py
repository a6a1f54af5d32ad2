"""Each mechanism of the Nomutar design alone, built through the registries at sizes no model uses, against the plain
implementation: the three mixers (whole, token by token, in portions and in batches through one cache; 32-bit bitwise equal
however a sequence is cut); a key that stands out just inside and just outside windows, at page borders, in prompts and in
decoding, for each of them; a far key among hundreds; sinks that take most of the weight, a number a head; values whose
rotation carries the result; the pairing and the stretch of the rotations; norms over whole projections; the norm over parts
of a row with the convolution behind it (every way of cutting, slots used again, long prompts); the embedding of pairs; the
router whose bias chooses and whose weights are a softmax over the chosen; experts with a weighted one for every token; the
block."""
import pytest
import torch

import citlali_b200 as cb
import plain_nomutar as plain
from citlali_b200 import ops
from citlali_b200.config.spec import LayerSpec, PartSpec
from citlali_b200.engine.step import StepEntry, pack_step
from citlali_b200.parts.base import build_part, part_class
from nomutar_models import draw_tensor, mixer, model, ramp, wavelength
from test_gpu_pivavik_parts import DEV, DTYPES, Harness, close, ctx_for, every_way, handles, inputs

pytestmark = pytest.mark.gpu
EPS = 1e-5


def draw(specs, seed):
    g = torch.Generator().manual_seed(seed)
    return {s.name: draw_tensor(s.name, tuple(s.shape), torch.randn(tuple(s.shape), generator=g)).to(torch.bfloat16) for s in specs}


def mixer_params(layer, hidden):
    """The part parameters a model's configuration gives this layer, under the prefix 'm'."""
    cfg = cb.config_from_dict(model(64, hidden, EPS, 1, 1.0, 1.0, None, None, None, None, [layer]))
    spec = cfg.to_model_spec().layers[0].parts["mixer"]
    assert spec.kind == "window_attention"
    return dict(spec.params, names={"q_norm": "m.q.norm", "k_norm": "m.k.norm"})


def harness(layer, hidden, dtype, weights=None, seed=3, **kw):
    params = mixer_params(layer, hidden)
    part = build_part("mixer", PartSpec("window_attention", params, "m"))
    return Harness("window_attention", params, dtype, weights=weights if weights is not None else draw(part.tensor_specs(), seed), **kw)


A, B, C = "attention", "attention_2", "attention_3"
MIXERS = [
    (40, mixer(A, 4, 2, 16, 24, 0.25, (8, 100.0), None, softcap=3.0, window=9, scaling=wavelength(8.0, 1.0, 4.0, 64))),
    (48, mixer(A, 3, 3, 20, 12, 0.3, (20, 1000.0), None, softcap=30.0, window=65)),              # no tensor-core sizes, value pairs 6
    (64, mixer(A, 8, 1, 64, 64, 0.125, (32, 50.0), None, softcap=5.0, window=130, scaling=wavelength(2.0, 0.5, 16.0, 4096))),
    (24, mixer(A, 2, 2, 14, 10, 0.3, (14, 10.0), None, window=1)),                               # single pieces, no cap, itself alone
    (32, mixer(A, 4, 4, 24, 48, 0.2, (24, 500.0), None, softcap=8.0)),                           # no window
    (40, mixer(B, 4, 2, 24, 16, 0.25, (24, 100.0), None, softcap=3.0, window=64, scaling=ramp(8.0, 64, 8.0, 1.0))),
    (32, mixer(B, 6, 3, 40, 40, 0.15, (12, 5000.0), None, softcap=40.0, window=33, scaling=ramp(2.0, 1024, 32.0, 1.0))),
    (56, mixer(B, 16, 2, 128, 128, 0.09, (128, 10000.0), None, window=100)),
    (24, mixer(B, 3, 1, 10, 6, 0.3, (6, 30.0), None, softcap=6.0)),
    (40, mixer(C, 4, 2, 16, 40, 0.3, (16, 100.0), None)),
    (64, mixer(C, 4, 1, 32, 32, 0.2, (8, 10000.0), None)),
    (32, mixer(C, 5, 5, 12, 20, 0.3, (4, 20.0), None)),
    (48, mixer(C, 2, 1, 256, 136, 0.06, (256, 1e6), None)),                                      # the widest tiles
    (48, mixer(C, 32, 2, 64, 64, 0.125, (64, 1e4), None)),                                       # sixteen query heads a key head
    # heads of 128: the prompt kernel with its tiles in tensor memory, with scores under a cap that zero serves as a reference
    # for, under one too wide for that, without a cap, and with an odd number of query heads a key head
    (64, mixer(A, 8, 2, 128, 128, 0.09, (64, 50.0), None, softcap=20.0, window=130, scaling=wavelength(2.0, 0.5, 16.0, 4096))),
    (32, mixer(A, 4, 2, 128, 128, 0.2, (128, 500.0), None, softcap=90.0)),
    (32, mixer(A, 3, 1, 128, 128, 0.09, (32, 100.0), None, window=70)),
    (40, mixer(C, 4, 2, 128, 128, 0.15, (128, 1e4), None)),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,layer", MIXERS)
def test_mixers(hidden, layer, dtype):
    hs = harness(layer, hidden, dtype)
    fn = lambda h: plain.attention(h, hs.weights, "m", layer["type"], layer["mixer"], EPS)
    every_way(hs, fn, inputs(150, hidden, 3), inputs(37, hidden, 4), dtype)


def changed(layer, **change):
    m = dict(layer["mixer"], **change)
    return {"type": layer["type"], "mixer": m, "mlp": None}


@pytest.mark.parametrize("which,drop", [(0, "softcap"), (0, "mask"), (0, "scaling"), (0, "sink"), (0, "value_rot_base"), (0, "halves"),
                                        (0, "whole"), (5, "softcap"), (5, "scaling"), (5, "sink"), (5, "biases"), (5, "pairs"), (9, "halves"),
                                        (9, "whole")])
def test_each_mechanism_matters(which, drop):
    """Switching one of them off, or to the other form, changes the mixer's output: none is silently dropped on the way."""
    hidden, layer = MIXERS[which]
    base = harness(layer, hidden, torch.float32)
    h = inputs(100, hidden, 8)
    full = base.run({"a": h}, [{"a": 100}])["a"]
    p = mixer_params(layer, hidden)
    w = dict(base.weights)
    edit = {"softcap": {"softcap": None}, "mask": {"window": None}, "scaling": {"rot_scaling": None}, "sink": {"sink": None},
            "value_rot_base": {"value_rot_base": None}, "biases": {"biases": False}, "halves": {"rot_layout": "pairs", "value_rot_layout": "halves"},
            "pairs": {"rot_layout": "halves"}, "whole": {"qk_norm_eps": None}}[drop]
    other = Harness("window_attention", dict(p, **edit), torch.float32, weights=w).run({"a": h}, [{"a": 100}])["a"]
    assert float((other - full).abs().max()) > 1e-2 * float(full.abs().max()), drop


def test_values_in_neighbouring_pairs():
    """The other layout of the values' pairs, against the plain rotation: both kernels (a prompt and single tokens)."""
    hidden, layer = MIXERS[2]
    p = dict(mixer_params(layer, hidden), value_rot_layout="pairs", sink=None, window=None, softcap=None, qk_norm_eps=None, rot_dims=0)
    for dtype in DTYPES:
        hs = Harness("window_attention", p, dtype, weights=harness(layer, hidden, dtype).weights)
        h, m, w = inputs(140, hidden, 5), layer["mixer"], hs.weights
        T, H, G, D, V = 140, m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        q, k, v = ((h @ w["m." + n].double().T).view(T, x, y) for n, x, y in (("q", H, D), ("k", G, D), ("v", G, V)))
        f = plain.base_frequencies(V, m["rot"]["base"])
        v = plain.rotate(v, range(T), f, "pairs")
        o = torch.stack([plain.weights_with_sink(q[:, i] @ k[:, i // (H // G)].T * m["scale"], plain.visible(T), None) @ v[:, i // (H // G)]
                         for i in range(H)], 1)
        want = plain.rotate(o, range(T), f, "pairs", sign=-1.0).reshape(T, H * V) @ w["m.o"].double().T
        for portions in ([{"a": T}], [{"a": 70}] + [{"a": 1}] * 70):
            close(hs.run({"a": h}, portions)["a"], want, dtype, f"{dtype} neighbouring pairs of values")


def standing_out(kind, d, window, cap, sink=None):
    """Queries, keys and values are the inputs themselves (normed where the mixer norms them), queries and keys do not turn."""
    layer = mixer(kind, 1, 1, d, d, 1.0, (0, 1e30), None, softcap=cap, window=window)     # (values hardly turn, but the first pair)
    eye, zero = torch.eye(d), torch.zeros(d)
    w = {"m.q": eye, "m.k": eye, "m.v": eye, "m.o": eye}
    if kind == B:
        w.update({"m.q.b": zero, "m.k.b": zero, "m.v.b": zero})
    else:
        w.update({"m.q.norm": torch.ones(d), "m.k.norm": torch.ones(d)})
    if kind == A:
        w["m.sink"] = torch.tensor([-20.0 if sink is None else sink])
    return layer, {k: v.to(torch.bfloat16) for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode_from", [None, 40])
@pytest.mark.parametrize("kind,window", [(A, 9), (A, 64), (A, 65), (A, 130), (A, 1), (B, 9), (B, 64), (B, 65), (B, 130), (B, 1), (C, None)])
def test_window_edges_with_one_key_that_stands_out(kind, window, decode_from, dtype):
    """One key's score is above the others' by twelve or more, so that a row returns that token's value (its second element is
    the mark) while it is inside the window: the row at distance window - 1 has it, the next one has lost it; over page
    borders; in prompts and in decoding."""
    d, T = 16, 210
    layer, weights = standing_out(kind, d, window, 60.0 if kind != C else None)
    for special in (0, 1, 63, 64, 100):
        g = torch.Generator().manual_seed(special)
        h = 0.02 * torch.randn(T, d, generator=g)
        h[:, 0] += 1.0
        h[special] = 0.0
        if kind == B:
            h[special, 0], h[special, 1] = 20.0, 16.0       # a long key: its capped score is 19 where an ordinary one's is 1
        else:                                               # all keys are normed: it stands out along an axis that the norm's
            h[:, 1] += 0.25                                 # weight makes count twelve times, where every query has a part
            h[special, 0], h[special, 1] = 1.0, 0.9
            gain = torch.ones(d)
            gain[1] = 12.0
            weights["m.k.norm"] = gain.to(torch.bfloat16)
        h = h.to(torch.bfloat16).double()
        m = layer["mixer"]
        hs = harness(layer, d, dtype, weights=weights)
        portions = [{"a": T}] if decode_from is None else [{"a": decode_from}] + [{"a": 1}] * (T - decode_from)
        got = hs.run({"a": h}, portions)["a"]
        want = plain.attention(h, weights, "m", kind, m, EPS)
        allowed = (1e-4 if dtype == torch.float32 else 0.03) * want.abs().amax(-1, keepdim=True).clamp(min=1.0)
        assert bool(((got - want).abs() <= allowed).all()), (kind, window, special)
        see = plain.visible(T, window)
        for i in range(special + 1, T):                     # the test's point: the special key decides the row
            if bool(see[i, special]):
                assert abs(float(want[i][1] - h[special, 1])) < 0.1 * float(h[special, 1]), (kind, window, special, i)
            elif i > special + 1:
                assert abs(float(want[i][1] - h[special, 1])) > 0.4 * float(h[special, 1]), (kind, window, special, i)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", [A, B, C])
def test_a_far_key_among_hundreds(kind, dtype):
    """One key at position 3 among 900 over fifteen pages: every later row returns its value, whether the row comes in the
    prompt, in a later portion or token by token."""
    d, T = 16, 900
    layer, weights = standing_out(kind, d, None, 80.0 if kind != C else None)
    g = torch.Generator().manual_seed(11)
    h = 0.02 * torch.randn(T, d, generator=g)
    h[:, 0] += 1.0
    h[:, 1] += 0.25
    h[3] = 0.0
    h[3, 0], h[3, 1] = (26.0, 20.0) if kind == B else (1.0, 0.9)
    if kind != B:
        kn = torch.ones(d)
        kn[1] = 20.0
        weights["m.k.norm"] = kn.to(torch.bfloat16)
    h = h.to(torch.bfloat16).double()
    m = dict(layer["mixer"])
    if kind == A:                                       # turned values: what is returned turns with the distance
        m["rot"] = dict(m["rot"], base=1e4)
        layer = {"type": kind, "mixer": m, "mlp": None}
    want = plain.attention(h, weights, "m", kind, m, EPS)
    length = want[10:].pow(2).sum(-1).sqrt()
    assert float((length - float(h[3].pow(2).sum().sqrt())).abs().max()) < 0.1 * float(length.max())
    hs = harness(layer, d, dtype, weights=weights, capacity=1024)
    for portions in ([{"a": T}], [{"a": 500}, {"a": 300}] + [{"a": 1}] * 100, [{"a": 2}] * 450):
        close(hs.run({"a": h}, portions)["a"], want, dtype, f"{kind} {dtype} {len(portions)}", tol=1e-4 if dtype == torch.float32 else 0.02)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sinks_take_their_share(dtype):
    """Heads with sinks far below, at, and far above their scores; alone at position 0 a key shares with the sink only."""
    hidden, layer = MIXERS[0]
    hs = harness(layer, hidden, dtype)
    w = dict(hs.weights)
    w["m.sink"] = torch.tensor([-60.0, 0.0, 3.0, 12.0]).to(torch.bfloat16)
    w["m.o"] = torch.eye(hidden, 4 * 24).to(torch.bfloat16)              # the first head and most of the second, as they are
    hs = harness(layer, hidden, dtype, weights=w)
    h = inputs(120, hidden, 7)
    want = plain.attention(h, w, "m", A, layer["mixer"], EPS)
    for portions in ([{"a": 120}], [{"a": 1}] * 120):
        close(hs.run({"a": h}, portions)["a"], want, dtype, f"{dtype} sinks")
    w["m.sink"] = torch.tensor([200.0, 150.0, 120.0, 1000.0]).to(torch.bfloat16)     # nothing is left for the keys
    got = harness(layer, hidden, dtype, weights=w).run({"a": h}, [{"a": 60}] + [{"a": 1}] * 60)["a"]
    assert bool(torch.isfinite(got).all()) and float(got.abs().max()) < 1e-3


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_projection_norm_is_not_a_norm_a_head(dtype):
    """One head's queries and keys are ten times the others': over the whole projection they stay so."""
    hidden, layer = 40, mixer(C, 4, 4, 16, 16, 0.2, (16, 100.0), None)
    hs = harness(layer, hidden, dtype)
    w = dict(hs.weights)
    for n in ("m.q", "m.k"):
        t = w[n].clone()
        t[16:32] *= 10
        w[n] = t
    hs = harness(layer, hidden, dtype, weights=w)
    h = inputs(90, hidden, 3)
    want = plain.attention(h, w, "m", C, layer["mixer"], EPS)
    for portions in ([{"a": 90}], [{"a": 30}] + [{"a": 1}] * 60):
        close(hs.run({"a": h}, portions)["a"], want, dtype, f"{dtype} whole norm")


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_positions_and_rotations(dtype):
    """A sequence that starts far out (its cache is declared to hold 5,000 tokens that a window no longer shows): angles are
    formed at the true position."""
    hidden, layer = 32, mixer(A, 2, 1, 16, 16, 0.25, (16, 10000.0), None, softcap=20.0, window=8)
    hs = harness(layer, hidden, dtype, capacity=6144, max_seq=6144, slots=1)
    slot = hs.cache.acquire()
    past, T = 5000, 40
    hs.cache.reserve(slot, past)
    hs.cache.commit(slot, past)
    h = inputs(T, hidden, 2)
    outs = []
    for n in (20, 1, 1, 18):
        done = sum(o.shape[0] for o in outs)
        batch = pack_step([StepEntry(slot, [0] * n, [])], [past + done], 1, DEV)
        hs.cache.reserve(slot, past + done + n)
        y = torch.empty((n, hidden), dtype=torch.float32, device=DEV)
        hs.part.forward(h[done:done + n].to(DEV).to(dtype).contiguous(), batch, hs.cache.view(0), y, True, overwrite=True)
        hs.cache.commit(slot, past + done + n)
        outs.append(y.double().cpu())
    # the same tokens at positions 0 .. T - 1: scores and turned values depend on distances alone
    want = plain.attention(h, hs.weights, "m", A, layer["mixer"], EPS)
    got = torch.cat(outs)
    scale = float(want.abs().max())
    err = (got[7:] - want[7:]).abs().max()                  # from here on the window holds these tokens only
    assert float(err) <= (2e-3 if dtype == torch.float32 else 3e-2) * scale, float(err)


# ---- the norm over parts of a row, with the convolution behind it -----------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,groups", [(64, 1), (64, 4), (60, 4), (60, 60), (40, 8), (2048, 2), (4096, 4), (1536, 1), (5120, 8), (4100, 4)])
def test_norm_over_parts(hidden, groups, dtype):
    part = build_part("norm", PartSpec("grouped_rms_norm", {"size": hidden, "groups": groups, "eps": 1e-3, "tensor": "n.norm1"}, "n"))
    w = draw(part.tensor_specs(), 1)
    part.bind(handles(w), ctx_for(dtype))
    x = torch.randn(9, hidden, generator=torch.Generator().manual_seed(2)) * torch.linspace(0.01, 30.0, hidden)     # parts of unequal size
    want = plain.group_norm(x.double(), w["n.norm1"], groups, 1e-3)
    tol = 1e-6 if dtype == torch.float32 else 5e-3
    got = part.forward(x.to(DEV)).double().cpu()
    assert bool(((got - want).abs() <= tol * (want.abs() + 1e-3)).all())
    index = torch.tensor([8, 0, 3], dtype=torch.int32, device=DEV)
    assert torch.equal(part.forward(x.to(DEV), row_index=index).double().cpu(), got[[8, 0, 3]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,groups,taps", [(64, 4, 3), (64, 1, 2), (60, 4, 4), (40, 8, 3), (64, 2, 1), (48, 4, 6), (96, 3, 16), (1024, 4, 4), (4096, 2, 3)])
def test_residual_convolution(hidden, groups, taps, dtype):
    norm = build_part("norm", PartSpec("grouped_rms_norm", {"size": hidden, "groups": groups, "eps": 1e-3, "tensor": "n.norm1"}, "n"))
    conv = build_part("mixer_input", PartSpec("residual_conv", {"hidden_size": hidden, "taps": taps}, "n.canon1"))
    w = draw(norm.tensor_specs() + conv.tensor_specs(), 4)
    ctx = ctx_for(dtype)
    norm.bind(handles(w), ctx)
    conv.bind(handles(w), ctx)
    req = conv.cache_requirement()
    assert (req is None) == (taps == 1)
    cache = cb.SequenceCache([req], 3, 64, 4096, dtype, DEV)

    def run(sequences, portions):
        slots, done, out = {}, {}, {n: [] for n in sequences}
        for step in portions:
            for n in step:
                if n not in slots:
                    slots[n], done[n] = cache.acquire(), 0
            batch = pack_step([StepEntry(slots[n], [0] * step[n], []) for n in step], [done[n] for n in step], 1, DEV)
            x = torch.cat([sequences[n][done[n]:done[n] + step[n]] for n in step]).float().to(DEV).contiguous()
            h, m = conv.forward(norm, x, batch, cache.view(0) if taps > 1 else None)
            at = 0
            for n in step:
                out[n].append((h[at:at + step[n]].double().cpu(), m[at:at + step[n]].double().cpu()))
                at += step[n]
                done[n] += step[n]
        for n in slots:
            cache.release(slots[n])
        return {n: tuple(torch.cat(v) for v in zip(*out[n])) for n in out if out[n]}

    T = 330
    x = {n: torch.randn(t, hidden, generator=torch.Generator().manual_seed(t), dtype=torch.float64).float() for n, t in (("a", T), ("b", 21))}
    want = {}
    for n in x:
        h = plain.group_norm(x[n].double(), w["n.norm1"], groups, 1e-3)
        want[n] = (h, h + plain.causal_conv(h, w["n.canon1"]))
    tol = 2e-6 if dtype == torch.float32 else 6e-3
    ways = {"whole": [{"a": T}], "two portions": [{"a": 307}, {"a": 23}], "twos": [{"a": 2}] * (T // 2), "one by one": [{"a": 1}] * T,
            "mixed": [{"a": 1}, {"a": 2}, {"a": 1}, {"a": 1}, {"a": 3}, {"a": 300}, {"a": 1}, {"a": 1}, {"a": 2}, {"a": 18}]}
    first = None
    for what, portions in ways.items():
        got = run(x, portions)["a"]
        for g, t in zip(got, want["a"]):
            assert bool(((g - t).abs() <= tol * (t.abs() + 1.0)).all()), what
        first = first or got
        assert torch.equal(got[0], first[0]) and torch.equal(got[1], first[1]), what            # the same bits, however it is cut
    both = run(x, [{"a": 310, "b": 2}, {"b": 1, "a": 1}, {"b": 1, "a": 2}, {"a": 1, "b": 1}, {"a": 16, "b": 16}])
    for n in x:
        for g, t in zip(both[n], want[n]):
            assert bool(((g - t).abs() <= tol * (t.abs() + 1.0)).all()), n
    assert torch.equal(both["a"][1], first[1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,groups,taps", [(64, 4, 3), (96, 1, 2), (128, 8, 4), (60, 4, 5)])
def test_residual_convolution_of_long_steps(hidden, groups, taps, dtype):
    """Steps of more than a thousand rows (a block then takes several rows): one sequence, and a batch whose sequences begin and
    end inside such a block, some of them with fewer new tokens than the convolution looks back."""
    norm = build_part("norm", PartSpec("grouped_rms_norm", {"size": hidden, "groups": groups, "eps": 1e-3, "tensor": "n.norm1"}, "n"))
    conv = build_part("mixer_input", PartSpec("residual_conv", {"hidden_size": hidden, "taps": taps}, "n.canon1"))
    w = draw(norm.tensor_specs() + conv.tensor_specs(), 4)
    ctx = ctx_for(dtype)
    norm.bind(handles(w), ctx)
    conv.bind(handles(w), ctx)
    tol = 2e-6 if dtype == torch.float32 else 6e-3
    for steps in ([[1300], [900], [1]], [[701, 1, 2, 3, 600, 1], [1, 1, 1, 1, 1, 1], [2, 640, 1, 700, 3, 5], [3, 2, 1, 1, 9, 1]]):
        n = len(steps[0])
        cache = cb.SequenceCache([conv.cache_requirement()], n, 64, 4096, dtype, DEV)
        slots = [cache.acquire() for _ in range(n)]
        total = [sum(st[i] for st in steps) for i in range(n)]
        x = [torch.randn(t, hidden, generator=torch.Generator().manual_seed(i)).float() for i, t in enumerate(total)]
        done, got = [0] * n, [[] for _ in range(n)]
        for st in steps:
            batch = pack_step([StepEntry(slots[i], [0] * st[i], []) for i in range(n)], done, 1, DEV)
            rows = torch.cat([x[i][done[i]:done[i] + st[i]] for i in range(n)]).to(DEV).contiguous()
            h, m = conv.forward(norm, rows, batch, cache.view(0))
            at = 0
            for i in range(n):
                got[i].append(m[at:at + st[i]].double().cpu())
                at += st[i]
                done[i] += st[i]
        for i in range(n):
            h = plain.group_norm(x[i].double(), w["n.norm1"], groups, 1e-3)
            want = h + plain.causal_conv(h, w["n.canon1"])
            assert bool(((torch.cat(got[i]) - want).abs() <= tol * (want.abs() + 1.0)).all()), (i, steps)


# ---- the embedding of pairs ----------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,vocab,buckets,mul_prev,mul_cur", [(24, 50, 13, 7, 3), (300, 1000, 4001, 1023, 31), (16, 152000, 97, 2147483647, 2147483646), (32, 9, 1, 0, 5)])
def test_embedding_of_pairs(hidden, vocab, buckets, mul_prev, mul_cur, dtype):
    part = build_part("embedding", PartSpec("hashed_pairs", {"hidden_size": hidden, "buckets": buckets, "mul_prev": mul_prev,
                                                             "mul_cur": mul_cur, "pair_scale": 0.5}, "bigram"))
    w = draw(part.tensor_specs(), 3)
    table = torch.randn(vocab, hidden, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16)
    ctx = ctx_for(dtype)
    part.bind(handles(w), ctx)
    cache = cb.SequenceCache([part.cache_requirement()], 2, 64, 1024, dtype, DEV)
    dev_table = table.to(DEV).to(dtype)

    def run(sequences, portions):
        slots, done, out = {}, {}, {n: [] for n in sequences}
        for step in portions:
            for n in step:
                if n not in slots:
                    slots[n], done[n] = cache.acquire(), 0
            batch = pack_step([StepEntry(slots[n], sequences[n][done[n]:done[n] + step[n]], []) for n in step], [done[n] for n in step], vocab, DEV)
            x = torch.empty((batch.rows, hidden), dtype=torch.float32, device=DEV)
            part.forward(dev_table, batch, x, cache.view(0), ctx.error_flag, 3.0)
            at = 0
            for n in step:
                out[n].append(x[at:at + step[n]].double().cpu())
                at += step[n]
                done[n] += step[n]
        for n in slots:
            cache.release(slots[n])
        return {n: torch.cat(v) for n, v in out.items() if v}

    g = torch.Generator().manual_seed(5)
    seqs = {n: torch.randint(0, vocab, (t,), generator=g).tolist() for n, t in (("a", 60), ("b", 33))}
    want = {n: 3.0 * table.double()[torch.tensor(t)] + 0.5 * w["bigram"].double()[torch.tensor(plain.bigram_rows(t, mul_prev, mul_cur, buckets))]
            for n, t in seqs.items()}
    for portions in ([{"a": 60}], [{"a": 1}] * 60, [{"a": 2}] * 30, [{"a": 3}, {"a": 1}, {"a": 1}, {"a": 55}]):
        assert torch.allclose(run(seqs, portions)["a"], want["a"], rtol=1e-6, atol=1e-6)
    both = run(seqs, [{"b": 20, "a": 40}, {"b": 1, "a": 1}, {"a": 1, "b": 1}, {"b": 11, "a": 18}])       # slots that were used before
    for n in seqs:
        assert torch.allclose(both[n], want[n], rtol=1e-6, atol=1e-6)
    assert not any(ctx.error_flag.tolist())


# ---- feed-forwards -----------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("experts,top", [(6, 2), (3, 3), (16, 4), (10, 1), (40, 5), (200, 8)])
@pytest.mark.parametrize("extra", [False, True])
def test_router_softmax_over_the_chosen(experts, top, extra):
    g = torch.Generator().manual_seed(experts)
    logits = (3.0 * torch.randn(50, experts + extra, generator=g)).float()
    bias = torch.randn(experts, generator=g).float() * 2.0
    logits[0, :experts] = 1.25 - bias                      # (nearly) ties
    logits[1, :experts] = -200.0                           # all far below zero: the softmax is over differences
    logits[2, 0] = 300.0
    out = torch.empty(50, experts, dtype=torch.float32, device=DEV)
    chosen = torch.empty(50, top, dtype=torch.int32, device=DEV)
    gate = torch.empty(50, dtype=torch.float32, device=DEV) if extra else None
    ops.moe_route(logits.to(DEV), out, None, None, top, chosen=chosen, score="softmax_chosen", bias=bias.to(DEV), extra=gate)
    z = logits[:, :experts] + bias                          # the same 32-bit sum
    order = torch.sort(z, dim=-1, descending=True, stable=True).indices[:, :top]
    assert torch.equal(chosen.cpu().long(), order)
    want = torch.zeros(50, experts, dtype=torch.float64).scatter_(1, order, torch.softmax(z.double().gather(1, order), -1))
    assert float((out.double().cpu() - want).abs().max()) < 1e-6
    if extra:
        assert float((gate.double().cpu() - torch.sigmoid(logits[:, experts].double())).abs().max()) < 1e-6
    # a bias moves the choice
    other = torch.empty_like(out)
    ops.moe_route(logits.to(DEV), other, None, None, top, score="softmax_chosen", extra=gate)
    assert not torch.equal(other, out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,experts,top,ff,shared", [(40, 6, 2, 32, 24), (60, 3, 3, 24, 40), (64, 16, 4, 16, 16), (32, 10, 1, 40, None), (48, 5, 2, 20, 12)])
def test_experts_with_a_weighted_one_for_every_token(hidden, experts, top, ff, shared, dtype):
    params = {"hidden_size": hidden, "experts": experts, "top": top, "intermediate_size": ff, "score": "softmax_chosen", "router_bias": True,
              "activation": "silu", "shared": None if shared is None else {"intermediate_size": shared, "weight": "sigmoid"}}
    part = build_part("feed_forward", PartSpec("routed_experts", params, "f"))
    w = draw(part.tensor_specs(), 7)
    assert "f.router.b" in w and ("f.shared.sg" in w) == (shared is not None)
    part.bind(handles(w), ctx_for(dtype))
    h = 1.5 * inputs(90, hidden, 8)
    mlp = {"router": {"experts": experts, "top": top}, "shared": None if shared is None else {"ff": shared}}
    want = plain.moe(h, w, "f", mlp)
    _, _, margin = plain.route(h, w, "f", mlp["router"])
    y = torch.zeros(90, hidden, dtype=torch.float32, device=DEV)
    part.forward(h.to(DEV).to(dtype).contiguous(), None, y)
    got = y.double().cpu()
    sure = margin > 1e-2                                   # rows whose choice no rounding can change
    assert int(sure.sum()) > 60
    close(got[sure], want[sure], dtype, f"{dtype} experts")
    one = torch.ones(1, hidden, dtype=torch.float32, device=DEV)
    part.forward(h[:1].to(DEV).to(dtype).contiguous(), None, one)
    close(one.double().cpu() - 1.0, want[:1], dtype, f"{dtype} one row")
    if shared is not None:                                 # the sigmoid is not one
        other = build_part("feed_forward", PartSpec("routed_experts", dict(params, shared={"intermediate_size": shared}), "f"))
        other.bind(handles(w), ctx_for(dtype))
        y2 = torch.zeros(90, hidden, dtype=torch.float32, device=DEV)
        other.forward(h.to(DEV).to(dtype).contiguous(), None, y2)
        assert float((y2.double().cpu() - want)[sure].abs().max()) > 0.05 * float(want.abs().max())


# ---- the block ------------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", [0, 1, 5, 9])
def test_block_whose_mixer_reads_convolved_rows(which, dtype):
    hidden, layer = MIXERS[which]
    layer = dict(layer, mlp={"kind": "dense", "ff": 48})
    d = model(64, hidden, 1e-4, 4, 1.0, 1.0, None, 3, None, None, [layer])
    spec = cb.config_from_dict(d).to_model_spec().layers[0]
    block = part_class("block", spec.block)(spec)
    w = draw(block.tensor_specs(), 2)
    block.bind(handles(w), ctx_for(dtype))
    cache = cb.SequenceCache([block.cache_requirement()], 1, 256, 256, dtype, DEV)
    T = 90
    x = torch.randn(T, hidden, generator=torch.Generator().manual_seed(4)).float()
    rin = (lambda t: t) if dtype == torch.float32 else (lambda t: t.to(torch.bfloat16).double())
    want = plain.layer(x.double(), w, 0, layer, d, rin, None)
    for portions in ([T], [1] * T, [40, 1, 2, 1, 46]):
        slot = cache.acquire()
        rows, done = [], 0
        for n in portions:
            batch = pack_step([StepEntry(slot, [0] * n, [])], [done], 1, DEV)
            cache.reserve(slot, done + n)
            xd = x[done:done + n].to(DEV).clone()
            block.forward(xd, batch, cache.view(0), True)
            cache.commit(slot, done + n)
            rows.append(xd.double().cpu())
            done += n
        cache.release(slot)
        close(torch.cat(rows), want, dtype, f"{dtype} block in {len(portions)}")


def test_parts_refuse_what_they_cannot_do():
    base = dict(hidden_size=32, heads=2, kv_heads=1, dim=16, vdim=16, scale=1.0)
    for edit, match in ((dict(qk_norm_eps=1e-5, rot_layout="halves", rot_dims=8), "convolution"), (dict(conv=4, value_rot_base=10.0), "convolution"),
                        (dict(rot_layout="thirds"), "layout"), (dict(qk_norm_over="rows"), "qk_norm_over"), (dict(sink="one"), "sink"),
                        (dict(vdim=15, value_rot_base=10.0), "even")):
        with pytest.raises(cb.CitlaliError, match=match):
            build_part("mixer", PartSpec("window_attention", dict(base, **edit), "m"))
    with pytest.raises(cb.CitlaliError, match="parts"):
        build_part("norm", PartSpec("grouped_rms_norm", {"size": 10, "groups": 3, "eps": 1e-5}, "n"))
    with pytest.raises(cb.CitlaliError, match="taps"):
        build_part("mixer_input", PartSpec("residual_conv", {"hidden_size": 8, "taps": 17}, "c"))
