"""Each mechanism of the Kopalorn design alone, built through the registries at sizes no model uses, against the plain
implementation: differential attention (whole, token by token, in portions and in batches through one cache; 32-bit bitwise equal
however a sequence is cut); a key that stands out in one of the two maps just inside and just outside windows, at page borders, in
prompts and in decoding; a far key among hundreds; positions far out; the matrix memory with exponential gates (gates that open and
close, a key sum that nearly cancels, maxima that run away) and the memory with fixed decays, each also 64 tokens at a time on the
tensor cores against token by token; the pair of normed mixers; the corrected grouped router and experts without a gate; the step
ahead of a repeated run of layers; the block and its multiplier."""
import math

import pytest
import torch

import citlali_b200 as cb
import plain_kopalorn as plain
from citlali_b200 import ops
from citlali_b200.config.spec import LayerSpec, PartSpec
from citlali_b200.engine.step import StepEntry, pack_step
from citlali_b200.parts.base import build_part, part_class
from kopalorn_models import attention, draw_tensor, mlstm, model, moe, parallel
from test_gpu_pivavik_parts import DEV, DTYPES, Harness, close, ctx_for, cuts, every_way, handles, inputs

pytestmark = pytest.mark.gpu
EPS = 1e-5


def draw(specs, seed):
    g = torch.Generator().manual_seed(seed)
    return {s.name: draw_tensor(s.name, tuple(s.shape), torch.randn(tuple(s.shape), generator=g)).to(torch.bfloat16) for s in specs}


def layer_spec(layer, hidden, mult=1.0):
    return cb.config_from_dict(model(64, hidden, EPS, mult, None, [layer])).to_model_spec().layers[0]


def harness(layer, hidden, dtype, weights=None, seed=3, side=None, **kw):
    """The layer's mixer under the prefix 'm' (``side``: one of a parallel layer's two) with a cache of its own."""
    spec = layer_spec(layer, hidden).parts["mixer"]
    spec = spec if side is None else spec.params[side]
    params = dict(spec.params)
    if spec.kind == "parallel":
        params["left"], params["right"] = (PartSpec(params[s].kind, params[s].params, "m." + s) for s in ("left", "right"))
        params["out_norms"] = dict(params["out_norms"], left="m.left.out", right="m.right.out", size=hidden)
        params["hidden_size"] = hidden
    part = build_part("mixer", PartSpec(spec.kind, params, "m"))
    return Harness(spec.kind, params, dtype, weights=weights if weights is not None else draw(part.tensor_specs(), seed), **kw)


# ---- differential attention -------------------------------------------------------------------------------------------------

DIFFERENTIAL = [
    (40, attention(4, 2, 16, 24, 0.3, 0.4, (8, 100.0), 9, None)),
    (48, attention(3, 3, 20, 12, 0.3, 0.7, (20, 1000.0), 65, None)),          # no tensor-core sizes for a value
    (32, attention(2, 2, 14, 10, 0.35, 0.2, (6, 10.0), 1, None)),             # single pieces, itself alone
    (64, attention(8, 1, 32, 64, 0.2, 0.6, (32, 50.0), 130, None)),           # sixteen maps a key head
    (24, attention(3, 1, 10, 6, 0.4, 0.5, (2, 30.0), None, None)),
    (40, attention(4, 4, 24, 48, 0.25, 0.0, None, None, None)),               # no rotation, no window, no constant
    (56, attention(16, 1, 64, 128, 0.12, 0.8, (64, 1e4), 100, None)),         # thirty-two maps a key head, two tiles of the decode kernel
    (64, attention(4, 2, 64, 128, 0.15, 0.3, (32, 500.0), 70, None)),         # the widest prompt kernel
    (48, attention(2, 1, 128, 136, 0.08, 0.5, (128, 1e6), 64, None)),         # the widest tiles
    (32, attention(1, 1, 8, 8, 0.4, 0.3, (4, 20.0), 33, None)),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,layer", DIFFERENTIAL)
def test_differential_attention(hidden, layer, dtype):
    hs = harness(layer, hidden, dtype)
    fn = lambda h: plain.differential_attention(h, hs.weights, "m", layer["mixer"], EPS)
    every_way(hs, fn, inputs(150, hidden, 3), inputs(37, hidden, 4), dtype)


@pytest.mark.parametrize("which,drop", [(0, "window"), (0, "rotation"), (0, "halves"), (0, "gate"), (0, "diff"), (0, "second map"), (7, "window"),
                                        (7, "second map")])
def test_each_mechanism_of_differential_attention_matters(which, drop):
    """Switching one of them off changes the mixer's output: none is silently dropped on the way."""
    hidden, layer = DIFFERENTIAL[which]
    base = harness(layer, hidden, torch.float32)
    h = inputs(100, hidden, 8)
    full = base.run({"a": h}, [{"a": 100}])["a"]
    p = dict(layer_spec(layer, hidden).parts["mixer"].params)
    w = dict(base.weights)
    if drop == "second map":                               # lambda of zero: exp(0) - exp(log(1 + diff)) + diff
        d = layer["mixer"]["dim"]
        w["m.lq1"] = torch.zeros(d)
        w["m.lq2"], w["m.lk2"] = torch.eye(d)[0], torch.eye(d)[0] * math.log(1.0 + layer["mixer"]["diff"])
    edit = {"window": {"window": None}, "rotation": {"rot_dims": 0}, "halves": {"rot_layout": "halves"}, "gate": {"gate": None},
            "diff": {"diff": 0.0}, "second map": {}}[drop]
    other = Harness("differential_attention", dict(p, **edit), torch.float32, weights=w).run({"a": h}, [{"a": 100}])["a"]
    assert float((other - full).abs().max()) > 1e-2 * float(full.abs().max()), drop


def standing_out(which_map, d, window):
    """One head whose map ``which_map`` scores the inputs themselves and whose other map scores nothing (an average)."""
    layer = attention(1, 1, d, d, 1.0, 0.9 if which_map else 0.05, None, window, None)
    eye, zero = torch.eye(d), torch.zeros(d, d)
    w = {"m.q": torch.cat([zero, eye] if which_map else [eye, zero]), "m.k": torch.cat([eye, eye]), "m.v": eye, "m.o": eye, "m.g": torch.zeros(1, d),
         "m.lq1": torch.zeros(d), "m.lk1": torch.zeros(d), "m.lq2": torch.zeros(d), "m.lk2": torch.zeros(d)}
    return layer, {k: v.to(torch.bfloat16) for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [8, 64])
@pytest.mark.parametrize("decode_from", [None, 40])
@pytest.mark.parametrize("which_map", [0, 1])
@pytest.mark.parametrize("window", [1, 9, 64, 65, 130])
def test_window_edges_with_one_key_that_stands_out(window, which_map, decode_from, d, dtype):
    """One key's score in one map is far above the others': the map returns that token's value while it is inside the window (which
    turns the head's direction), and loses it at the next row; over page borders; in prompts and in decoding."""
    T = 210
    layer, weights = standing_out(which_map, d, window)
    for special in (0, 1, 63, 64, 100):
        g = torch.Generator().manual_seed(special)
        h = 0.02 * torch.randn(T, d, generator=g)
        h[:, 0] += 1.0
        h[special, 0], h[special, 1] = 20.0, 16.0
        h = h.to(torch.bfloat16).double()
        hs = harness(layer, d, dtype, weights=weights)
        portions = [{"a": T}] if decode_from is None else [{"a": decode_from}] + [{"a": 1}] * (T - decode_from)
        got = hs.run({"a": h}, portions)["a"]
        want = plain.differential_attention(h, weights, "m", layer["mixer"], EPS)
        allowed = (1e-4 if dtype == torch.float32 else 0.03) * want.abs().amax(-1, keepdim=True).clamp(min=1e-3)
        if window == 1:                    # both maps return the token itself: the difference is (1 - lambda) of it, no cancellation
            assert bool(((got - want).abs() <= allowed).all())
            continue
        assert bool(((got - want).abs() <= allowed).all()), (window, special, float(((got - want).abs() / allowed).max()))
        see = plain.visible(T, window)
        for i in range(special + 1, T):                     # the test's point: the special key decides the row's direction
            slope = float(want[i][1] / want[i][0])
            if bool(see[i, special]):
                assert slope > 0.5, (window, special, i)
            elif i > special + 1:
                assert abs(slope) < 0.2, (window, special, i)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which_map", [0, 1])
def test_a_far_key_among_hundreds(which_map, dtype):
    """One key at position 3 among 900 over fifteen pages decides every later row, whether the row comes in the prompt, in a later
    portion or token by token."""
    d, T = 16, 900
    layer, weights = standing_out(which_map, d, None)
    h = 0.02 * torch.randn(T, d, generator=torch.Generator().manual_seed(11))
    h[:, 0] += 1.0
    h[3, 0], h[3, 1] = 26.0, 20.0
    h = h.to(torch.bfloat16).double()
    want = plain.differential_attention(h, weights, "m", layer["mixer"], EPS)
    assert float((want[4:, 1] / want[4:, 0]).min()) > 0.5
    hs = harness(layer, d, dtype, weights=weights, capacity=1024)
    for portions in ([{"a": T}], [{"a": 500}, {"a": 300}] + [{"a": 1}] * 100, [{"a": 2}] * 450):
        close(hs.run({"a": h}, portions)["a"], want, dtype, f"{dtype} {len(portions)}", tol=1e-4 if dtype == torch.float32 else 0.02)


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_positions(dtype):
    """A sequence that starts far out (its cache is declared to hold 5,000 tokens that a window no longer shows): angles are formed at
    the true position."""
    hidden, layer = 32, attention(2, 1, 16, 16, 0.25, 0.5, (16, 10000.0), 8, None)
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
    want = plain.differential_attention(h, hs.weights, "m", layer["mixer"], EPS)      # scores depend on distances alone
    got = torch.cat(outs)
    assert float((got[7:] - want[7:]).abs().max()) <= (2e-3 if dtype == torch.float32 else 3e-2) * float(want.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,V", [(1, 6), (3, 36), (5, 128), (9, 250), (16, 256)])
def test_differential_output(H, V, dtype):
    rows = 7
    g = torch.Generator().manual_seed(V)
    a = torch.randn(rows, 2 * H, V, generator=g)
    a[:, 1::2] += 0.9 * a[:, 0::2]                          # the maps are alike: the difference is small
    z = torch.randn(rows, H + 3, generator=g)
    y = torch.empty((rows, H * V), dtype=dtype, device=DEV)
    ops.differential_output(a.view(rows, -1).to(DEV), 0.85, 0.4, 1e-4, z.to(DEV)[:, 2:2 + H], y, H, V)
    o = plain.rms(a[:, 0::2].double() - 0.85 * a[:, 1::2].double(), 1e-4) * 0.4 * torch.sigmoid(z[:, 2:2 + H].double())[..., None]
    close(y.double().cpu(), o.reshape(rows, -1), dtype, "differential output", tol=3e-6 if dtype == torch.float32 else 5e-3)
    ops.differential_output(a.view(rows, -1).to(DEV), 0.85, 0.4, 1e-4, None, y, H, V)
    close(y.double().cpu(), (o / torch.sigmoid(z[:, 2:2 + H].double())[..., None]).reshape(rows, -1), dtype, "no gate",
          tol=3e-6 if dtype == torch.float32 else 5e-3)


# ---- memories ---------------------------------------------------------------------------------------------------------------

MATRIX = [
    (40, mlstm(3, 16, 24, 6.0, None)),
    (60, mlstm(5, 12, 20, 15.0, None)),                    # rows that no 16-byte word divides
    (32, mlstm(1, 7, 5, 2.0, None)),
    (64, mlstm(2, 64, 64, 12.0, None)),
    (48, mlstm(2, 128, 96, 8.0, None)),
    (40, mlstm(1, 250, 70, 10.0, None)),
    (24, mlstm(4, 8, 6, 30.0, None)),
]
DECAYS = [
    (40, (16, 24, (0.5, 0.9, 0.99))),
    (60, (20, 12, (0.0, 0.3, 0.7, 0.95, 1.0))),            # nothing is kept; everything is
    (32, (7, 5, (0.97,))),
    (64, (64, 64, (0.8, 0.999))),
    (48, (128, 33, (0.99, 0.2))),
    (40, (256, 70, (0.999,))),
]


def memory_close(got, want, dtype, what):
    """In bfloat16 a head whose result nearly cancels is blown up, rounding and all, by the norm behind it: nearly all rows are held
    tightly, all of them loosely, and the rounding of the sums themselves is held in the test of the kernels below."""
    if dtype == torch.float32:
        close(got, want, dtype, what)
        return
    err = (got - want).abs().amax(-1) / want.abs().max()
    assert float(err.max()) < 0.3 and float(err.median()) < 6e-3 and float((err < 3e-2).double().mean()) >= 0.93, (what, err.topk(5).values)


def every_way_of_a_memory(hs, fn, h, other, dtype):
    if dtype == torch.float32:
        every_way(hs, fn, h, other, dtype)
        return
    T, n, want = h.shape[0], other.shape[0], fn(h)
    for what, portions in cuts(T).items():
        memory_close(hs.run({"a": h}, portions)["a"], want, dtype, what)
    both = hs.run({"a": h, "b": other}, [{"a": 50, "b": 20}, {"a": 1, "b": 1}, {"a": 1, "b": 1}, {"a": T - 52, "b": n - 22}])
    memory_close(both["a"], want, dtype, "batched a")
    memory_close(both["b"], fn(other), dtype, "batched b")
    memory_close(hs.run({"c": other}, [{"c": n}])["c"], fn(other), dtype, "a slot used again")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,layer", MATRIX)
def test_matrix_memory(hidden, layer, dtype):
    hs = harness(layer, hidden, dtype)
    fn = lambda h: plain.mlstm(h, hs.weights, "m", layer["mixer"], EPS)
    every_way_of_a_memory(hs, fn, inputs(150, hidden, 3), inputs(37, hidden, 4), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,right", DECAYS)
def test_memory_with_fixed_decays(hidden, right, dtype):
    layer = parallel((1, 1, 8, 8, 0.3), right, None)
    hs = harness(layer, hidden, dtype, side="right")
    assert all(n.startswith("m.") for n in hs.weights)
    fn = lambda h: plain.lightning(h, hs.weights, "m", layer["mixer"]["right"], EPS)
    every_way_of_a_memory(hs, fn, inputs(150, hidden, 3), inputs(37, hidden, 4), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", [0, 3])
def test_long_memories(which, dtype):
    """Twelve chunks of a prompt, a second prompt behind it, and tokens one by one."""
    T = 800
    hidden, layer = MATRIX[which]
    h = inputs(T, hidden, 12)
    hs = harness(layer, hidden, dtype)
    want = plain.mlstm(h, hs.weights, "m", layer["mixer"], EPS)
    hidden2, right = DECAYS[which]
    lay2 = parallel((1, 1, 8, 8, 0.3), right, None)
    hs2 = harness(lay2, hidden2, dtype, side="right")
    h2 = inputs(T, hidden2, 13)
    want2 = plain.lightning(h2, hs2.weights, "m", lay2["mixer"]["right"], EPS)
    for portions in ([{"a": T}], [{"a": 333}, {"a": 400}, {"a": 7}] + [{"a": 1}] * 60):
        memory_close(hs.run({"a": h}, portions)["a"], want, dtype, f"{dtype} matrix memory")
        memory_close(hs2.run({"a": h2}, portions)["a"], want2, dtype, f"{dtype} fixed decays")


def test_each_mechanism_of_the_memories_matters():
    hidden, layer = MATRIX[0]
    h = inputs(100, hidden, 8)
    base = harness(layer, hidden, torch.float32)
    full = base.run({"a": h}, [{"a": 100}])["a"]
    p = dict(layer_spec(layer, hidden).parts["mixer"].params)
    changed = lambda edit, w=None: Harness("linear_memory", dict(p, **edit), torch.float32, weights=dict(base.weights, **(w or {}))).run({"a": h}, [{"a": 100}])["a"]
    zero = torch.zeros(3)
    for what, other in (("cap", changed({"gate_cap": 0.5})), ("row norm", changed({"norm_over": "row"})),
                        ("silu", changed({"act": "silu"})), ("input bias", changed({}, {"m.i.b": zero})), ("forget bias", changed({}, {"m.f.b": zero}))):
        assert float((other - full).abs().max()) > 1e-2 * float(full.abs().max()), what


def memory_case(seed, lengths, H, D, V, kind):
    """Random q, k, v of sequences of ``lengths`` and gates ``kind``: a batch, its state region and the plain results."""
    g = torch.Generator().manual_seed(seed)
    rows = sum(lengths)
    q, k, v = (torch.randn(rows, H, n, generator=g).to(torch.bfloat16).float() for n in (D, D, V))
    if kind == "decay":
        decay = torch.tensor([(0.0, 1.0, 0.999, 0.9, 0.3, 0.6, 0.99, 0.05)[j % 8] for j in range(H)])
        return q, k, v, decay, None, None
    zi, zf = torch.randn(rows, H, generator=g), torch.randn(rows, H, generator=g)
    if kind == "calm":
        zf = zf + 3.0
    elif kind == "wild":                                   # maxima that run up and down by tens, gates that shut for good
        zi, zf = 12.0 * zi, 12.0 * zf
    elif kind == "shut":                                   # nothing is written: the floor exp(-m) decides
        zi, zf = zi - 14.0, zf + 2.0
    elif kind == "kept":                                   # nothing is forgotten
        zf = zf + 14.0
    return q, k, v, None, zi, zf


@pytest.mark.parametrize("D,V", [(16, 24), (64, 32), (96, 100), (128, 128), (200, 33), (256, 64), (10, 6)])
@pytest.mark.parametrize("kind", ["decay", "calm", "wild", "shut", "kept"])
def test_chunks_against_single_steps(kind, D, V):
    """The kernel that takes 64 tokens at a time against the one that takes them one by one and against the plain walk: results, key
    sums and the state they leave, for sequences around a chunk's length, and on from that state."""
    H, lengths = 3, [1, 63, 64, 65, 130, 2, 200]
    q, k, v, decay, zi, zf = memory_case(D + V, lengths, H, D, V, kind)
    rows, B = sum(lengths), len(lengths)
    proj = torch.cat([q.reshape(rows, -1), k.reshape(rows, -1), v.reshape(rows, -1)], 1).to(DEV)
    hd, cap, gated = H * D, 15.0, decay is None
    floats = H * D * V + hd + H
    outs = {}
    for form in (ops.MEMORY_SCAN, ops.MEMORY_CHUNKS):
        state = torch.zeros((B + 1, floats), dtype=torch.float32, device=DEV)
        slots = [(3 * b + 1) % B for b in range(B)]
        got, keys, logged = [], [], []
        for part in range(2):                              # each sequence twice: the second time from the state it left
            batch = pack_step([StepEntry(slots[b], [0] * n, []) for b, n in enumerate(lengths)], [0] * B, 1, DEV)
            logs = sums = floors = None
            if gated:
                logs, sums, floors = (torch.empty(s, dtype=torch.float32, device=DEV) for s in ((rows, H, 2), (rows, H), (rows, H)))
                z = torch.cat([zi, zf], 1).to(DEV)
                ops.memory_gates(z[:, :H], z[:, H:], None, None, cap, state, H * D * V + hd, batch, logs, floors)
            o = torch.empty((rows, H * V), dtype=torch.float32, device=DEV)
            ops.linear_memory(proj[:, :hd], proj[:, hd:2 * hd], proj[:, 2 * hd:], state, batch, H, D, V, o, decay=decay.to(DEV) if not gated else None,
                              logs=logs, sums=sums, sum_off=H * D * V, q_scale=D ** -0.5, form=form)
            got.append(o.double().cpu().view(rows, H, V))
            if gated:
                keys.append((sums.double().cpu(), floors.double().cpu()))
                logged.append(logs.double().cpu())
        outs[form] = (got, keys, state.double().cpu())
        assert torch.equal(state[B], torch.zeros_like(state[B]))              # a slot nobody uses
    at = 0
    for b, n in enumerate(lengths):
        for h in range(H):
            twice = lambda t: torch.cat([t[at:at + n, h]] * 2).double()
            qq, kk, vv = twice(q) * D ** -0.5, twice(k), twice(v)
            # what token t keeps of token s, from the gates' own logs (or the decay), and the size of what is summed
            steps = torch.arange(2 * n)
            if gated:
                l = torch.cat([t[at:at + n, h] for t in logged])
                total = torch.cumsum(l[:, 0], 0)
                W = torch.exp(total[:, None] - total[None, :] + l[None, :, 1])
            else:
                W = float(decay[h].double()) ** (steps[:, None] - steps[None, :]).clamp(min=0).double()
            W = torch.where(steps[:, None] >= steps[None, :], W, torch.zeros_like(W))
            P, terms = (qq @ kk.T) * W, (qq.abs() @ kk.abs().T) * W
            want, size = P @ vv, terms @ vv.abs() + 1e-30
            for form, tol in ((ops.MEMORY_SCAN, 1e-5), (ops.MEMORY_CHUNKS, 6e-3)):
                o = torch.cat([outs[form][0][p][at:at + n, h] for p in range(2)])
                assert bool(((o - want).abs() <= tol * size).all()), (kind, form, b, h, float(((o - want).abs() / size).max()))
                if gated:
                    s = torch.cat([t[0][at:at + n, h] for t in outs[form][1]])
                    assert bool(((s - P.sum(-1)).abs() <= tol * (terms.sum(-1) + 1e-30)).all()), (kind, form, b, h, "key sums")
            if gated:                                      # the gates themselves, through the ratio the plain walk gives
                i = cap * torch.tanh(twice(zi[..., None])[:, 0] / cap)
                f = torch.nn.functional.logsigmoid(cap * torch.tanh(twice(zf[..., None])[:, 0] / cap))
                exact = plain.stabilised_memory(qq, kk, vv, i, f)
                s, floor = (torch.cat([t[x][at:at + n, h] for t in outs[ops.MEMORY_SCAN][1]]) for x in (0, 1))
                den = torch.maximum(s.abs(), floor) + 1e-6
                o = torch.cat([outs[ops.MEMORY_SCAN][0][p][at:at + n, h] for p in range(2)]) / den[:, None]
                assert bool(((o - exact).abs() <= 1e-4 * (size + exact.abs() * terms.sum(-1)[:, None]) / den[:, None]).all()), (kind, b, h)
        at += n
    a, c = outs[ops.MEMORY_SCAN][2], outs[ops.MEMORY_CHUNKS][2]
    assert float((a - c).norm()) <= 6e-3 * float(a.norm()), kind


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,V,groups", [(3, 20, 3), (5, 33, 1), (1, 300, 1), (8, 128, 8), (4, 2000, 1), (2, 5000, 1), (2, 700, 2)])
@pytest.mark.parametrize("with_sums", [False, True])
def test_memory_output(H, V, groups, with_sums, dtype):
    rows, g = 5, torch.Generator().manual_seed(V)
    o, z, w = torch.randn(rows, H * V, generator=g), torch.randn(rows, H * V, generator=g), torch.randn(H * V, generator=g)
    sums, floors = torch.randn(rows, H, generator=g), torch.rand(rows, H, generator=g)
    sums[0, 0], floors[0, 0] = 0.0, 0.0                     # only the small constant is left
    y = torch.empty((rows, H * V), dtype=dtype, device=DEV)
    dev = lambda t: t.to(DEV) if with_sums else None
    ops.linear_memory_output(o.to(DEV), dev(sums), dev(floors), torch.cat([z, z], 1).to(DEV)[:, H * V:], w.to(DEV), y, H, V, groups, 1e-5)
    x = o.double().view(rows, H, V)
    if with_sums:
        x = x / (torch.maximum(sums.abs(), floors).double() + 1e-6)[..., None]
    want = plain.rms(x.reshape(rows, groups, -1), 1e-5).reshape(rows, -1) * w.double() * torch.sigmoid(z.double())
    close(y.double().cpu(), want, dtype, "memory output", tol=5e-6 if dtype == torch.float32 else 5e-3)


# ---- two mixers side by side ------------------------------------------------------------------------------------------------

PARALLEL = [
    (64, parallel((4, 2, 16, 8, 0.25), (16, 24, (0.5, 0.9, 0.99)), None)),
    (60, parallel((5, 5, 12, 20, 0.3), (20, 12, (0.0, 0.3, 0.7, 0.95, 1.0)), None)),
    (72, parallel((8, 1, 128, 128, 0.1), (64, 64, (0.97, 0.8)), None)),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,layer", PARALLEL)
def test_normed_mixers_side_by_side(hidden, layer, dtype):
    hs = harness(layer, hidden, dtype)
    fn = lambda h: plain.parallel(h, hs.weights, "m", layer["mixer"], EPS)
    every_way(hs, fn, inputs(150, hidden, 3), inputs(37, hidden, 4), dtype)
    # either side's norm weighs: the left output ten times as large changes nothing, its weight does
    h = inputs(60, hidden, 5)
    base = hs.run({"a": h}, [{"a": 60}])["a"]
    loud = dict(hs.weights, **{"m.left.o": (hs.weights["m.left.o"].float() * 16.0).to(torch.bfloat16)})
    close(harness(layer, hidden, dtype, weights=loud).run({"a": h}, [{"a": 60}])["a"], base, dtype, "a louder left side", tol=2e-2)
    other = dict(hs.weights, **{"m.left.out": hs.weights["m.left.out"] * 2})
    assert float((harness(layer, hidden, dtype, weights=other).run({"a": h}, [{"a": 60}])["a"] - base).abs().max()) > 0.1 * float(base.abs().max())


@pytest.mark.parametrize("hidden", [6, 60, 1026, 4096, 5000, 9001, 12288])
def test_normed_pair_sum(hidden):
    g = torch.Generator().manual_seed(hidden)
    l, r = torch.randn(5, hidden, generator=g), 7.0 * torch.randn(5, hidden, generator=g)
    wl, wr = torch.randn(hidden, generator=g), torch.randn(hidden, generator=g)
    want = 0.5 * plain.rms(l.double(), 1e-3) * wl.double() + 0.25 * plain.rms(r.double(), 1e-2) * wr.double()
    ld, out = l.to(DEV), torch.empty((5, hidden), dtype=torch.float32, device=DEV)
    ops.normed_pair_sum(0.5, ld, wl.to(DEV), 1e-3, 0.25, r.to(DEV), wr.to(DEV), 1e-2, out)
    close(out.double().cpu(), want, torch.float32, "pair", tol=2e-6)
    ops.normed_pair_sum(0.5, ld, wl.to(DEV), 1e-3, 0.25, r.to(DEV), wr.to(DEV), 1e-2, ld)
    assert torch.equal(ld, out)


# ---- experts ----------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("experts,top,groups", [(6, 2, (2, 1)), (16, 4, (4, 2)), (8, 8, None), (40, 5, (5, 2)), (9, 1, (9, 3)), (200, 8, (8, 3)), (12, 3, (2, 2)),
                                                (64, 6, (32, 4)), (10, 5, (2, 1))])
@pytest.mark.parametrize("extra", [False, True])
def test_router_with_corrections_and_groups(experts, top, groups, extra):
    g = torch.Generator().manual_seed(experts)
    rows = 60
    logits = (2.0 * torch.randn(rows, experts + extra, generator=g)).float()
    correction = (0.5 * torch.randn(experts, generator=g) - 0.4).float()          # choice scores of either sign
    logits[1] = -100.0                                     # scores that are nothing but their corrections; weights of equal shares
    out = torch.empty(rows, experts, dtype=torch.float32, device=DEV)
    chosen = torch.empty(rows, top, dtype=torch.int32, device=DEV)
    gate = torch.empty(rows, dtype=torch.float32, device=DEV) if extra else None
    route = lambda c, best, again, to: ops.moe_route(logits.to(DEV), to, groups and groups[0], groups and groups[1], top, chosen=chosen, weight_scale=1.7,
                                                     score="sigmoid", extra=gate, correction=None if c is None else c.to(DEV), group_best=best,
                                                     renormalise=again)
    route(correction, 2, True, out)
    picked, got = chosen.cpu().long(), out.double().cpu()
    r = {"top": top, "scale": 1.7}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    same = 0
    for t in range(rows):
        want = plain.route_row(logits[t, :experts].double(), correction.double(), r)
        if set(want) == set(picked[t].tolist()):           # (a choice within rounding may fall either way)
            same += 1
            w = torch.zeros(experts, dtype=torch.float64)
            if t == 1:
                assert all(float(got[t][e]) >= 0.0 for e in want)          # (no score left: shares of almost nothing)
                continue
            for e, v in want.items():
                w[e] = v
            assert float((got[t] - w).abs().max()) < 1e-5
    assert same >= rows - 2
    if extra:
        assert float((gate.double().cpu() - torch.sigmoid(logits[:, experts].double())).abs().max()) < 1e-6
    if top < experts:
        other = torch.empty_like(out)
        if top < experts and (groups is None or groups[1] * (experts // groups[0]) > top or groups[1] < groups[0]):
            route(None, 2, True, other)
            assert not torch.equal(other, out)             # the corrections move choices
        route(correction, 2, False, other)
        assert float((other[2:].sum(-1) - 1.7).abs().max()) > 1e-2 and float((out[2:].sum(-1) - 1.7).abs().max()) < 1e-5


def test_group_scores_by_hand():
    """The group with the best single expert against the one with the best pair; choice scores below zero; groups of one."""
    z = torch.tensor([[4.0, -3.0, 0.5, 0.4, 3.0, -4.0]], device=DEV)
    def chosen_of(correction, groups, keep, top, best):
        out, chosen = torch.empty(1, 6, device=DEV), torch.empty(1, top, dtype=torch.int32, device=DEV)
        c = None if correction is None else torch.tensor(correction, device=DEV)
        ops.moe_route(z, out, groups, keep, top, chosen=chosen, score="sigmoid", correction=c, group_best=best, renormalise=True)
        assert abs(float(out.sum()) - 1.0) < 1e-6 and int((out > 0).sum()) == top
        return set(chosen[0].tolist())
    assert chosen_of(None, 3, 1, 2, 2) == {2, 3} and chosen_of(None, 3, 1, 2, 1) == {0, 1}
    assert chosen_of([-5.0, -5.0, -1.0, -5.0, -5.0, -5.0], 3, 1, 2, 2) == {2, 3}       # closed groups count as minus infinity, not zero
    assert chosen_of(None, 6, 2, 2, 2) == {0, 4}
    assert chosen_of([0.0, 0.0, 0.0, 0.0, 1.0, 1.0], 2, 1, 3, 2) == {3, 4, 5}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,mlp", [(40, moe(6, 2, 32, 24, (2, 1), 1.7)), (60, moe(3, 3, 22, 41)), (64, moe(16, 4, 16, 16, (4, 2), 2.5)), (32, moe(10, 1, 40)),
                                        (48, moe(8, 3, 20, None, (4, 2), 0.5))])
def test_experts_without_a_gate(hidden, mlp, dtype):
    layer = attention(1, 1, 8, 8, 0.3, 0.5, None, None, mlp)
    p = layer_spec(layer, hidden).parts["feed_forward"].params
    part = build_part("feed_forward", PartSpec("routed_experts", p, "f"))
    w = draw(part.tensor_specs(), 7)
    assert "f.correction" in w and "f.e0.gate" not in w and ("f.shared.sg" in w) == ("shared" in mlp)
    part.bind(handles(w), ctx_for(dtype))
    h = 1.5 * inputs(90, hidden, 8)
    want = plain.moe(h, w, "f", mlp)
    y = torch.zeros(90, hidden, dtype=torch.float32, device=DEV)
    part.forward(h.to(DEV).to(dtype).contiguous(), None, y)
    err = (y.double().cpu() - want).abs().amax(-1) / want.abs().max()
    # a choice that is closer than rounding may fall the other way in bfloat16
    assert float((err <= (2e-5 if dtype == torch.float32 else 2e-2)).double().mean()) >= (1.0 if dtype == torch.float32 else 0.95)
    one = torch.ones(1, hidden, dtype=torch.float32, device=DEV)
    part.forward(h[:1].to(DEV).to(dtype).contiguous(), None, one)
    again = torch.empty_like(one)
    part.forward(h[:1].to(DEV).to(dtype).contiguous(), None, again, overwrite=True)
    close(one.double().cpu() - 1.0, again.double().cpu(), dtype, "added and stored", tol=1e-5)


# ---- around the layers --------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [6, 60, 1028, 1030, 4096, 6000, 9001, 16384])
def test_input_addition_and_the_next_norm(hidden, dtype):
    """Ahead of the first pass the step alone, ahead of the others the embedding's rows too; the next block's first norm in the same
    kernel, or nothing if there is none."""
    block = part_class("block", "input_addition")(LayerSpec("input_addition", {}, {"hidden_size": hidden, "passes": 3, "steps": "s"}))
    norm = build_part("norm", PartSpec("layer_norm", {"size": hidden, "eps": 1e-3, "tensor": "n.norm1", "bias": "n.norm1.b"}, "n"))
    w = draw(block.tensor_specs() + norm.tensor_specs(), 5)
    ctx = ctx_for(dtype)
    block.bind(handles(w), ctx)
    norm.bind(handles(w), ctx)
    g = torch.Generator().manual_seed(hidden)
    x, x0 = torch.randn(7, hidden, generator=g) + 2.0, torch.randn(7, hidden, generator=g)
    for visit in range(3):
        for nxt in (norm, None):
            batch = pack_step([StepEntry(0, [0] * 7, [])], [0], 1, DEV)
            batch.visit, batch.embedding_output, batch.next_first_norm = visit, x0.to(DEV), nxt
            xd = x.to(DEV)
            block.forward(xd, batch, None)
            want = x.double() + w["s"].double()[visit] + (x0.double() if visit else 0.0)
            close(xd.double().cpu(), want, torch.float32, "rows", tol=1e-6)
            assert (batch.normed_carry is None) == (nxt is None)
            if nxt is not None:
                assert batch.normed_carry[1] is norm
                close(batch.normed_carry[0].double().cpu(), plain.layer_norm(want, w["n.norm1"], w["n.norm1.b"], 1e-3), dtype, "normed",
                      tol=5e-6 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", range(4))
def test_block_with_a_multiplier(which, dtype):
    """Norms around both sub-layers, with biases, times the model's multiplier; a layer without a feed-forward."""
    hidden, layer = (DIFFERENTIAL[0], MATRIX[0], PARALLEL[0], DIFFERENTIAL[3])[which]
    layer = dict(layer, mlp=None if which == 3 else moe(3, 3, 24, 16, None, 1.5))
    for mult in (0.37, 1.0, 2.0):
        spec = layer_spec(layer, hidden, mult)
        block = part_class("block", spec.block)(spec)
        w = draw(block.tensor_specs(), 2)
        block.bind(handles(w), ctx_for(dtype))
        cache = cb.SequenceCache([block.cache_requirement()], 1, 256, 256, dtype, DEV)
        T = 90
        x = torch.randn(T, hidden, generator=torch.Generator().manual_seed(4)).float()
        norm = lambda n, v: plain.layer_norm(v, w[f"l0.{n}"], w[f"l0.{n}.b"], EPS)
        want = x.double() + mult * norm("norm1b", plain.mix(norm("norm1", x.double()), w, "l0.mix", layer, EPS))
        if layer["mlp"] is not None:
            want = want + mult * norm("norm2b", plain.moe(norm("norm2", want), w, "l0.mlp", layer["mlp"]))
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
    base = dict(hidden_size=32, heads=2, dim=16, scale=1.0, diff=0.5, eps=1e-5)
    for edit, match in ((dict(rot_dims=18), "rotated"), (dict(rot_layout="thirds"), "layout"), (dict(gate="elements"), "gate"), (dict(dim=130), "exceed"),
                        (dict(kv_heads=3), "multiple"), (dict(window=0), "window")):
        with pytest.raises(cb.CitlaliError, match=match):
            build_part("mixer", PartSpec("differential_attention", dict(base, **edit), "m"))
    base = dict(hidden_size=32, heads=2, dim=16, norm_eps=1e-5, gate_cap=3.0)
    for edit, match in ((dict(decay=[0.5, 0.5]), "either"), (dict(gate_cap=None), "either"), (dict(gate_cap=None, decay=[0.5]), "decays"),
                        (dict(norm_over="group"), "norm_over"), (dict(act="relu"), "act"), (dict(dim=300), "exceeds"), (dict(gate_cap=-1.0), "positive")):
        with pytest.raises(cb.CitlaliError, match=match):
            build_part("mixer", PartSpec("linear_memory", dict(base, **edit), "m"))
    base = dict(hidden_size=32, experts=4, top=2, intermediate_size=8)
    for edit, match in ((dict(activation="relu_squared", weight_on="input"), "output"), (dict(group_score="mean"), "group_score")):
        with pytest.raises(cb.CitlaliError, match=match):
            build_part("feed_forward", PartSpec("routed_experts", dict(base, **edit), "f"))
