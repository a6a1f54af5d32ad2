"""The fast attention kernels with everything at once (soft cap, sinks, outputs turned back in both layouts, gates, key and
value sizes that differ), kernel by kernel against the same formulas in float64 on the bfloat16 numbers they read: split-context
decoding of a few rows and of many rows of very unequal lengths, the prompt kernels on prompts and on runs behind a past, with
windows and without, with scores that run away from a row's first reference, over pages in a shuffled order with junk in unused
places."""
import random

import pytest
import torch

import plain_nomutar as plain
from citlali_b200 import ops
from citlali_b200.cache import KVRequirement, KVView
from citlali_b200.engine.step import StepEntry, pack_step

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
PAGE = 64


def build(sequences, nq, nkv, d, vd, seed, q_size=1.0, k_size=1.0):
    """``sequences``: [(past, new)].  Random pools whose unused places hold junk; a batch; queries, and the visible keys and values
    of every sequence in order, as float64."""
    g = torch.Generator().manual_seed(seed)
    need = [(p + n + PAGE - 1) // PAGE for p, n in sequences]
    pages = list(range(sum(need) + 3))
    random.Random(seed).shuffle(pages)
    keys = torch.full((len(pages), nkv, PAGE, d), 1e4)
    values = torch.full((len(pages), nkv, PAGE, vd), float("inf"))
    values[:] = -3e4
    table = torch.zeros((len(sequences) + 2, max(need) + 1), dtype=torch.int32)
    ks, vs, at = [], [], 0
    for s, (p, n) in enumerate(sequences):
        k = (k_size * torch.randn(p + n, nkv, d, generator=g)).to(torch.bfloat16)
        v = torch.randn(p + n, nkv, vd, generator=g).to(torch.bfloat16)
        ks.append(k.double())
        vs.append(v.double())
        for i in range(need[s]):
            page = pages[at]
            at += 1
            table[s + 1, i] = page
            part = slice(i * PAGE, min((i + 1) * PAGE, p + n))
            keys[page, :, :part.stop - part.start] = k[part].float().transpose(0, 1)
            values[page, :, :part.stop - part.start] = v[part].float().transpose(0, 1)
    kv = KVView(keys.to(torch.bfloat16).to(DEV), values.to(torch.bfloat16).to(DEV), table.to(DEV), PAGE, KVRequirement(nkv, d, value_dim=vd))
    batch = pack_step([StepEntry(s + 1, [0] * n, []) for s, (_, n) in enumerate(sequences)], [p for p, _ in sequences], 1, DEV)
    q = (q_size * torch.randn(batch.rows, nq * d, generator=g)).to(torch.bfloat16)
    return kv, batch, q, ks, vs


def options(rows, nq, vd, seed, cap, with_sink, layout, with_gate):
    g = torch.Generator().manual_seed(seed)
    opt = {"softcap": cap, "sink": torch.randn(nq, generator=g) * 2.0 if with_sink else None, "turns": None, "turn_pairs": layout == "pairs", "gate": None}
    if layout is not None:
        a = 6.0 * torch.rand(rows, vd // 2, generator=g)
        opt["turns"] = torch.stack([torch.cos(a), torch.sin(a)], -1).float().contiguous()
    if with_gate:
        opt["gate"] = torch.randn(rows, nq * vd + 8, generator=g).float()[:, 4:4 + nq * vd]
    return opt


def on_device(opt):
    out = dict(opt)
    for n in ("sink", "turns"):
        out[n] = None if opt[n] is None else opt[n].float().to(DEV)
    if opt["gate"] is not None:
        wide = torch.zeros(opt["gate"].shape[0], opt["gate"].shape[1] + 8, device=DEV)
        wide[:, 4:-4] = opt["gate"].to(DEV)
        out["gate"] = wide[:, 4:-4]
    return out


def reference(sequences, q, ks, vs, nq, nkv, d, vd, window, scale, opt):
    outs, row = [], 0
    for s, (p, n) in enumerate(sequences):
        T = p + n
        see = plain.visible(T, window)[p:]
        o = torch.empty(n, nq, vd, dtype=torch.float64)
        qs = q[row:row + n].double().view(n, nq, d)
        for h in range(nq):
            g = h // (nq // nkv)
            sc = qs[:, h] @ ks[s][:, g].T * scale
            if opt["softcap"]:
                sc = plain.soft_cap(sc, opt["softcap"])
            o[:, h] = plain.weights_with_sink(sc, see, None if opt["sink"] is None else float(opt["sink"][h])) @ vs[s][:, g]
        if opt["turns"] is not None:
            c, sn = opt["turns"][row:row + n, None, :, 0].double(), opt["turns"][row:row + n, None, :, 1].double()
            iu = torch.arange(0, vd, 2) if opt["turn_pairs"] else torch.arange(vd // 2)
            iv = iu + 1 if opt["turn_pairs"] else iu + vd // 2
            u, v = o[..., iu], o[..., iv]
            o = o.clone()
            o[..., iu], o[..., iv] = u * c + v * sn, v * c - u * sn
        o = o.reshape(n, nq * vd)
        if opt["gate"] is not None:
            o = o * torch.sigmoid(opt["gate"][row:row + n].double())
        outs.append(o)
        row += n
    return torch.cat(outs)


def agree(got, want, what):
    err, scale = float((got.double().cpu() - want).abs().max()), float(want.abs().max())
    assert err <= 1.5e-2 * scale, f"{what}: {err:.3e} of {scale:.3e}"
    each = (got.double().cpu() - want).pow(2).mean(-1).sqrt() / (want.pow(2).mean(-1).sqrt() + 1e-3 * scale)
    assert float(each.max()) <= 2e-2, f"{what}: a row is off by {float(each.max()):.3e}"


SIZES = [(8, 2, 128, 128), (6, 2, 96, 80), (4, 4, 64, 64), (5, 1, 40, 24), (4, 2, 256, 136), (34, 2, 16, 16), (4, 1, 48, 112)]
EVERYTHING = [(0.0, True, None, False), (5.0, True, "halves", True), (60.0, False, "pairs", False), (0.0, False, "halves", True), (90.0, True, "halves", False)]


@pytest.mark.parametrize("nq,nkv,d,vd", SIZES)
@pytest.mark.parametrize("window", [None, 1, 64, 100, 1000])
def test_decoding(nq, nkv, d, vd, window):
    """One row, a few rows (clusters merge them), and many rows of very unequal lengths (a long row is dealt to several blocks)."""
    rng = random.Random(nq + d)
    for rows, longest in ((1, 3000), (7, 700), (100, 60)):
        sequences = [(rng.randrange(longest), 1) for _ in range(rows)]
        sequences[0] = (longest - 1, 1)
        sequences[-1] = (0 if rows > 1 else longest, 1)
        if rows == 100:
            sequences[3], sequences[50] = (2600, 1), (1900, 1)
        kv, batch, q, ks, vs = build(sequences, nq, nkv, d, vd, rows + d)
        cap, sink, layout, gate = EVERYTHING[(rows + d + (window or 0)) % len(EVERYTHING)]
        opt = options(rows, nq, vd, d, cap, sink, layout, gate)
        out = torch.empty(rows, nq * vd, dtype=torch.bfloat16, device=DEV)
        ops.attention_decode_with(q.to(DEV), kv, batch, out, nq, nkv, d, vd, window, 2.0 / d ** 0.5, **on_device(opt))
        agree(out, reference(sequences, q, ks, vs, nq, nkv, d, vd, window, 2.0 / d ** 0.5, opt), f"{rows} rows of up to {longest}")


@pytest.mark.parametrize("nq,nkv,d,vd", SIZES + [(3, 1, 128, 128), (4, 4, 128, 128)])
@pytest.mark.parametrize("window", [None, 1, 70, 300])
def test_prompts(nq, nkv, d, vd, window):
    sequences = [(0, 330), (200, 140), (0, 1), (77, 65), (63, 2)]
    kv, batch, q, ks, vs = build(sequences, nq, nkv, d, vd, d)
    dev_q = q.to(DEV)
    common = lambda opt: dict(on_device(opt))
    for k, (cap, sink, layout, gate) in enumerate(EVERYTHING):
        opt = options(batch.rows, nq, vd, d + k, cap, sink, layout, gate)
        want = reference(sequences, q, ks, vs, nq, nkv, d, vd, window, 2.0 / d ** 0.5, opt)
        args = (dev_q, nq * d, kv.keys, kv.values, kv.page_table, batch.seq_start, batch.seq_slot, batch.seq_past)
        out = torch.zeros(batch.rows, nq * vd, dtype=torch.bfloat16, device=DEV)
        ops.attention_prefill(*args, out, batch.sequences, batch.max_new, nq, nkv, d, PAGE, window, 2.0 / d ** 0.5, value_dim=vd, **common(opt))
        agree(out, want, f"prompt kernel {k}")
        if d == vd == 128:
            out = torch.zeros(batch.rows, nq * vd, dtype=torch.bfloat16, device=DEV)
            flag = torch.zeros(4, dtype=torch.int32, device=DEV)
            ops.attention_prefill_tc(*args, out, batch.sequences, batch.max_new, nq, nkv, d, PAGE, window, 2.0 / d ** 0.5, flag, **common(opt))
            agree(out, want, f"prompt kernel with tiles in tensor memory {k}")
            assert not any(flag.tolist())


@pytest.mark.parametrize("cap", [0.0, 50.0, 69.0, 80.0])
def test_scores_far_from_a_rows_first_reference(cap):
    """Keys that grow along the sequence: a row's scores run from near zero to hundreds (capped: to the cap and to minus the
    cap), so that references move, or, under a cap that needs none, weights span the whole range."""
    nq, nkv, d, T = 4, 2, 128, 520
    sequences = [(0, T)]
    kv, batch, q, ks, vs = build(sequences, nq, nkv, d, d, 3)
    grow = torch.linspace(0.1, 6.0, T)[:, None, None].double()
    ks[0] = (ks[0] * grow).to(torch.bfloat16).double()
    for i in range((T + PAGE - 1) // PAGE):
        part = ks[0][i * PAGE:(i + 1) * PAGE]
        kv.keys[int(kv.page_table[1, i]), :, :part.shape[0]] = part.transpose(0, 1).to(torch.bfloat16).to(DEV)
    opt = options(T, nq, d, 5, cap, True, "halves", False)
    want = reference(sequences, q, ks, vs, nq, nkv, d, d, None, 1.0, opt)
    out = torch.zeros(T, nq * d, dtype=torch.bfloat16, device=DEV)
    flag = torch.zeros(4, dtype=torch.int32, device=DEV)
    ops.attention_prefill_tc(q.to(DEV), nq * d, kv.keys, kv.values, kv.page_table, batch.seq_start, batch.seq_slot, batch.seq_past, out, 1, T, nq,
                             nkv, d, PAGE, None, 1.0, flag, **on_device(opt))
    agree(out, want, f"cap {cap}")
    assert not any(flag.tolist())
    # all of a row's scores at minus the cap: nothing underflows to an empty sum
    if cap:
        opt = options(T, nq, d, 5, cap, False, None, False)
        low = -q.to(DEV).abs()
        kv.keys.copy_(kv.keys.abs())
        kabs = [ks[0].abs()]
        ops.attention_prefill_tc(low, nq * d, kv.keys, kv.values, kv.page_table, batch.seq_start, batch.seq_slot, batch.seq_past, out, 1, T, nq, nkv,
                                 d, PAGE, None, 50.0, flag, **on_device(opt))
        agree(out, reference(sequences, low.cpu(), kabs, vs, nq, nkv, d, d, None, 50.0, opt), f"all at minus {cap}")
