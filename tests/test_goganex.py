"""Goganex against the plain statement in ``plain_goganex.py``: every mechanism alone, whole prompts, portions, single tokens,
mixed batches on reused pages and slots, and greedy generation through the rollout engine.

Every case runs on the CPU ops, and on a GPU in 32-bit and bf16 (weights and inputs are bf16 values, so the oracle sees
the same numbers)."""
import json
import random

import pytest
import torch

from areal_b200.engine.ragged_step import Entry
from areal_b200.engine.state_cache import StateCache
from areal_b200.models import hf_io, mixers
from areal_b200.models.config import ModelConfig, preset
from areal_b200.models.decoder import build_model
from areal_b200.ops import functional as OF
from areal_b200.ops import mixer_ops as M

from . import plain_goganex as plain
from .test_bumotar import make_table, page_rows
from .test_mixer_stack import (TARGETS, Driver, _one_thread, assert_close, bf16_values, dev, f32, generate, make_engine,  # noqa: F401
                               make_model, ragged, tokens)


def rot(dims, base=300.0, **scaling):
    return dict(base=base, dims=dims, scaling=scaling) if scaling else dict(base=base, dims=dims)


def llama3(dims, base=200.0, factor=5.0, low=1.0, high=3.0, original=90):
    """Scaled so that short prompts have pairs that are kept, blended and slowed."""
    return rot(dims, base, factor=factor, low=low, high=high, original=original)


def att(heads=4, kv=2, dim=32, vdim=32, peak=1.7, turn=None):
    """``peak``: standard deviation of the scores under random weights; wide scores make every key count."""
    return "attention", dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=peak * dim ** -0.5, rot=turn or llama3(dim // 2))


def par(heads=6, kv=2, dim=24, width=40, peak=1.7):
    return "parallel", dict(left=dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=peak * dim ** -0.5), right=dict(width=width))


def dense(ff=80, limit=1.2):
    return dict(kind="dense", ff=ff, limit=limit)


def config(*layers, vocab=104, width=64, loop=(0, 2, 2), eps=1e-5, scale=0.6):
    return dict(architecture="Goganex", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale),
                loop=dict(start=loop[0], stop=loop[1], times=loop[2]) if loop else None,
                layers=[dict(type=t, mixer=m, mlp=f) for (t, m), f in layers])


CONFIGS = {
    "mixed": config((att(), dense()), (par(), dense(72, 0.8)), (par(heads=4, kv=4, dim=32, width=64), None)),
    # sizes that no vector width divides; what runs before, in and after the loop; three passes; an epsilon that counts
    "odd": config((att(heads=3, kv=1, dim=20, vdim=12, turn=llama3(6)), dense(33)), (par(heads=6, kv=3, dim=22, width=35), None),
                  (att(heads=6, kv=2, dim=14, vdim=18, turn=rot(14)), dense(20, 3.0)), vocab=101, width=60, loop=(1, 2, 3), eps=1e-2),
    # more than a tile of heads per key head, values wider than keys, widths of several tiles, a loop of one pass
    "wide": config((att(heads=17, kv=1, dim=64, vdim=96, turn=llama3(64)), dense(96)), (par(heads=20, kv=4, dim=96, width=200), dense(40)),
                   width=128, vocab=96, loop=(1, 2, 1), scale=1.0),
    "dim128": config((par(heads=2, kv=1, dim=128, width=8), dense(64)), (att(heads=2, kv=2, dim=128, vdim=128, turn=llama3(128)), dense(64)), loop=(1, 2, 2), scale=2.5),
    # no loop, parallel branches first and last, a key head per query head, small and very large heads, few channels
    "edges": config((par(heads=3, kv=3, dim=8, width=10), dense(16)), (att(heads=2, kv=1, dim=136, vdim=24, turn=rot(100)), None),
                    (att(heads=2, kv=2, dim=8, vdim=40, turn=llama3(2)), dense()), (par(heads=2, kv=1, dim=136, width=130), dense(24)), width=40, loop=None),
}


def make_weights(cfg, seed=0):
    """Random weights under the checkpoint's names (float64 holding bf16 values)."""
    g = torch.Generator().manual_seed(seed)
    H, V = cfg["width"], cfg["vocab"]
    W = {"embed": bf16_values((V, H), g, 1 / cfg["embedding"]["scale"]), "head": bf16_values((V, H), g, 2 * H ** -0.5), "final.norm": bf16_values((H,), g, 0.2, 1.0)}

    def mat(name, *shape, std=1.0):
        W[name] = bf16_values(shape, g, std * shape[-1] ** -0.5)

    def vec(name, n, std=0.2, mean=1.0):
        W[name] = bf16_values((n,), g, std, mean)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        for n in ("norm1", "norm2") if layer["mlp"] else ("norm1",):
            vec(f"l{i}.{n}", H)
        W[f"l{i}.shift"] = torch.rand(H, generator=g, dtype=torch.float64).bfloat16().double()
        if layer["type"] == "attention":
            mat(p + "q", m["heads"] * m["dim"], H), mat(p + "k", m["kv_heads"] * m["dim"], H), mat(p + "v", m["kv_heads"] * m["vdim"], H)
            mat(p + "o", H, m["heads"] * m["vdim"]), vec(p + "temp", m["heads"], 0.4)
        else:
            a, w = m["left"], m["right"]["width"]
            mat(p + "left.q", a["heads"] * a["dim"], H), mat(p + "left.k", a["kv_heads"] * a["dim"], H), mat(p + "left.o", H, a["heads"] * a["dim"])
            for n in ("z", "x", "g"):
                mat(f"{p}right.{n}", w, H, std=1.5)
            mat(p + "right.o", H, w)
            vec(p + "right.z.b", w, 1.0, -1.5), vec(p + "right.x.b", w, 0.5, 0.0)
            vec(p + "left.out", H), vec(p + "right.out", H)
        f, p = layer["mlp"], f"l{i}.mlp."
        if f:
            mat(p + "gate", f["ff"], H, std=1.5), mat(p + "up", f["ff"], H, std=1.5), mat(p + "down", H, f["ff"])
    return W


_ORACLE: dict = {}


def oracle(name, n, seed):
    """Tokens, logits and residual streams of a random prompt under a named configuration (cached: shared by the targets and
    the schedules)."""
    if (name, n, seed) not in _ORACLE:
        cfg = CONFIGS[name]
        t = tokens(n, cfg["vocab"], seed)
        _ORACLE[name, n, seed] = (t, *plain.forward(make_weights(cfg), cfg, t))
    return _ORACLE[name, n, seed]


# ----------------------------------------------------------------------------- schedules
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_portions_and_single_tokens_agree(name, target):
    cfg = CONFIGS[name]
    eng = make_engine(cfg, make_weights(cfg), target)
    n = 150
    t, want, _ = oracle(name, n, 1)
    cuts = {"whole": [n], "decoded": [90] + [1] * 60, "pairs": [2] * 35 + [80], "ragged": [1, 2, 61, 3, 64, 2, 1, 16]}
    for what, sizes in cuts.items():
        d, at = Driver(eng), 0
        assert sum(sizes) == n
        for s in sizes:
            d.step([("a", t[at:at + s])], end=["a"] if at + s == n else [])
            at += s
        assert_close(d.logits("a"), want, target[1], f"{name} {what}")
    assert len(eng.cache.free) == eng.cache.num_pages and len(eng.cache.free_slots) == eng.cache.num_slots


@pytest.mark.parametrize("target", TARGETS)
def test_long_prompt_and_long_decoding(target):
    """Several blocks and query tiles in one portion; a state and keys that are carried over 200 single tokens."""
    name, n = "wide", 620
    cfg = CONFIGS[name]
    t, want, _ = oracle(name, n, 2)
    eng = make_engine(cfg, make_weights(cfg), target)
    d = Driver(eng)
    d.step([("a", t)], end=["a"])
    assert_close(d.logits("a"), want, target[1], "whole")
    d = Driver(eng)
    d.step([("a", t[:270])])
    for i in range(270, 420):
        d.step([("a", t[i:i + 1])])
    d.step([("a", t[420:570])])
    for i in range(570, n):
        d.step([("a", t[i:i + 1])], end=["a"] if i == n - 1 else [])
    assert_close(d.logits("a"), want, target[1], "decoded")


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("page_size", [16, 64])
def test_mixed_batches_on_reused_pages_and_slots(target, page_size):
    """Seven requests over three slots and a pool that holds only what is live: portions beside single tokens, requests
    that pause, pages and slots that change hands. Each must see what it would see alone."""
    name = "mixed"
    cfg = CONFIGS[name]
    lens = {f"r{i}": n for i, n in enumerate([130, 7, 97, 1, 64, 49, 33])}
    ref = {rid: oracle(name, n, 10 + i) for i, (rid, n) in enumerate(lens.items())}
    eng = make_engine(cfg, make_weights(cfg), target, pages=6 * 64 // page_size, page_size=page_size, slots=4)
    d, rnd = Driver(eng), random.Random(4)
    waiting, live, at = list(lens), [], {rid: 0 for rid in lens}
    while waiting or live:
        while waiting and len(live) < 3:
            live.append(waiting.pop(0))
        portions = []
        for rid in live:
            if rnd.random() < 0.2 and len(live) > 1:
                continue                             # left out of this step
            s = min(rnd.choice([1, 1, 1, 2, 3, 17, 40]), lens[rid] - at[rid])
            portions.append((rid, ref[rid][0][at[rid]:at[rid] + s]))
            at[rid] += s
        if not portions:
            continue
        done = [rid for rid, _ in portions if at[rid] == lens[rid]]
        d.step(portions, end=done)
        live = [r for r in live if r not in done]
    for rid in lens:
        assert_close(d.logits(rid), ref[rid][1], target[1], rid)
    assert len(eng.cache.free) == eng.cache.num_pages


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_layer_outputs_match(name, target):
    """Every run of a layer, looped ones once per pass."""
    cfg = CONFIGS[name]
    t, _, states = oracle(name, 70, 5)
    eng = make_engine(cfg, make_weights(cfg), target)
    c, seen = eng.cache.open(), []
    eng.cache.grow(c, 70)
    eng.runner.step([Entry(c, t, [69])], on_layer=lambda i, r: seen.append(r.double().cpu().clone()))
    assert len(seen) == len(states) == len(eng.cache.layers) == len(eng.model.layer_runs)
    for i, (a, b) in enumerate(zip(seen, states)):
        assert_close(a, b, target[1], f"layer run {i}")


@pytest.mark.parametrize("target", [TARGETS[0], TARGETS[1]])
def test_a_far_token_reaches_the_last_one(target):
    """The first token alone tells two prompts apart; what is left of it 300 tokens later is the same however they were cut."""
    name, n = "mixed", 300
    cfg = CONFIGS[name]
    W = make_weights(cfg, 6)
    t = tokens(n, cfg["vocab"], 6)
    other = [(t[0] + 50) % cfg["vocab"]] + t[1:]
    a, b = (plain.forward(W, cfg, x)[0][-1] for x in (t, other))
    apart = (a - b).pow(2).mean().sqrt()
    eng = make_engine(cfg, W, target)
    got = []
    for x, cut in ((t, [n]), (other, [1] * 3 + [2] * 100 + [97])):
        d, at = Driver(eng), 0
        for s in cut:
            d.step([("a", x[at:at + s])], end=["a"] if at + s == n else [])
            at += s
        got.append(d.logits("a")[-1])
    assert apart > 0.01 and (got[0] - got[1] - (a - b)).pow(2).mean().sqrt() < 0.02 * apart


# what each mechanism would be if it were read wrongly; the logits under the tests' weights must tell
FAULTS = {
    "no shift": ("shifted", lambda h, s: h),
    "shift the other way round": ("shifted", lambda h, s: plain.previous(h) + (h - plain.previous(h)) * s),
    "the row before taken after its own shift": ("shifted", lambda h, s: (lambda out: [out.append(r + ((out[-1] if out else 0 * r) - r) * s) for r in h] and torch.stack(out))([])),
    "the first token shifted by itself": ("previous", lambda h: torch.cat([h[:1], h[:-1]])),
    "halves turned instead of neighbours": ("pairs", lambda d: [(i, i + d // 2) for i in range(d // 2)]),
    "frequencies not scaled": ("scaled_frequencies", lambda r: plain.base_frequencies(r)),
    "every frequency slowed": ("scaled_frequencies", lambda r: [f / r["scaling"]["factor"] for f in plain.base_frequencies(r)]),
    "no blend between kept and slowed": ("scaled_frequencies", lambda r, f=plain.scaled_frequencies: f(dict(r, scaling=dict(r["scaling"], low=r["scaling"]["high"])))),
    "nothing added to the denominator": ("SINK", 0.0),
    "queries and keys not normed": ("unit", lambda x, eps: x),
    "no factor per head": ("attend", lambda q, k, v, s, t, e, f=plain.attend: f(q, k, v, s, torch.ones_like(t), e)),
    "one added to every denominator": ("attend", lambda q, k, v, s, t, e, f=plain.attend: f(q, k, v, s, t, 1.0)),
    "values normed like the keys": ("values_of", lambda k, eps: plain.unit(k, eps)),
    "the first token unseen": ("first_visible", lambda i: min(i, 1)),
    "candidate sigmoid everywhere": ("candidate", lambda u: plain.sigmoid(u)),
    "candidate the projection itself": ("candidate", lambda u: u),
    "gate kept instead of taken": ("recur", lambda z, c, f=plain.recur: f(1 - z, c)),
    "state read before the token": ("recur", lambda z, c, f=plain.recur: torch.cat([torch.zeros_like(z[:1]), f(z, c)[:-1]])),
    "no recurrence": ("recur", lambda z, c: z * c),
    "sum instead of half the sum": ("join", lambda a, b: a + b),
    "gate not limited": ("clipped", lambda g, u, m: (g, u.clamp(-m, m))),
    "gate limited below too": ("clipped", lambda g, u, m: (g.clamp(-m, m), u.clamp(-m, m))),
    "up not limited below": ("clipped", lambda g, u, m: (g.clamp(max=m), u.clamp(max=m))),
    "embedding not scaled": ("embed", lambda W, c, t: W["embed"][torch.as_tensor(t)]),
    "one pass too few": ("runs", lambda c, f=plain.runs: f(dict(c, loop=dict(c["loop"], times=1)))),
}
FAINT = {"gate limited below too", "the first token shifted by itself", "the first token unseen", "one added to every denominator"}   # tell most at some tokens


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_a_wrong_reading_shows_in_the_logits(fault, monkeypatch):
    """Planted in the plain statement: no mechanism is drowned by the random weights of the other tests (whose rows may be off
    by 0.0002 in 32-bit and by 0.06 in bf16)."""
    name, fn = FAULTS[fault]
    t, want, _ = oracle("mixed", 130, 10)
    monkeypatch.setattr(plain, name, fn)
    cfg = CONFIGS["mixed"]
    got = plain.forward(make_weights(cfg), cfg, t)[0]
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert err.max() > 0.1 and err.median() > (0.002 if fault in FAINT else 0.02), (float(err.median()), float(err.max()))


# ----------------------------------------------------------------------------- rotation, norms, cache
@pytest.mark.parametrize("r", [llama3(16), llama3(64, 500000.0, 8.0, 1.0, 4.0, 8192), llama3(8, 50.0, 2.0, 0.001, 0.002, 20), llama3(32, 1e4, 8.0, 1.0, 2.0, 3),
                               llama3(24, 300.0, 4.0, 2.0, 2.0, 50), rot(12)])
def test_frequencies_by_wavelength(r):
    """With pairs kept, blended and slowed, all kept, all slowed, no stretch between the two, and without scaling."""
    got, want = mixers.llama3_frequencies(r), plain.scaled_frequencies(r)
    assert got[1] == 1.0 and torch.allclose(torch.tensor(got[0]).double(), torch.tensor(want).double(), rtol=1e-12)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("Hq,Hkv,D,Dv,dims", [(4, 2, 32, 48, 16), (3, 1, 22, 10, 6), (9, 9, 128, 64, 128), (2, 1, 136, 24, 100), (5, 5, 7, 3, 2), (3, 1, 24, 8, 0)])
def test_heads_are_turned_brought_to_unit_length_and_scaled(Hq, Hkv, D, Dv, dims, target):
    g = torch.Generator().manual_seed(D)
    b, _, rows = ragged([1, 20], [133, 7], target[0])
    n = Hq * D + Hkv * (D + Dv)
    z, factor = bf16_values((21, n + 8), g, 2.0), bf16_values((Hq,), g, 0.5, 1.0)
    z[5] = (z[5] * 1e-3).bfloat16().double()           # where the epsilon counts
    kc, vc = (torch.full((rows, Hkv, d), 9.0, dtype=target[1], device=target[0]) for d in (D, Dv))
    freqs = plain.base_frequencies(rot(dims)) if dims else []
    pos = b.pos.cpu().tolist()
    b.slots[3] = -1                                    # a padding row leaves the cache alone
    table = make_table(freqs, 1.0, b.pos, target[0]) if dims else None
    q = M.qk_head_norm_append(dev(z, target), None, None, 1e-4, table, True, b, kc, vc, Hq, unit=True, q_factor=f32(factor, target)).double().cpu()
    tol = 2e-5 if target[1] == torch.float32 else 0.02

    def want(x):
        return plain.unit(plain.rotate(x, pos, freqs, plain.pairs(dims)), 1e-4)
    wq, wk = want(z[:, :Hq * D].view(21, Hq, D)) * factor[:, None], want(z[:, Hq * D:(Hq + Hkv) * D].view(21, Hkv, D))
    assert (q - wq).abs().max() < tol * wq.abs().max()
    at, keep = b.slots.long().cpu(), [i for i in range(21) if i != 3]
    assert (kc.double().cpu()[at[keep]] - wk[keep]).abs().max() < tol * wk.abs().max()
    assert torch.equal(vc.double().cpu()[at[keep]], z[keep, (Hq + Hkv) * D:n].view(-1, Hkv, Dv))
    assert (vc == 9.0).flatten(1).all(-1).sum() == rows - 20


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("Hq,Hkv,D", [(4, 2, 32), (3, 1, 22), (9, 3, 128), (2, 1, 136), (5, 5, 7)])
def test_keys_are_cached_as_they_are_beside_what_norms_them(Hq, Hkv, D, target):
    g = torch.Generator().manual_seed(D)
    b, _, rows = ragged([1, 20], [133, 7], target[0])
    z = bf16_values((21, (Hq + Hkv) * D + 8), g, 2.0)
    z[5] = (z[5] * 1e-3).bfloat16().double()
    kc = torch.full((rows, Hkv, D), 9.0, dtype=target[1], device=target[0])
    kf = torch.full((rows, Hkv), 9.0, dtype=torch.float32, device=target[0])
    b.slots[3] = -1
    q = M.qk_head_norm_append(dev(z, target), None, None, 1e-4, None, False, b, kc, None, Hq, unit=True, key_factor=kf).double().cpu()
    tol = 2e-5 if target[1] == torch.float32 else 0.02
    wq, k = plain.unit(z[:, :Hq * D].view(21, Hq, D), 1e-4), z[:, Hq * D:(Hq + Hkv) * D].view(21, Hkv, D)
    assert (q - wq).abs().max() < tol * wq.abs().max()
    at, keep = b.slots.long().cpu(), [i for i in range(21) if i != 3]
    assert torch.equal(kc.double().cpu()[at[keep]], k[keep])
    want = 1 / plain.rms(k, 1e-4)[..., 0]
    assert ((kf.double().cpu()[at[keep]] - want[keep]) / want[keep]).abs().max() < 1e-5       # 32-bit whatever the activations are
    assert (kf == 9.0).all(-1).sum() == rows - 20 and (kc == 9.0).flatten(1).all(-1).sum() == rows - 20


# ----------------------------------------------------------------------------- attention
SCHEDULES = (([1, 1, 1, 1, 130, 300, 2], [0, 47, 333, 90, 0, 70, 118]), ([1, 2, 9, 16], [80, 62, 300, 0]))


def stand_out(q, key, L, n, s, gain):
    """For some queries one key stands out: the first ones, their own, at page and tile borders, far away."""
    for i in {L - 1, L - 2, s, s + n // 2, min(L - 1, 63), min(L - 1, 64), min(L - 1, 127), min(L - 1, 128)}:
        for j in (0, 1, i, i // 16 * 16, i // 16 * 16 - 1, i // 64 * 64, i // 64 * 64 - 1, i // 2):
            if 0 <= j <= i and (i * 7 + j * 3) % 4 == 0:
                k = key(j)
                q[i] = (k / k.norm(dim=-1, keepdim=True) * gain).bfloat16().double()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("Hq,Hkv,D,Dv,values,sink", [(4, 2, 32, 48, True, 0.0), (6, 2, 96, 64, True, 0.0), (20, 1, 64, 128, True, 0.0), (3, 1, 20, 12, True, 0.0),
                                                     (4, 2, 32, 32, False, None), (16, 1, 128, 128, False, None), (34, 2, 96, 96, False, None), (6, 3, 8, 8, False, 1.0),
                                                     (3, 3, 22, 22, False, None), (2, 1, 136, 136, False, None), (40, 20, 64, 64, False, None)])
def test_attention_over_everything_before(Hq, Hkv, D, Dv, values, sink, target):
    """With values of their own and one more in the denominator; and with keys that are the values, of very different lengths, which
    only their factors bring to one length in the scores."""
    g = torch.Generator().manual_seed(D + Dv)
    tol, scale, ones = 1e-4 if target[1] == torch.float32 else 0.04, D ** -0.5, torch.ones(Hq, dtype=torch.float64)
    for lens, starts in SCHEDULES:
        b, entries, rows = ragged(lens, starts, target[0])
        kc, vc = torch.zeros(rows, Hkv, D, dtype=target[1], device=target[0]), torch.zeros(rows, Hkv, Dv, dtype=target[1], device=target[0])
        kf = torch.full((rows, Hkv), 7.0, dtype=torch.float32, device=target[0])
        qs, wants = [], []
        for e, (n, s) in enumerate(zip(lens, starts)):
            L = n + s
            q, k, v = bf16_values((L, Hq, D), g), bf16_values((L, Hkv, D), g), bf16_values((L, Hkv, Dv), g)
            if not values:
                k = (k * torch.exp(torch.randn(L, Hkv, 1, generator=g, dtype=torch.float64))).bfloat16().double()
            keys = k if values else plain.unit(k, 1e-5)
            stand_out(q, lambda j: keys[j].repeat_interleave(Hq // Hkv, 0), L, n, s, 2.5 * D ** 0.5)
            at = page_rows(entries[e], L, target[0])
            kc[at], vc[at] = dev(k, target), dev(v, target)
            kf[at] = f32(1 / plain.rms(k, 1e-5)[..., 0], target)
            qs.append(q[s:])
            wants.append(plain.attend(q, keys, v if values else k, scale, ones, 0.0 if sink is None else torch.exp(torch.tensor(sink, dtype=torch.float64)))[s:])
        q_rows = dev(torch.cat(qs), target).contiguous()
        got = M.chunk_attention(q_rows, kc, vc if values else None, b, scale, sink=sink, key_factor=None if values else kf).double().cpu()
        at = 0
        for e, n in enumerate(lens):
            err = (got[at:at + n] - wants[e]).abs().amax() / wants[e].abs().amax()
            assert err < tol, (e, float(err))
            at += n


@pytest.mark.parametrize("target", TARGETS)
def test_factors_of_keys_go_with_caps_and_distance_biases(target):
    """The plain kernel takes what the tiled one does not; windows and factors go together in both."""
    g = torch.Generator().manual_seed(3)
    lens, starts = [1, 70], [40, 25]
    b, entries, rows = ragged(lens, starts, target[0])
    q, kc, kf = dev(bf16_values((71, 4, 32), g), target), dev(bf16_values((rows, 2, 32), g), target), torch.rand(rows, 2, generator=g).to(target[0]) + 0.5
    r1, r2 = torch.rand(4, generator=g).to(target[0]), torch.rand(4, generator=g).to(target[0])
    folded = (kc.float() * kf[..., None])
    for kw in (dict(), dict(window=30), dict(chunk=24), dict(softcap=4.0), dict(r1=r1, r2=r2), dict(softcap=4.0, r1=r1, r2=r2, chunk=32)):
        got = M.chunk_attention(q, kc, None, b, 0.3, key_factor=kf, **kw).double().cpu()
        args = [kw.get("softcap", 0.0), *(None if x is None else x.cpu() for x in (kw.get("r1"), kw.get("r2"))), kw.get("chunk", 0), kw.get("window", 0)]
        cpu = M.RaggedBatch(*(t.cpu() for t in (b.tokens, b.pos, b.slots, b.row_entry, b.cu, b.start, b.state, b.pages, b.page_base)), None, None, b.n_dec, b.page_size)
        want = M.chunk_attention_ref(q.float().cpu(), folded.cpu(), kc.float().cpu(), cpu, 0.3, *args).double()
        assert (got - want).abs().max() < (1e-4 if target[1] == torch.float32 else 0.04) * want.abs().max(), kw


# ----------------------------------------------------------------------------- recurrence
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("width", [64, 40, 7, 200, 1, 130])
@pytest.mark.parametrize("lens,starts", [([1, 1, 1, 130, 64, 2, 200], [0, 47, 5, 0, 63, 118, 3]), ([1, 700, 513, 2], [9, 0, 20, 0]), ([3, 2, 64], [0, 1, 30])])
def test_min_gru(lens, starts, width, target):
    """Portions and single tokens from carried states, in slots that hold what an earlier request left; gates from nearly shut to
    nearly open. Portions of one block, of several, and of several rounds of blocks, by one CTA and by clusters."""
    g = torch.Generator().manual_seed(width)
    b, entries, _ = ragged(lens, starts, target[0])
    R, bias = sum(lens), bf16_values((2 * width,), g, 1.0)
    S = torch.full((len(lens), width), 3.0, dtype=torch.float32, device=target[0])           # of requests that are gone
    rows, ends, wants = [], [], []
    for e, (n, s) in enumerate(zip(lens, starts)):
        x = bf16_values((n + s, 3 * width), g, 2.0)
        x[:, :width] -= 2.0
        x = x.bfloat16().double()
        states = plain.recur(plain.sigmoid(x[:, :width] + bias[:width]), plain.candidate(x[:, width:2 * width] + bias[width:]))
        if s:
            S[entries[e].carry.slot] = states[s - 1].float().to(target[0])
        rows.append(x[s:]), ends.append(states[-1]), wants.append((states * plain.silu(x[:, 2 * width:]))[s:])
    wide = torch.zeros(R, 3 * width + 9, dtype=target[1], device=target[0])                  # rows of a wider product, not aligned
    wide[:, 1:3 * width + 1] = dev(torch.cat(rows), target)
    for zug, cluster in [(wide[:, 1:3 * width + 1], 0), *((wide[:, 1:3 * width + 1].contiguous(), c) for c in (0, 1, 2, 4, 8))]:
        S2 = S.clone()
        got, at = M.min_gru(zug, f32(bias, target), b, S2, cluster=cluster).double().cpu(), 0
        for e, n in enumerate(lens):
            err = (got[at:at + n] - wants[e]).abs().max() / wants[e].abs().max()
            assert err < (1e-5 if target[1] == torch.float32 else 0.01), (e, float(err))
            # the state is 32-bit whatever the activations are
            st = S2[entries[e].carry.slot].double().cpu()
            assert (st - ends[e]).abs().max() < 1e-5 * ends[e].abs().max(), (e, float((st - ends[e]).abs().max()))
            at += n


@pytest.mark.parametrize("target", TARGETS)
def test_a_shut_gate_keeps_the_state_over_long_decoding(target):
    W = 48
    z = torch.full((421, 3 * W), -20.0, dtype=torch.float64)
    z[0, :2 * W] = 4.0                                 # taken in once, then kept
    z[:, 2 * W:] = 1.0
    S, bias = torch.zeros(1, W, dtype=torch.float32, device=target[0]), torch.zeros(2 * W, device=target[0])
    at, zt = 0, dev(z, target)
    for n in [2] + [1] * 417 + [2]:
        b, _, _ = ragged([n], [at], target[0])
        out = M.min_gru(zt[at:at + n], bias, b, S)
        at += n
    want = float(plain.sigmoid(torch.tensor(4.0, dtype=torch.float64)) * 4.5 * plain.silu(torch.tensor(1.0, dtype=torch.float64)))
    assert at == 421 and (out[-1].double().cpu() - want).abs().max() < (2e-5 if target[1] == torch.float32 else 0.02) * want


# ----------------------------------------------------------------------------- the stream: sums, norms, token shift
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H", [64, 60, 42, 2048, 5120])
@pytest.mark.parametrize("source", ["nothing", "row", "branches", "embedding", "experts"])
def test_what_a_mixer_reads(source, H, target):
    """Sum, norm and shift of every kind of source; portions and single tokens whose row before is in a slot, in the same step, or
    missing, in slots that hold what an earlier request left; a padding entry; with and without the shift."""
    g = torch.Generator().manual_seed(H)
    lens, starts = [1, 1, 1, 1, 130, 64, 2, 9, 65], [0, 47, 5, 8, 0, 63, 118, 0, 3]
    b, entries, _ = ragged(lens, starts, target[0])
    b.state[3] = -1
    R, eps, tol = sum(lens), 1e-3, 1e-5 if target[1] == torch.float32 else 0.02
    resid, w, share, vec = torch.randn(R, H, generator=g, dtype=torch.float64).float().double(), bf16_values((H,), g, 0.3, 1.0), bf16_values((H,), g, 0.5), bf16_values((H,), g)
    wide = bf16_values((R, 2 * H + 8), g, 3.0)
    wt = dev(wide, target)
    start = resid
    if source == "nothing":
        src, add = None, torch.zeros(R, H, dtype=torch.float64)
    elif source == "row":
        src, add = wt[:, 8:8 + H], wide[:, 8:8 + H]
    elif source == "branches":
        wl, wr = bf16_values((H,), g, 0.3, 1.0), bf16_values((H,), g, 0.3, 1.0)
        src = M.BranchSum(wt[:, :H], wt[:, H:2 * H], f32(wl, target), f32(wr, target), 0.5, eps)
        add = 0.5 * (plain.norm(wide[:, :H], wl, eps) + plain.norm(wide[:, H:2 * H], wr, eps))
    elif source == "embedding":
        table, ids = bf16_values((37, H), g), torch.randint(0, 37, (R,), generator=g)
        src, add, start = M.EmbeddingRows(ids.int().to(target[0]), dev(table, target), 0.3), 0.3 * table[ids], None
    else:
        rt = OF.moe_route(torch.randn(R, 4, generator=g).to(target[0]), 2, want_host=False)
        y = bf16_values((2 * R, H), g)
        src, add = M.ExpertSum(dev(y, target), rt, None, rt.topw), (y[rt.inv.long().cpu().view(R, 2)] * rt.topw.double().cpu()[..., None]).sum(1)
    stream = (0.0 if start is None else start) + add
    for shift, v in ((True, None), (True, vec), (False, None), (False, vec)):
        want_s = stream if v is None else stream + v
        h = plain.norm(want_s, w, eps)
        S = torch.full((len(lens), H), 3.0, dtype=torch.float32, device=target[0])
        olds = [bf16_values((H,), g) if s else torch.zeros(H, dtype=torch.float64) for s in starts]
        for e, s in enumerate(starts):
            if s:
                S[entries[e].carry.slot] = f32(olds[e], target)
        before = S.clone()
        r0 = None if start is None else f32(start, target).contiguous()
        got_s, x = M.stream_norm(src, r0, f32(w, target), eps, target[1], None if v is None else f32(v, target), f32(share, target) if shift else None, b, S)
        ok = [i for i in range(R) if i != 3]                # the row of the padding entry may hold anything
        assert got_s.dtype == torch.float32 and (got_s.double().cpu() - want_s)[ok].abs().max() < 1e-5 * want_s.abs().max()
        want, at = h, 0
        if shift:
            want = torch.cat([plain.previous(h[:0])] + [torch.cat([olds[e][None], h[a:a + n - 1]]) for e, (a, n) in enumerate(zip(b.cu.tolist(), lens))])
            want = h + (want - h) * share
        assert x.dtype == target[1] and (x.double().cpu() - want)[ok].abs().max() < tol * want.abs().max()
        for e, n in enumerate(lens):
            at += n
            slot = entries[e].carry.slot
            if e == 3 or not shift:
                assert torch.equal(S[slot], before[slot])
            else:                                          # 32-bit whatever the activations are
                assert (S[slot].double().cpu() - h[at - 1]).abs().max() < 1e-5 * h.abs().max(), e


@pytest.mark.parametrize("target", TARGETS)
def test_shifted_rows_do_not_depend_on_the_cuts(target):
    """One portion, pairs, single tokens: the same numbers to the last bit (every row's sums are made in the same order)."""
    g = torch.Generator().manual_seed(4)
    H, L = 96, 140
    resid, w, share = torch.randn(L, H, generator=g).to(target[0]), torch.rand(H, generator=g).to(target[0]) + 0.5, torch.rand(H, generator=g).to(target[0])
    outs = []
    for cut in ([L], [2] * 70, [1] * 20 + [90] + [1] * 30, [67, 73]):
        S, at, xs = torch.zeros(1, H, device=target[0]), 0, []
        for n in cut:
            b, _, _ = ragged([n], [at], target[0])
            xs.append(M.stream_norm(None, resid[at:at + n].clone(), w, 1e-5, target[1], None, share, b, S)[1])
            at += n
        outs.append((torch.cat(xs), S))
    for x, S in outs[1:]:
        if target[0] == "cuda":
            assert torch.equal(x, outs[0][0]) and torch.equal(S, outs[0][1])
        else:
            assert torch.allclose(x, outs[0][0], atol=1e-6) and torch.allclose(S, outs[0][1], atol=1e-6)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H", [64, 42, 5120])
def test_branches_are_summed_into_the_last_norm(H, target):
    """In place and with the factor of the logits, as behind the last layer."""
    g = torch.Generator().manual_seed(H)
    a, c, wl, wr, w = bf16_values((7, H), g, 3.0), bf16_values((7, H), g, 0.2), *(bf16_values((H,), g, 0.3, 1.0) for _ in range(3))
    resid = torch.randn(7, H, generator=g, dtype=torch.float64).float().double()
    r = f32(resid, target).contiguous()
    x = M.residual_norm(M.BranchSum(dev(a, target), dev(c, target), f32(wl, target), f32(wr, target), 0.5, 1e-3), r, f32(w, target), 1e-3, target[1], mult=0.25)
    want_r = resid + plain.join(plain.norm(a, wl, 1e-3), plain.norm(c, wr, 1e-3))
    want = 0.25 * plain.norm(want_r, w, 1e-3)
    assert (r.double().cpu() - want_r).abs().max() < 1e-5 * want_r.abs().max()
    assert (x.double().cpu() - want).abs().max() < (1e-5 if target[1] == torch.float32 else 0.02) * want.abs().max()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name,layer", [("mixed", 0), ("mixed", 1), ("odd", 0), ("wide", 1)])
def test_clamped_units(name, layer, target):
    cfg = CONFIGS[name]
    W, mlp, p = make_weights(cfg, seed=7), cfg["layers"][layer]["mlp"], f"l{layer}.mlp."
    block = make_model(cfg, W, target).layers[layer].mlp
    x = bf16_values((40, cfg["width"]), torch.Generator().manual_seed(8))
    with torch.no_grad():
        got = block(dev(x, target)).double().cpu()
    assert_close(got, plain.feed_forward(W, p, x, mlp), target[1], "feed-forward")


# ----------------------------------------------------------------------------- engine
def greedy(W, cfg, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(plain.forward(W, cfg, t)[0][-1].argmax()))
    return t[len(prompt):]


@pytest.mark.parametrize("target", TARGETS)
def test_greedy_generation_through_the_engine(target):
    """More requests than slots, prompts absorbed in portions of at most 24 tokens beside decoding ones."""
    cfg = config((att(), dense()), (par(), None), (par(heads=2, kv=1, dim=16, width=24), dense()), vocab=40)
    W = make_weights(cfg, seed=2)
    W["head"] *= 4                                     # clear winners: rounding does not flip a choice
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (1, 30, 5, 61, 18)]
    eng = make_engine(cfg, W, target, pages=40, page_size=16, slots=2, loop=True, max_prefill_tokens=24)
    res = generate(eng, prompts, 12)
    for p, r in zip(prompts, res):
        full = p + r.output_tokens
        lp = torch.log_softmax(plain.forward(W, cfg, full[:-1])[0][len(p) - 1:], -1)
        best = lp.max(-1).values
        mine = lp.gather(1, torch.tensor(r.output_tokens)[:, None])[:, 0]
        assert (best - mine).max() < (1e-3 if target[1] == torch.float32 else 0.5)
        assert (mine - torch.tensor(r.output_logprobs, dtype=torch.float64)).abs().max() < (1e-3 if target[1] == torch.float32 else 0.5)
        if target[1] == torch.float32:
            assert r.output_tokens == greedy(W, cfg, p, 12)
    assert eng.stats["prefill_tokens"] > 0 and len(eng.cache.free) == eng.cache.num_pages and len(eng.cache.free_slots) == 2
    eng.destroy()


def test_generation_survives_a_short_pool():
    cfg = config((att(), None), (par(), None), vocab=40)
    W = make_weights(cfg, seed=3)
    prompts = [tokens(20, cfg["vocab"], 40 + i) for i in range(3)]
    alone = [greedy(W, cfg, p, 30) for p in prompts]
    eng = make_engine(cfg, W, ("cpu", torch.float32), pages=6, page_size=16, slots=4, loop=True)
    res = generate(eng, prompts, 30)                   # three sequences of 50 tokens need 12 pages: someone is pre-empted
    assert [r.output_tokens for r in res] == alone and eng.stats["preempted"] > 0
    eng.destroy()


# ----------------------------------------------------------------------------- configuration, checkpoints, trace runner
def test_config_round_trip_and_errors(tmp_path):
    for name in ("tiny-goganex", "goganex-8b-layers"):
        mc = preset(name)
        mc.save_pretrained(str(tmp_path))
        back = ModelConfig.from_pretrained(str(tmp_path))
        assert back == mc and back.is_mixer_stack and back.num_params() > 0
    d = preset("tiny-goganex").to_hf_dict()
    a, p = d["layers"][0], d["layers"][1]
    left, right = p["mixer"]["left"], p["mixer"]["right"]
    bad_layer = (dict(a, type="rglru"), dict(a, mlp=dict(a["mlp"], kind="moe")), dict(a, mixer=dict(a["mixer"], kv_heads=3)),
                 dict(a, mixer=dict(a["mixer"], rot=dict(a["mixer"]["rot"], dims=64))), dict(a, mixer=dict(a["mixer"], rot=dict(a["mixer"]["rot"], dims=7))),
                 dict(p, mixer=dict(left=dict(left, vdim=left["dim"] + 8), right=right)), dict(p, mixer=dict(left=dict(left, kv_heads=4), right=right)),
                 dict(p, mixer=dict(left=left, right=dict(width=0))))
    loops = [dict(start=2, stop=2, times=2), dict(start=0, stop=5, times=2), dict(start=0, stop=1, times=0)]
    for bad in [dict(d, architecture="goganex"), *(dict(d, layers=[b], loop=None) for b in bad_layer), *(dict(d, loop=x) for x in loops)]:
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(bad)
    # a loop may be missing; what one design builds is not another's
    assert ModelConfig.from_hf_dict({k: v for k, v in d.items() if k != "loop"}).layer_loop is None
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(dict(d, architecture="Bumotar"))


def test_checkpoint_round_trip(tmp_path):
    mc = preset("tiny-goganex")
    a, b = (build_model(mc, dtype=torch.float32, seed=s) for s in (1, 2))
    hf_io.save_model_hf(a, str(tmp_path))
    hf_io.load_model_hf(b, str(tmp_path))
    for (n, p), (_, q) in zip(a.named_parameters(), b.named_parameters()):
        assert torch.equal(p, q), n


def test_checkpoint_names_and_shapes_are_the_design_s():
    for cfg in CONFIGS.values():
        W = make_weights(cfg)
        mc = ModelConfig.from_hf_dict(cfg)
        model = build_model(mc, dtype=torch.float32)
        back = dict(hf_io.native_to_hf_tensors(mc, ((n, p.detach()) for n, p in model.named_parameters())))
        assert {n: tuple(t.shape) for n, t in back.items()} == {n: tuple(t.shape) for n, t in W.items()}


def test_every_pass_has_pages_states_and_a_row_of_its_own():
    mc = preset("tiny-goganex")                        # four layers, the middle two twice
    model = build_model(mc, dtype=torch.bfloat16, seed=1)
    assert model.layer_runs == [0, 1, 2, 1, 2, 3] and not hasattr(model, "loop_in")
    cache = StateCache(model.cache_mixers(), 4, 16, 2, "cpu", torch.bfloat16)
    assert len(cache.layers) == 6 and len({lc.k.data_ptr() for lc in cache.layers}) == 6 and len({lc.shift.data_ptr() for lc in cache.layers}) == 6
    parallel = [False, True, True, True, True, False]
    assert [lc.state is not None for lc in cache.layers] == parallel
    # keys that are values are held once, with a number per key
    assert [lc.v is None for lc in cache.layers] == parallel and [lc.key_factor is not None for lc in cache.layers] == parallel
    assert cache.span == 0 and cache.windows == set() and cache.first_visible(1000) == 0
    assert StateCache.bytes_per_slot(model.cache_mixers()) == (6 * 128 + 4 * 96) * 4
    assert StateCache.bytes_per_page(model.cache_mixers(), 16, 2) == 16 * (2 * 2 * (32 + 48) * 2 + 4 * (2 * 40 * 2 + 2 * 4))
    held = [t for lc in cache.layers for t in (lc.k, lc.v, lc.key_factor) if t is not None]
    assert sum(t.numel() * t.element_size() for t in held) == 4 * StateCache.bytes_per_page(model.cache_mixers(), 16, 2)


@pytest.mark.parametrize("target", TARGETS)
def test_trace_runner_replays_steps(tmp_path, target):
    import numpy as np
    from safetensors.torch import save_file

    from areal_b200.tools.trace_run import make_engine as trace_engine
    from areal_b200.tools.trace_run import replay

    name = "mixed"
    cfg = CONFIGS[name]
    model, out = tmp_path / "model", tmp_path / "out"
    model.mkdir(), out.mkdir()
    (model / "config.json").write_text(json.dumps(cfg))
    save_file({n: t.bfloat16().contiguous() for n, t in make_weights(cfg).items()}, str(model / "model.safetensors"))
    eng = trace_engine(str(model), "float32" if target[1] == torch.float32 else "bfloat16", 256, target[0])
    assert eng.cache.num_pages == 4 and eng.cache.num_slots == 4
    ta, wa, _ = oracle(name, 97, 12)
    tb, wb, _ = oracle(name, 7, 11)
    steps = [dict(step=0, entries=[dict(id="a", tokens=ta[:90], want=[3, 89])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=ta[90:92], want=[]), dict(id="b", tokens=tb[:1], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=ta[92:], want=[4, 0]), dict(id="b", tokens=tb[1:2], want=[0])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=tb[2:], want=[4])], end=["b"])]
    said = []
    replay(eng, [json.dumps(s) for s in steps], str(out), said.append)
    assert said == [f"done {i}" for i in range(4)]
    got = {i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"]).double() for i in (0, 2, 3)}
    assert not (out / "1.f32").exists()
    assert_close(got[0], wa[[3, 89]], target[1])
    assert_close(got[2], torch.stack([wa[96], wa[92], wb[1]]), target[1])
    assert_close(got[3], wb[[6]], target[1])
    assert len(eng.cache.free) == 4 and len(eng.cache.free_slots) == 4
