"""Bumotar against the plain statement in ``plain_bumotar.py``: every mechanism alone, whole prompts, portions, single
tokens, mixed batches on reused pages and slots, and greedy generation through the rollout engine.

Every case runs on the CPU ops, and on a GPU in 32-bit and bf16 (weights and inputs are bf16 values, so the oracle sees
the same numbers)."""
import json
import math
import random

import pytest
import torch

from areal_b200.engine.ragged_step import Entry
from areal_b200.models import hf_io, mixers
from areal_b200.models.config import ModelConfig, preset
from areal_b200.models.decoder import build_model
from areal_b200.ops import functional as OF
from areal_b200.ops import mixer_ops as M

from . import plain_bumotar as plain
from .test_mixer_stack import (TARGETS, Driver, _one_thread, assert_close, bf16_values, dev, f32, generate, make_engine,  # noqa: F401
                               make_model, ragged, tokens)


def rot(dims, base=300.0, **scaling):
    return dict(base=base, dims=dims, scaling=scaling) if scaling else dict(base=base, dims=dims)


def yarn(dims, base=100.0, factor=6.0, original=60, fast=4.0, slow=0.5):
    return rot(dims, base, factor=factor, original=original, fast=fast, slow=slow)


def window(heads=4, kv=2, dim=32, vdim=32, size=40, softcap=5.0, turn=None, peak=1.7):
    """``peak``: standard deviation of the scores under random weights; wide scores make every visible key count."""
    return dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=peak * dim ** -0.5, softcap=softcap, mask=dict(size=size) if size else None,
                rot=turn or rot(dim // 2, factor=2.5))


def ret(heads=3, dim=32, vdim=32, turn=None, decay=(0.8, 0.97, 0.995, 0.9)):
    return dict(heads=heads, dim=dim, vdim=vdim, rot=turn or rot(dim), decay=[decay[i % len(decay)] for i in range(heads)])


def par(left=None, right=None, scales=(0.7, 0.45)):
    return "parallel", dict(left=left or window(), left_scale=scales[0], right=right or ret(), right_scale=scales[1])


def lat(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=48, peak=1.7, turn=None):
    return "latent_attention", dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=peak * (dim + rot_dim) ** -0.5,
                                    rot=turn or yarn(rot_dim))


def moe(experts=6, top=2, ff=48, shared=40):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top), **(dict(shared=dict(ff=shared)) if shared else {}))


def config(*layers, vocab=104, width=64, loop=(0, 2, 2), eps=1e-5, logit_scale=0.5):
    return dict(architecture="Bumotar", vocab=vocab, width=width, norm=dict(eps=eps), logit_scale=logit_scale,
                loop=dict(start=loop[0], stop=loop[1], times=loop[2]) if loop else None,
                layers=[dict(type=t, mixer=m, mlp=f) for (t, m), f in layers])


CONFIGS = {
    "mixed": config((par(), moe()), (lat(), moe(experts=3, top=3, shared=0)), (par(window(size=24, vdim=48), ret(heads=4, vdim=48)), None)),
    # sizes that no vector width divides; what runs before, in and after the loop; three passes
    "odd": config((lat(heads=3, dim=20, rot_dim=6, vdim=12, kv_rank=30), moe(experts=5, top=3, ff=20, shared=27)),
                  (par(window(heads=6, kv=2, dim=22, vdim=10, size=33, turn=rot(10)), ret(heads=5, dim=14, vdim=18, turn=rot(6))), None),
                  (lat(heads=1, dim=7, rot_dim=2, vdim=9, kv_rank=21, turn=rot(2)), None), vocab=101, width=60, loop=(1, 2, 3), eps=1e-2),
    # more than one tile of heads, windows longer than a query tile, 64 rotated numbers, every expert chosen, a loop of one pass
    "wide": config((lat(heads=20, dim=64, rot_dim=64, vdim=96, kv_rank=136, peak=1.4), moe(experts=3, top=3)),
                   (par(window(heads=17, kv=1, dim=64, vdim=96, size=320), ret(heads=2, dim=96, vdim=72, turn=rot(64))), None),
                   width=128, vocab=96, loop=(1, 2, 1), logit_scale=1.0),
    "rank512": config((lat(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=512, peak=1.0), moe(experts=9, top=1)),
                      (par(window(heads=2, kv=2, dim=128, vdim=128, size=200, turn=rot(128)), ret(heads=2, dim=128, vdim=128)), None), loop=(0, 1, 2)),
    # a token that sees itself only, a window of a page, no window, no cap, no loop; states that forget at once or never
    "edges": config((par(window(size=1, softcap=None), ret(decay=(0.0, 1.0, 0.5))), None), (par(window(size=64, turn=rot(32)), ret(heads=1, vdim=8)), moe()),
                    (par(window(size=0), ret(heads=2, dim=16, vdim=80)), None), loop=None, logit_scale=2.0),
}


def make_weights(cfg, seed=0):
    """Random weights under the checkpoint's names (float64 holding bf16 values)."""
    g = torch.Generator().manual_seed(seed)
    H, V = cfg["width"], cfg["vocab"]
    W = {"embed": bf16_values((V, H), g), "head": bf16_values((V, H), g, 2 * H ** -0.5 / cfg["logit_scale"]), "final.norm": bf16_values((H,), g, 0.2, 1.0)}
    if cfg["loop"]:
        W["loop.in"] = bf16_values((H, 2 * H), g, (2 * H) ** -0.5)
        W["loop.step"] = bf16_values((cfg["loop"]["times"], H), g, 0.5)

    def mat(name, *shape, std=1.0):
        W[name] = bf16_values(shape, g, std * shape[-1] ** -0.5)

    def vec(name, n, std=0.2, mean=1.0):
        W[name] = bf16_values((n,), g, std, mean)

    def experts(p, I):
        mat(p + "gate", I, H, std=1.5), mat(p + "up", I, H), mat(p + "down", H, I)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        if layer["type"] == "parallel":
            for n, k in (("left", m["left"].get("kv_heads")), ("right", m["right"]["heads"])):
                b, pb = m[n], f"{p}{n}."
                mat(pb + "q", b["heads"] * b["dim"], H), mat(pb + "k", k * b["dim"], H), mat(pb + "v", k * b["vdim"], H)
                mat(pb + "g", b["heads"] * b["vdim"], H), mat(pb + "o", H, b["heads"] * b["vdim"])
            vec(p + "left.q.norm", m["left"]["dim"]), vec(p + "left.k.norm", m["left"]["dim"])
        else:
            n = m["heads"]
            mat(p + "q", n * (m["dim"] + m["rot_dim"]), H), mat(p + "dkv", m["kv_rank"] + m["rot_dim"], H), vec(p + "dkv.norm", m["kv_rank"])
            mat(p + "uk", n * m["dim"], m["kv_rank"]), mat(p + "uv", n * m["vdim"], m["kv_rank"]), mat(p + "o", H, n * m["vdim"])
            mat(p + "g", n, H), vec(p + "sink", n, 1.0, 2.0)
        for n in ("norm1", "norm2") if layer["mlp"] else ("norm1",):
            vec(f"l{i}.{n}", H)
        f, p = layer["mlp"], f"l{i}.mlp."
        if f:
            mat(p + "router", f["router"]["experts"], H, std=2.0)
            for e in range(f["router"]["experts"]):
                experts(f"{p}e{e}.", f["expert"]["ff"])
            if f.get("shared"):
                experts(p + "shared.", f["shared"]["ff"])
                mat(p + "shared.sg", 1, H)
    return W


CLEAR = 0.15             # router logits by which the last chosen expert is ahead of the first one left out
STEADY = 0.02            # size of a head's retention output beside its terms
_ORACLE: dict = {}


def oracle(name, n, seed):
    """Tokens, logits and residual streams of a prompt under a named configuration (cached: shared by the targets and the
    schedules). Tokens whose choice of experts is close, or whose retention terms cancel, are drawn again until there are none:
    bf16 rounding may turn a close choice, or the sign of an output, which is another result for this token and for those that
    look back at it."""
    if (name, n, seed) not in _ORACLE:
        cfg, rnd = CONFIGS[name], random.Random(seed)
        W, t = make_weights(cfg), tokens(n, cfg["vocab"], seed)
        for _ in range(60):
            margins, steady = [torch.full((n,), CLEAR)], [torch.full((n,), STEADY)]
            logits, states = plain.forward(W, cfg, t, margins, steady)
            low = lambda x: torch.stack([m.double() for m in x]).amin(0)             # noqa: E731
            close = torch.where((low(margins) < CLEAR - 1e-6) | (low(steady) < STEADY - 1e-6))[0].tolist()
            if not close:
                break
            for i in close:
                t[i] = rnd.randrange(cfg["vocab"])
        else:
            raise AssertionError(f"{name}: no prompt of {n} tokens with clear choices")
        _ORACLE[name, n, seed] = (t, logits, states)
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
    name, n = "wide", 480
    cfg = CONFIGS[name]
    t, want, _ = oracle(name, n, 2)
    eng = make_engine(cfg, make_weights(cfg), target)
    d = Driver(eng)
    d.step([("a", t)], end=["a"])
    assert_close(d.logits("a"), want, target[1], "whole")
    d = Driver(eng)
    d.step([("a", t[:270])])
    for i in range(270, 400):                      # the window's far end walks over the page border at 64
        d.step([("a", t[i:i + 1])])
    d.step([("a", t[400:477])])
    for i in range(477, n):
        d.step([("a", t[i:i + 1])], end=["a"] if i == n - 1 else [])
    assert_close(d.logits("a"), want, target[1], "decoded")


@pytest.mark.parametrize("target", TARGETS)
def test_windows_alone_give_their_pages_back(target):
    cfg = config((par(window(size=30), ret()), None), (par(window(size=50)), None), loop=(0, 1, 2))
    W = make_weights(cfg, 5)
    t = tokens(210, cfg["vocab"], 5)
    want = plain.forward(W, cfg, t)[0]
    eng = make_engine(cfg, W, target, pages=8, page_size=16, slots=1)
    d, at = Driver(eng), 0
    for s in [20, 40] + [1] * 70 + [33, 17] + [1] * 30:         # 14 pages of tokens through a pool of 8
        d.step([("a", t[at:at + s])])
        at += s
    assert at == 210 and d.live["a"].first_page == (210 - 49) // 16
    assert_close(d.logits("a"), want, target[1])


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


# what each mechanism would be if it were read wrongly; the logits under the tests' weights must tell
FAULTS = {
    "window one longer": ("first_visible", lambda i, w: max(0, i - w) if w else 0),
    "window one shorter": ("first_visible", lambda i, w: max(0, i - w + 2) if w else 0),
    "nothing added to the denominator": ("ONE_SINK", None),
    "no sinks at all": ("weights", lambda s, sink: torch.softmax(s, -1)),
    "no cap": ("cap", lambda s, c: s),
    "neighbours turned instead of halves": ("halves", lambda d: plain.neighbours(d)),
    "halves turned instead of neighbours": ("neighbours", lambda d: [(i, i + d // 2) for i in range(d // 2)]),
    "positions not stretched": ("linear_frequencies", lambda r: plain.base_frequencies(r)),
    "no YaRN": ("yarn_frequencies", lambda r: (plain.base_frequencies(r), 1.0)),
    "YaRN without its factor": ("yarn_frequencies", lambda r, f=plain.yarn_frequencies: (f(r)[0], 1.0)),
    "latents not normed": ("latents", lambda W, p, h, m, eps: (lambda z: (z[:, :m["kv_rank"]], z[:, m["kv_rank"]:]))(h @ W[p + "dkv"].T)),
    "state without decay": ("retain", lambda q, k, v, a, f=plain.retain: f(q, k, v, [1.0] * len(a))),
    "state read before the token": ("retain", lambda q, k, v, a, f=plain.retain: f(q, k, v, a) - (q * k).sum(-1, keepdim=True) * v),
    "weights not renormalised": ("route", lambda h, r, top: (lambda s: (s.topk(top).indices, s.topk(top).values))(torch.softmax(h @ r.T, -1))),
    "shared expert without its gate": ("shared_expert", lambda W, p, h: plain.expert(W, p, h)),
    "embedding not mixed in": ("enter_pass", lambda W, x, x0, t: x @ W["loop.in"][:, :x.shape[1]].T + W["loop.step"][t]),
    "no vector of the pass": ("enter_pass", lambda W, x, x0, t: torch.cat([x, x0], -1) @ W["loop.in"].T),
    "stream and embedding swapped": ("enter_pass", lambda W, x, x0, t: torch.cat([x0, x], -1) @ W["loop.in"].T + W["loop.step"][t]),
    "one pass too few": ("runs", lambda c, f=plain.runs: f(dict(c, loop=dict(c["loop"], times=1)))),
}


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
    assert err.median() > 0.008 and err.max() > 0.1, (float(err.median()), float(err.max()))


# ----------------------------------------------------------------------------- rotation
@pytest.mark.parametrize("r", [yarn(16), yarn(64, 10000.0, 4.0, 4096, 32.0, 1.0), yarn(8, 50.0, 2.0, 20, 1e-3, 1e-4), yarn(32, 1e6, 8.0, 1 << 20, 1e5, 1e4), rot(12)])
def test_yarn_frequencies(r):
    """With ramps inside the pairs, before the first, behind the last, and without scaling."""
    got, want = mixers.yarn_frequencies(r), plain.yarn_frequencies(r)
    assert torch.allclose(torch.tensor(got[0]).double(), torch.tensor(want[0]).double(), rtol=1e-12) and abs(got[1] - want[1]) < 1e-12


def make_table(freqs, mult, pos, device):
    """[R, P, 2] with foreign columns in front, as in a model with several rotations."""
    f = torch.tensor([0.123] * 3 + [x / (2 * math.pi) for x in freqs], dtype=torch.float64, device=device)
    m = torch.tensor([9.0] * 3 + [mult] * len(freqs), dtype=torch.float32, device=device)
    return M.rotary_table(pos, f, m)[:, 3:]


@pytest.mark.parametrize("target", TARGETS[:2])
def test_angles_far_out_are_exact(target):
    freqs = [1.0, 0.37, 1e-3, 1e-7]
    pos = torch.tensor([0, 1, 999, 100_000, 16_000_001], dtype=torch.int32, device=target[0])
    got = make_table(freqs, 1.25, pos, target[0]).double().cpu()
    ang = pos.double().cpu()[:, None] * torch.tensor(freqs, dtype=torch.float64)
    assert (got - 1.25 * torch.stack([torch.cos(ang), torch.sin(ang)], -1)).abs().max() < 2e-6


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("Hq,Hkv,D,Dv,dims,norm", [(4, 2, 32, 48, 16, True), (3, 1, 22, 10, 6, True), (9, 9, 128, 64, 128, True), (2, 1, 40, 24, 40, False), (5, 5, 7, 3, 0, True)])
def test_heads_are_normed_turned_and_cached(Hq, Hkv, D, Dv, dims, norm, interleaved, target):
    g = torch.Generator().manual_seed(D)
    b, _, rows = ragged([1, 20], [133, 7], target[0])
    n = Hq * D + Hkv * (D + Dv)
    z, wq, wk = bf16_values((21, n + 8), g, 2.0), bf16_values((D,), g, 0.5, 1.0), bf16_values((D,), g, 0.5, 1.0)
    kc, vc = (torch.full((rows, Hkv, d), 9.0, dtype=target[1], device=target[0]) for d in (D, Dv))
    freqs = plain.base_frequencies(rot(dims)) if dims else []
    pos = b.pos.cpu().tolist()
    b.slots[3] = -1                                    # a padding row leaves the cache alone
    q = M.qk_head_norm_append(dev(z, target), f32(wq, target) if norm else None, f32(wk, target) if norm else None, 1e-3, make_table(freqs, 1.0, b.pos, target[0]),
                              interleaved, b, kc, vc, Hq).double().cpu()
    pairs = (plain.neighbours if interleaved else plain.halves)(dims)

    def want(x, w):
        return plain.rotate(plain.norm(x, w, 1e-3) if norm else x, pos, freqs, pairs)
    tol = 2e-5 if target[1] == torch.float32 else 0.02
    wq_, wk_ = want(z[:, :Hq * D].view(21, Hq, D), wq), want(z[:, Hq * D:(Hq + Hkv) * D].view(21, Hkv, D), wk)
    assert (q - wq_).abs().max() < tol * wq_.abs().max()
    at, keep = b.slots.long().cpu(), [i for i in range(21) if i != 3]
    assert (kc.double().cpu()[at[keep]] - wk_[keep]).abs().max() < tol * wk_.abs().max()
    assert torch.equal(vc.double().cpu()[at[keep]], z[keep, (Hq + Hkv) * D:n].view(-1, Hkv, Dv))
    assert (vc == 9.0).flatten(1).all(-1).sum() == rows - 20


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,D,r,C", [(4, 32, 16, 48), (3, 20, 6, 30), (1, 7, 2, 21), (32, 128, 64, 512)])
def test_latents_and_shared_keys_are_cached(H, D, r, C, target):
    g = torch.Generator().manual_seed(D)
    b, _, rows = ragged([1, 20], [133, 7], target[0])
    nq = H * (D + r)
    z, wc = bf16_values((21, nq + C + r + H), g, 2.0), bf16_values((C,), g, 0.5, 1.0)
    cache = torch.full((rows, 1, C + r), 9.0, dtype=target[1], device=target[0])
    freqs, mult = plain.yarn_frequencies(yarn(r))
    pos = b.pos.cpu().tolist()
    b.slots[3] = -1
    zt = dev(z, target).clone()
    M.latent_rope_append(zt, f32(wc, target), 1e-3, make_table(freqs, mult, b.pos, target[0]), True, b, cache, H, D)
    got, tol = zt.double().cpu(), 2e-5 if target[1] == torch.float32 else 0.02
    q = z[:, :nq].view(21, H, D + r)
    want_q = torch.cat([q[..., :D], plain.rotate(q[..., D:], pos, freqs, plain.neighbours(r), mult)], -1)
    assert (got[:, :nq].view(21, H, D + r) - want_q).abs().max() < tol * want_q.abs().max()
    assert torch.equal(got[:, :nq].view(21, H, D + r)[..., :D], q[..., :D]) and torch.equal(got[:, nq + C + r:], z[:, nq + C + r:])
    want = torch.cat([plain.norm(z[:, nq:nq + C], wc, 1e-3), plain.rotate(z[:, nq + C:nq + C + r], pos, freqs, plain.neighbours(r), mult)], -1)
    at, keep = b.slots.long().cpu(), [i for i in range(21) if i != 3]
    assert (cache.double().cpu()[at[keep], 0] - want[keep]).abs().max() < tol * want.abs().max()
    assert (cache == 9.0).flatten(1).all(-1).sum() == rows - 20


# ----------------------------------------------------------------------------- attention
def stand_out(q, keys, L, n, s, size, gain):
    """For some queries one key stands out: just inside or just outside the window, at a page border, far away, the first ones."""
    for i in {L - 1, L - 2, s, s + n // 2, min(L - 1, size), min(L - 1, 127), min(L - 1, 128)}:
        for back in (size, size - 1, 16, i, i % 16):
            if i >= 0 and 0 <= back <= i and (i * 7 + back * 3) % 3 == 0:
                k = keys(i - back)
                q[i] = (k / k.norm(dim=-1, keepdim=True) * gain).bfloat16().double()


SCHEDULES = (([1, 1, 1, 1, 130, 300, 2], [0, 47, 333, 90, 0, 70, 118]), ([1, 2, 9, 16], [80, 62, 300, 0]))


def page_rows(entry, L, device):
    j = torch.arange(L)
    return (torch.tensor(entry.carry.pages)[j // 16] * 16 + j % 16).to(device)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("Hq,Hkv,D,Dv,size,cap,sink", [(4, 2, 32, 48, 40, 5.0, 0.0), (6, 2, 96, 64, 112, 9.0, "heads"), (32, 2, 64, 128, 200, 0.0, 0.0),
                                                       (3, 1, 20, 12, 33, 6.0, "heads"), (2, 2, 8, 40, 1, 3.0, 0.0), (17, 1, 128, 72, 0, 12.0, 1.5),
                                                       (40, 20, 128, 128, 257, 4.0, None), (2, 1, 136, 24, 64, 0.0, "heads")])
def test_window_attention_with_sinks_and_gates(Hq, Hkv, D, Dv, size, cap, sink, target):
    g = torch.Generator().manual_seed(D + Dv)
    sinks = bf16_values((Hq,), g, 1.0, 2.0) if sink == "heads" else sink
    tol, scale = 1e-4 if target[1] == torch.float32 else 0.04, D ** -0.5
    for lens, starts in SCHEDULES:
        b, entries, rows = ragged(lens, starts, target[0])
        kc, vc = (torch.zeros(rows, Hkv, d, dtype=target[1], device=target[0]) for d in (D, Dv))
        qs, kvs = [], []
        for e, (n, s) in enumerate(zip(lens, starts)):
            L = n + s
            q, k, v = bf16_values((L, Hq, D), g), bf16_values((L, Hkv, D), g), bf16_values((L, Hkv, Dv), g)
            stand_out(q, lambda j: k[j].repeat_interleave(Hq // Hkv, 0), L, n, s, size, 2.5 * D ** 0.5)
            at = page_rows(entries[e], L, target[0])
            kc[at], vc[at] = dev(k, target), dev(v, target)
            qs.append(q), kvs.append((k, v))
        R = sum(lens)
        wide = bf16_values((R, Hq * Dv + 24), g)                   # the gate is a stretch of a wider product, the output of a wider row
        gate = wide[:, 16:16 + Hq * Dv]
        out = torch.zeros(R, Hq * Dv + 16, dtype=target[1], device=target[0])
        q_rows = dev(torch.cat([q[s:] for q, s in zip(qs, starts)]), target).contiguous()
        M.chunk_attention(q_rows, kc, vc, b, scale, cap, window=size, sink=f32(sinks, target) if sink == "heads" else sink,
                          gate=dev(wide, target)[:, 16:16 + Hq * Dv], out_scale=0.625, out=out[:, 8:8 + Hq * Dv])
        assert (out[:, :8] == 0).all() and (out[:, 8 + Hq * Dv:] == 0).all()
        got, at = out[:, 8:8 + Hq * Dv].double().cpu(), 0
        for e, (n, s) in enumerate(zip(lens, starts)):
            o = plain.attend(qs[e], *kvs[e], scale, cap, size, torch.full((Hq,), sinks) if isinstance(sinks, float) else sinks)[s:]
            want = o.reshape(n, -1) * plain.sigmoid(gate[at:at + n]) * 0.625
            assert (got[at:at + n] - want).abs().amax() < tol * want.abs().amax(), e
            at += n


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,D,r,Dv,C,size", [(4, 32, 16, 32, 48, 0), (6, 64, 8, 48, 128, 112), (20, 128, 64, 128, 512, 0), (3, 20, 6, 12, 30, 0), (2, 8, 64, 40, 520, 90),
                                             (17, 16, 24, 96, 256, 0), (1, 72, 48, 8, 8, 257), (40, 24, 40, 16, 136, 64), (5, 128, 72, 64, 96, 0)])
def test_latent_attention_with_positions_sinks_and_gates(H, D, r, Dv, C, size, target):
    """Portions (long ones, and ones short enough to read the latents as single tokens do) and single tokens."""
    g = torch.Generator().manual_seed(D + Dv + C)
    w_k, w_v = (bf16_values((H, n, C), g, C ** -0.5) for n in (D, Dv))
    w_kv = dev(torch.cat([w_k.reshape(-1, C), w_v.reshape(-1, C)]), target)
    sink, tol, scale = bf16_values((H,), g, 1.0, 2.0), 1e-4 if target[1] == torch.float32 else 0.04, (D + r) ** -0.5
    for lens, starts in SCHEDULES:
        b, entries, rows = ragged(lens, starts, target[0], windows=[size])
        cache = torch.zeros(rows, 1, C + r, dtype=target[1], device=target[0])
        qs, kvs = [], []
        for e, (n, s) in enumerate(zip(lens, starts)):
            L = n + s
            q, c = bf16_values((L, H, D + r), g), bf16_values((L, C + r), g)
            k = torch.cat([torch.einsum("hdc,lc->lhd", w_k, c[:, :C]), c[:, None, C:].expand(L, H, r)], -1)
            stand_out(q, lambda j: k[j], L, n, s, size, 2.5 * (D + r) ** 0.5)
            cache[page_rows(entries[e], L, target[0]), 0] = dev(c, target)
            qs.append(q), kvs.append((k, torch.einsum("hdc,lc->lhd", w_v, c[:, :C])))
        R, nq = sum(lens), H * (D + r)
        z = torch.cat([torch.cat([q[s:] for q, s in zip(qs, starts)]).reshape(R, nq), bf16_values((R, H + 5), g)], 1)
        zt = torch.zeros(R, -(-z.shape[1] // 8) * 8, dtype=target[1], device=target[0])
        zt[:, :z.shape[1]] = dev(z, target)
        got = M.latent_attention(zt[:, :nq].unflatten(1, (H, D + r)), cache, w_kv, Dv, b, scale, size, r, f32(sink, target), zt[:, nq:nq + H]).double().cpu()
        at = 0
        for e, (n, s) in enumerate(zip(lens, starts)):
            want = plain.attend(qs[e], *kvs[e], scale, None, size, sink)[s:] * plain.sigmoid(z[at:at + n, nq:nq + H])[..., None]
            err = (got[at:at + n] - want).abs().amax() / want.abs().amax()
            assert err < tol, (e, float(err))
            at += n


@pytest.mark.parametrize("target", TARGETS)
def test_portions_and_single_tokens_read_the_same_latents(target, monkeypatch):
    """One long portion through worked-out keys and values, and the same rows through the latents."""
    g = torch.Generator().manual_seed(1)
    H, D, r, Dv, C = 5, 32, 16, 24, 64
    w = dev(bf16_values((H * (D + Dv), C), g, C ** -0.5), target)
    b, _, rows = ragged([100, 130], [30, 0], target[0], windows=[0])
    q, cache, gate = dev(bf16_values((230, H, D + r), g), target), dev(bf16_values((rows, 1, C + r), g), target), dev(bf16_values((230, H), g), target)
    sink = f32(bf16_values((H,), g), target)
    a = M.latent_attention(q, cache, w, Dv, b, 0.2, 0, r, sink, gate)
    monkeypatch.setattr(M, "SHORT_PORTION", 1000)
    z = M.latent_attention(q, cache, w, Dv, b, 0.2, 0, r, sink, gate)
    assert (a - z).abs().max() < (1e-5 if target[1] == torch.float32 else 0.05)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("R,H,N,K,extra", [(3, 5, 16, 24, 8), (130, 3, 512, 72, 64), (64, 33, 40, 136, 16), (4, 3, 7, 9, 2), (70, 1, 128, 64, 24)])
def test_heads_of_a_wider_row_have_their_own_products(R, H, N, K, extra, target):
    g = torch.Generator().manual_seed(R + N)
    z, w = bf16_values((R, H * (K + extra) + 8), g), bf16_values((H, N, K), g, K ** -0.5)
    x = z[:, :H * (K + extra)].view(R, H, K + extra)[..., :K]
    want = torch.einsum("rhk,hnk->rhn", x, w)
    xt = dev(z, target)[:, :H * (K + extra)].unflatten(1, (H, K + extra))[..., :K]
    tol = 1e-5 if target[1] == torch.float32 else 0.02
    assert (M.head_linear(xt, dev(w, target)).double().cpu() - want).abs().max() < tol * want.abs().max()
    got = M.head_linear(xt, dev(w.transpose(1, 2).contiguous(), target), w_kn=True)
    assert (got.double().cpu() - want).abs().max() < tol * want.abs().max()


# ----------------------------------------------------------------------------- retention
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,N,P,dims", [(3, 32, 32, 32), (5, 14, 18, 6), (2, 128, 128, 128), (1, 96, 72, 64), (4, 64, 8, 24), (2, 40, 200, 0), (2, 256, 24, 256), (3, 30, 5, 30),
                                        (2, 8, 64, 8)])
def test_retention(H, N, P, dims, target):
    """Portions and single tokens from carried states, in slots that hold what an earlier request left; strong and weak decays."""
    g = torch.Generator().manual_seed(N + P)
    lens, starts = [1, 1, 1, 130, 64, 2, 200], [0, 47, 5, 0, 63, 118, 3]
    b, entries, _ = ragged(lens, starts, target[0])
    decay = [0.0, 1.0, 0.5, 0.999, 0.93][:H] if H > 1 else [0.97]
    freqs, R = plain.base_frequencies(rot(dims)) if dims else [], sum(lens)
    S = torch.full((len(lens), H, P, N), 3.0, dtype=torch.float32, device=target[0])        # of requests that are gone
    width = H * (2 * N + 2 * P)
    rows, wants, ends = [], [], []
    for e, (n, s) in enumerate(zip(lens, starts)):
        L = n + s
        z = bf16_values((L, width), g)
        q, k = (plain.rotate(z[:, i * H * N:(i + 1) * H * N].view(L, H, N), range(L), freqs, plain.halves(dims)) for i in (0, 1))
        k, v = k * N ** -0.5, z[:, 2 * H * N:2 * H * N + H * P].view(L, H, P)
        o = plain.retain(q, k, v, decay)

        def state(T):
            w = torch.tensor(decay, dtype=torch.float64)[None, :] ** torch.arange(T - 1, -1, -1)[:, None]
            return torch.einsum("th,thn,thp->hpn", w, k[:T], v[:T])
        if s:
            S[entries[e].carry.slot] = state(s).float().to(target[0])
        rows.append(z[s:]), ends.append(state(L))
        wants.append(((o / plain.rms(o, 1e-5)).reshape(L, -1) * plain.silu(z[:, width - H * P:]) * 0.5)[s:])
    zt = torch.zeros(R, -(-width // 8) * 8 + 8, dtype=target[1], device=target[0])
    zt[:, :width] = dev(torch.cat(rows), target)
    out = torch.zeros(R, H * P + 8, dtype=target[1], device=target[0])
    dec = torch.tensor(decay, dtype=torch.float32, device=target[0])
    log2 = torch.tensor([math.log2(a) if a else -1e4 for a in decay], dtype=torch.float32, device=target[0])
    M.retention(zt[:, :width], dec, log2, make_table(freqs, 1.0, b.pos, target[0]), 1e-5, 0.5, out[:, :H * P], H, N, P, b, S)
    assert (out[:, H * P:] == 0).all()
    got, at = out[:, :H * P].double().cpu(), 0
    for e, n in enumerate(lens):
        err = (got[at:at + n] - wants[e]).pow(2).mean(-1).sqrt() / wants[e].pow(2).mean().sqrt()
        assert err.max() < (2e-4 if target[1] == torch.float32 else 0.03), (e, float(err.max()))
        # the state is 32-bit whatever the activations are
        st = S[entries[e].carry.slot].double().cpu()
        assert (st - ends[e]).abs().max() < 2e-4 * ends[e].abs().max(), (e, float((st - ends[e]).abs().max()))
        at += n


@pytest.mark.parametrize("target", TARGETS)
def test_long_decoding_keeps_the_state(target):
    """A key that was taken in 400 tokens ago still answers a query along its direction."""
    g = torch.Generator().manual_seed(9)
    H, N, P, L = 2, 32, 16, 420
    z = bf16_values((L, H * (2 * N + 2 * P)), g, 0.3)
    z[0, H * N:2 * H * N] *= 20
    z[L - 1, :H * N] = z[0, H * N:2 * H * N]
    decay = [1.0 - 2.0 ** -10, 1.0 - 2.0 ** -12]
    q, k, v = z[:, :H * N].view(L, H, N), z[:, H * N:2 * H * N].view(L, H, N) * N ** -0.5, z[:, 2 * H * N:2 * H * N + H * P].view(L, H, P)
    o = plain.retain(q, k, v, decay)
    want = ((o / plain.rms(o, 1e-6)).reshape(L, -1) * plain.silu(z[:, -H * P:]))[-1]
    S = torch.zeros(1, H, P, N, dtype=torch.float32, device=target[0])
    dec = torch.tensor(decay, dtype=torch.float32, device=target[0])
    at, zt = 0, dev(z, target)
    for n in [2] + [1] * 417 + [1]:
        b, _, _ = ragged([n], [at], target[0])
        out = torch.zeros(n, H * P, dtype=target[1], device=target[0])
        M.retention(zt[at:at + n], dec, torch.log2(dec), make_table([], 1.0, b.pos, target[0]), 1e-6, 1.0, out, H, N, P, b, S)
        at += n
    assert at == L and (out[0].double().cpu() - want).abs().max() < (2e-4 if target[1] == torch.float32 else 0.02) * want.abs().max()


# ----------------------------------------------------------------------------- residual sum, feed-forward
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H", [64, 60, 42, 2048, 5120])
def test_residual_sum_and_norm(H, target):
    g = torch.Generator().manual_seed(H)
    R, k, E = 6, 2, 4
    h, resid, w, vec = bf16_values((R, H), g, 3.0), torch.randn(R, H, generator=g, dtype=torch.float64), bf16_values((H,), g, 0.3, 1.0), bf16_values((H,), g)
    tol = 1e-5 if target[1] == torch.float32 else 0.02

    def check(src, dense, v=None, nxt=w, mult=1.0, strided=False):
        r = f32(resid, target).contiguous()
        out = torch.zeros(R, 2 * H, dtype=target[1], device=target[0])[:, :H] if strided else None
        x = M.residual_norm(src, r, None if nxt is None else f32(nxt, target), 1e-3, target[1], None if v is None else f32(v, target), mult, out)
        want_r = resid.float().double() + dense + (0 if v is None else v)
        assert (r.double().cpu() - want_r).abs().max() < 1e-5 * want_r.abs().max()      # the residual sum is 32-bit whatever the activations are
        want = want_r if nxt is None else mult * plain.norm(want_r, nxt, 1e-3)
        assert x.dtype == target[1] and (x.double().cpu() - want).abs().max() < tol * want.abs().max()
        assert out is None or (x.data_ptr() == out.data_ptr() and x.stride(0) == 2 * H)
    check(None, 0.0)
    check(None, 0.0, vec)
    check(dev(h, target), h, mult=0.25)
    check(dev(h, target), h, nxt=None, strided=True)
    check(dev(torch.cat([h, h], 1), target)[:, :H], h, vec)                             # rows of a wider product
    rt = OF.moe_route(torch.randn(R, E, generator=g).to(target[0]), k, want_host=False)
    y, lg = bf16_values((R * k, H), g), torch.randn(R, 8, generator=g, dtype=torch.float64).float().double()
    inv, tw = rt.inv.long().cpu().view(R, k), rt.topw.double().cpu()
    summed, gated = (y[inv] * tw[..., None]).sum(1), h * plain.sigmoid(lg[:, 5:6])
    check(M.ExpertSum(dev(y, target), rt, None, rt.topw), summed)
    check(M.ExpertSum(dev(y, target), rt, dev(h, target), rt.topw), summed + h, mult=2.0)
    check(M.ExpertSum(dev(y, target), rt, dev(h, target), rt.topw, lg.float().to(target[0])[:, 5]), summed + gated, nxt=None)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name,layer", [("mixed", 0), ("mixed", 1), ("odd", 0), ("wide", 0), ("rank512", 0)])
def test_experts_beside_a_gated_shared_one(name, layer, target):
    cfg = CONFIGS[name]
    W, mlp, p = make_weights(cfg, seed=7), cfg["layers"][layer]["mlp"], f"l{layer}.mlp."
    block = make_model(cfg, W, target).layers[layer].mlp
    x = bf16_values((40, cfg["width"]), torch.Generator().manual_seed(8))
    margins = [torch.ones(40)]
    want = plain.feed_forward(W, p, x, mlp, margins)
    with torch.no_grad():
        got = block(dev(x, target)).dense().double().cpu()
    assert_close(got, want, target[1], "experts", torch.stack([m.double() for m in margins]).amin(0) > 0.02)


@pytest.mark.parametrize("target", TARGETS)
def test_router_logits_may_be_part_of_a_row(target):
    z = torch.randn(33, 16, generator=torch.Generator().manual_seed(2)).to(target[0])
    a, b = (OF.moe_route(t, 3, want_host=False) for t in (z[:, :9], z[:, :9].contiguous()))
    assert torch.equal(a.tope, b.tope) and torch.equal(a.topw, b.topw) and torch.equal(a.inv, b.inv)
    assert torch.allclose(a.topw.sum(-1), torch.ones(33, device=target[0]))


# ----------------------------------------------------------------------------- engine
def greedy(W, cfg, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(plain.forward(W, cfg, t)[0][-1].argmax()))
    return t[len(prompt):]


@pytest.mark.parametrize("target", TARGETS)
def test_greedy_generation_through_the_engine(target):
    """More requests than slots, prompts absorbed in portions of at most 24 tokens beside decoding ones."""
    cfg = config((par(window(size=20)), moe()), (lat(), None), (par(window(size=31)), None), vocab=40)
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
    cfg = config((lat(), None), (par(window(size=30)), None), vocab=40)
    W = make_weights(cfg, seed=3)
    prompts = [tokens(20, cfg["vocab"], 40 + i) for i in range(3)]
    alone = [greedy(W, cfg, p, 30) for p in prompts]
    eng = make_engine(cfg, W, ("cpu", torch.float32), pages=6, page_size=16, slots=4, loop=True)
    res = generate(eng, prompts, 30)                   # three sequences of 50 tokens need 12 pages: someone is pre-empted
    assert [r.output_tokens for r in res] == alone and eng.stats["preempted"] > 0
    eng.destroy()


# ----------------------------------------------------------------------------- configuration, checkpoints, trace runner
def test_config_round_trip_and_errors(tmp_path):
    for name in ("tiny-bumotar", "bumotar-8b-layers"):
        mc = preset(name)
        mc.save_pretrained(str(tmp_path))
        back = ModelConfig.from_pretrained(str(tmp_path))
        assert back == mc and back.is_mixer_stack and back.num_params() > 0
    d = preset("tiny-bumotar").to_hf_dict()
    p, lt = d["layers"][0], d["layers"][1]
    left, right = p["mixer"]["left"], p["mixer"]["right"]
    bad_layer = (dict(p, type="attention"), dict(p, mlp=dict(p["mlp"], kind="dense")), dict(p, mixer=dict(p["mixer"], left=dict(left, kv_heads=3))),
                 dict(p, mixer=dict(p["mixer"], right=dict(right, decay=[0.5]))), dict(p, mixer=dict(p["mixer"], left=dict(left, rot=dict(left["rot"], dims=64)))),
                 dict(lt, mixer=dict(lt["mixer"], kv_rank=0)), dict(lt, mixer=dict(lt["mixer"], rot=dict(lt["mixer"]["rot"], dims=8))),
                 dict(p, mlp=dict(p["mlp"], router=dict(experts=4, top=5))))
    loops = [dict(start=2, stop=2, times=2), dict(start=0, stop=5, times=2), dict(start=0, stop=1, times=0)]
    for bad in [dict(d, architecture="bumotar"), *(dict(d, layers=[b], loop=None) for b in bad_layer), *(dict(d, loop=x) for x in loops)]:
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(bad)
    # what one design builds is not another's
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(dict(preset("tiny-vogilix").to_hf_dict(), architecture="Kagolix"))


def test_checkpoint_round_trip(tmp_path):
    mc = preset("tiny-bumotar")
    a, b = (build_model(mc, dtype=torch.float32, seed=s) for s in (1, 2))
    hf_io.save_model_hf(a, str(tmp_path))
    hf_io.load_model_hf(b, str(tmp_path))
    used = {n: p for n, p in a.named_parameters()}
    for n, q in b.named_parameters():
        p = used[n]
        if n.endswith("router"):                       # rows behind the shared expert's gate have no use and no name
            p, q = p[:7], q[:7]
        assert torch.equal(p, q), n


def test_checkpoint_names_and_shapes_are_the_design_s():
    for cfg in CONFIGS.values():
        W = make_weights(cfg)
        mc = ModelConfig.from_hf_dict(cfg)
        model = build_model(mc, dtype=torch.float32)
        back = dict(hf_io.native_to_hf_tensors(mc, ((n, p.detach()) for n, p in model.named_parameters())))
        assert {n: tuple(t.shape) for n, t in back.items()} == {n: tuple(t.shape) for n, t in W.items()}


def test_designs_name_their_kernel_sources():
    from areal_b200.ops import build

    for d in mixers.DESIGNS.values():
        names = build.STEP_SOURCES + d.kernels
        assert len(build.sources(names)) == len(set(names)) == len(names)


def test_every_pass_has_pages_and_states_of_its_own():
    mc = preset("tiny-bumotar")                        # four layers, the middle two twice
    model = build_model(mc, dtype=torch.float32, seed=1)
    assert model.layer_runs == [0, 1, 2, 1, 2, 3]
    from areal_b200.engine.state_cache import StateCache

    cache = StateCache(model.cache_mixers(), 4, 16, 2, "cpu", torch.float32)
    assert len(cache.layers) == 6 and len({lc.k.data_ptr() for lc in cache.layers}) == 6
    assert [lc.state is not None for lc in cache.layers] == [True, False, True, False, True, False]
    assert cache.span == 0 and cache.windows == {0} and cache.first_visible(1000) == 0
    assert StateCache.bytes_per_slot(model.cache_mixers()) == 3 * 2 * 48 * 32 * 4


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
