"""Vogilix against the plain statement in ``plain_vogilix.py``: every mechanism alone, whole prompts, portions, single
tokens, mixed batches on reused pages and slots, and greedy generation through the rollout engine.

Every case runs on the CPU ops, and on a GPU in 32-bit and bf16 (weights and inputs are bf16 values, so the oracle sees
the same numbers)."""
import json
import random

import pytest
import torch

from areal_b200.engine.ragged_step import Entry
from areal_b200.models import hf_io
from areal_b200.models.config import ModelConfig, preset
from areal_b200.models.decoder import build_model
from areal_b200.ops import functional as OF
from areal_b200.ops import mixer_ops as M

from . import plain_vogilix as plain
from .test_mixer_stack import (TARGETS, Driver, _one_thread, assert_close, bf16_values, dev, f32, generate, make_engine,  # noqa: F401
                               make_model, ragged, tokens)


def mixer(heads=4, dim=32, vdim=32, q_rank=40, kv_rank=48, size=40, peak=3.0):
    """``peak``: standard deviation of the scores under random weights; wide scores make every visible key count."""
    return dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=peak * dim ** -0.5, mask=dict(size=size) if size else None)


def dense(ff=80):
    return dict(kind="dense", ff=ff)


def moe(experts=6, top=2, ff=48, limit=1.25, shared=72, shared_limit=0.75):
    m = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))
    return dict(m, shared=dict(ff=shared, limit=shared_limit)) if shared else m


def config(*layers, vocab=104, width=64, mult=0.7, side=24, positions=1024, eps=1e-5):
    return dict(architecture="Vogilix", vocab=vocab, width=width, max_positions=positions, norm=dict(eps=eps), residual_mult=mult,
                token_side=dict(dim=side) if side else None, layers=[dict(type="latent_attention", mixer=m, mlp=f) for m, f in layers])


CONFIGS = {
    "mixed": config((mixer(), dense()), (mixer(size=24, vdim=48), moe()), (mixer(heads=3, size=72, kv_rank=64), None), (mixer(size=33), moe(top=3, shared=0))),
    # sizes that no vector width divides
    "odd": config((mixer(heads=3, dim=20, vdim=12, q_rank=18, kv_rank=30, size=33, peak=1.5), moe(experts=5, top=3, ff=20, shared=27)),
                  (mixer(heads=5, dim=7, vdim=10, q_rank=9, kv_rank=21, size=17, peak=1.5), dense(33)), vocab=101, width=60, side=6, mult=0.5, eps=1e-2),
    # more than one tile of heads, windows longer than a query tile, every expert chosen
    "wide": config((mixer(heads=20, dim=64, vdim=96, q_rank=72, kv_rank=136, size=320, peak=2.0), dense(96)),
                   (mixer(heads=17, dim=16, vdim=8, q_rank=24, kv_rank=32, size=130), moe(experts=3, top=3)), width=128, vocab=96, mult=0.25),
    "rank512": config((mixer(heads=2, dim=128, vdim=128, q_rank=160, kv_rank=512, size=200, peak=1.25), moe(experts=9, top=1, limit=0.5)),
                      (mixer(heads=33, dim=8, vdim=16, q_rank=8, kv_rank=264, size=96, peak=1.25), None), mult=1.25),
    # a token that sees itself only, windows of a page, no window, no token input
    "edges": config((mixer(heads=2, size=1), dense()), (mixer(size=64), None), (mixer(heads=1, size=65, vdim=112), None), (mixer(size=0, peak=2.0), None), side=0),
}


def make_weights(cfg, seed=0):
    """Random weights under the checkpoint's names (float64 holding bf16 values)."""
    g = torch.Generator().manual_seed(seed)
    H, V = cfg["width"], cfg["vocab"]
    W = {"embed": bf16_values((V, H), g), "pos": bf16_values((cfg["max_positions"], H), g, 0.5), "head": bf16_values((V, H), g, 2 * H ** -0.5),
         "final.norm": bf16_values((H,), g, 0.2)}
    side = (cfg["token_side"] or {}).get("dim", 0)
    if side:
        W["side.embed"] = bf16_values((V, side * len(cfg["layers"])), g)

    def mat(name, *shape, std=1.0):
        W[name] = bf16_values(shape, g, std * shape[-1] ** -0.5)

    def experts(p, I, std=1.5):
        mat(p + "gate", I, H, std=std), mat(p + "up", I, H, std=std), mat(p + "down", H, I)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        mat(p + "dq", m["q_rank"], H), mat(p + "dkv", m["kv_rank"], H), mat(p + "uq", m["heads"] * m["dim"], m["q_rank"])
        mat(p + "uk", m["heads"] * m["dim"], m["kv_rank"]), mat(p + "uv", m["heads"] * m["vdim"], m["kv_rank"])
        mat(p + "o", H, m["heads"] * m["vdim"])
        W[p + "dq.norm"], W[p + "dkv.norm"] = bf16_values((m["q_rank"],), g, 0.2, 1.0), bf16_values((m["kv_rank"],), g, 0.2, 1.0)
        for n in ("norm1", "norm2") if layer["mlp"] else ("norm1",):
            W[f"l{i}.{n}"] = bf16_values((H,), g, 0.2)
        f, p = layer["mlp"], f"l{i}.mlp."
        if f and f["kind"] == "dense":
            mat(p + "up", f["ff"], H), mat(p + "down", H, f["ff"])
        elif f:
            mat(p + "router", f["router"]["experts"], H, std=2.0)
            for e in range(f["router"]["experts"]):
                experts(f"{p}e{e}.", f["expert"]["ff"])
            if f.get("shared"):
                experts(p + "shared.", f["shared"]["ff"])
        if side:
            mat(f"l{i}.side.gate", side, H), mat(f"l{i}.side.proj", H, side)
            W[f"l{i}.side.norm"] = bf16_values((H,), g, 0.2, 1.0)
    return W


CLEAR = 0.3              # router logits by which the last chosen expert is ahead of the first one left out
_ORACLE: dict = {}


def oracle(name, n, seed):
    """Tokens, logits and residual streams of a prompt under a named configuration (cached: shared by the targets and the
    schedules). Tokens whose choice of experts is close are drawn again, until none is: bf16 rounding may turn a close choice,
    which is another result for this token and for those that look back at it."""
    if (name, n, seed) not in _ORACLE:
        cfg, rnd = CONFIGS[name], random.Random(seed)
        W, t = make_weights(cfg), tokens(n, cfg["vocab"], seed)
        for _ in range(40):
            margins = [torch.full((n,), CLEAR)]
            logits, states = plain.forward(W, cfg, t, margins)
            close = torch.where(torch.stack([m.double() for m in margins]).amin(0) < CLEAR - 1e-6)[0].tolist()
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
def test_long_prompt_and_long_decoding_cross_many_windows(target):
    name, n = "wide", 700
    cfg = CONFIGS[name]
    t, want, _ = oracle(name, n, 2)
    eng = make_engine(cfg, make_weights(cfg), target)
    d = Driver(eng)
    d.step([("a", t)], end=["a"])
    assert_close(d.logits("a"), want, target[1], "whole")
    d = Driver(eng)
    d.step([("a", t[:330])])
    for i in range(330, 450):                      # the window's far end walks over the page borders at 64 and 128
        d.step([("a", t[i:i + 1])])
    assert d.live["a"].first_page == (450 - 319) // 64 and len(d.live["a"].pages) == 8 - (450 - 319) // 64
    d.step([("a", t[450:637])])
    for i in range(637, n):
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
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_layer_outputs_match(name, target):
    cfg = CONFIGS[name]
    t, _, states = oracle(name, 70, 5)
    eng = make_engine(cfg, make_weights(cfg), target)
    c, seen = eng.cache.open(), []
    eng.cache.grow(c, 70)
    eng.runner.step([Entry(c, t, [69])], on_layer=lambda i, r: seen.append(r.double().cpu().clone()))
    assert len(seen) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(seen, states)):
        assert_close(a, b, target[1], f"layer {i}")


# what each mechanism would be if it were read wrongly; the logits under the tests' weights must tell
FAULTS = {
    "window one longer": ("visible", lambda i, w: max(0, i - w) if w else 0),
    "window one shorter": ("visible", lambda i, w: max(0, i - w + 2) if w > 1 else (i if w else 0)),
    "no position vectors": ("embed", lambda W, t: W["embed"][t]),
    "positions from one": ("embed", lambda W, t: W["embed"][t] + W["pos"][1:len(t) + 1]),
    "norm weights not around zero": ("offset_norm", lambda x, w, eps: x / plain.rms(x, eps) * w),
    "latents not normed": ("latents", lambda W, pre, h, eps: (h @ W[pre + "dq"].T, h @ W[pre + "dkv"].T)),
    "router weights renormalised": ("route", lambda h, r, top, f=plain.route: (lambda c, s: (c, s / s.sum(-1, keepdim=True)))(*f(h, r, top))),
    "no limit on the units": ("expert", lambda W, p, h, lim, f=plain.expert: f(W, p, h, 1e9)),
    "the same token input in every layer": ("side_input", lambda W, i, x, t, d: (plain.gelu_tanh(x @ W[f"l{i}.side.gate"].T) * W["side.embed"][t][:, :d])
                                            @ W[f"l{i}.side.proj"].T),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_a_wrong_reading_shows_in_the_logits(fault, monkeypatch):
    """Planted in the plain statement: no mechanism is drowned by the random weights of the other tests."""
    name, fn = FAULTS[fault]
    t, want, _ = oracle("mixed", 130, 10)
    monkeypatch.setattr(plain, name, fn)
    cfg = CONFIGS["mixed"]
    got = plain.forward(make_weights(cfg), cfg, t)[0]
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    assert err.median() > 0.03 and err.max() > 0.18, (float(err.median()), float(err.max()))


# ----------------------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,D,Dv,C,window", [(4, 32, 32, 48, 40), (6, 64, 48, 128, 112), (20, 128, 128, 512, 200), (3, 20, 12, 30, 33), (2, 8, 40, 520, 1),
                                             (17, 16, 96, 256, 0), (1, 72, 8, 8, 257), (40, 24, 16, 136, 64)])
def test_latent_attention(H, D, Dv, C, window, target):
    """Portions (long ones, and ones short enough to read the latents as single tokens do) and single tokens. For some
    queries one key stands out: just inside or just outside the window, at a page border, far away, the very first ones."""
    g = torch.Generator().manual_seed(D + Dv + C)
    w_k, w_v = (bf16_values((H, n, C), g, C ** -0.5) for n in (D, Dv))
    w_kv = dev(torch.cat([w_k.reshape(-1, C), w_v.reshape(-1, C)]), target)
    tol = 1e-4 if target[1] == torch.float32 else 0.04
    for lens, starts in (([1, 1, 1, 1, 130, 300, 2], [0, 47, 333, window, 0, 70, 118]), ([1, 2, 9, 16], [80, 62, 300, 0])):
        b, entries, rows = ragged(lens, starts, target[0], windows=[window])
        cache = torch.zeros(rows, 1, C, dtype=target[1], device=target[0])
        qs, cs = [], []
        for e, (n, s) in enumerate(zip(lens, starts)):
            L = n + s
            q, c = bf16_values((L, H, D), g), bf16_values((L, C), g)
            for i in {L - 1, L - 2, s, s + n // 2, min(L - 1, window), min(L - 1, 127), min(L - 1, 128)}:
                for back in (window, window - 1, 16, i, i % 16):
                    if i >= 0 and 0 <= back <= i and (i * 7 + back * 3) % 3 == 0:
                        # a query along one key's direction: its score is far above the others'
                        k = torch.einsum("hdc,c->hd", w_k, c[i - back])
                        q[i] = (k / k.norm(dim=-1, keepdim=True) * 2.5 * D ** 0.5).bfloat16().double()
            qs.append(q), cs.append(c)
            j = torch.arange(L)
            at = (torch.tensor(entries[e].carry.pages)[j // 16] * 16 + j % 16).to(target[0])
            cache[at, 0] = dev(c, target)
        q_rows = dev(torch.cat([q[s:] for q, s in zip(qs, starts)]), target).contiguous()
        scale = D ** -0.5
        got = M.latent_attention(q_rows, cache, w_kv, Dv, b, scale, window).double().cpu()
        at = 0
        for e, (n, s) in enumerate(zip(lens, starts)):
            k, v = (torch.einsum("hdc,lc->lhd", w, cs[e]) for w in (w_k, w_v))
            want = plain.attend(qs[e], k, v, scale, window)[s:]
            err = (got[at:at + n] - want).abs().amax() / want.abs().amax()
            assert err < tol, (e, float(err))
            at += n


@pytest.mark.parametrize("target", TARGETS)
def test_portions_and_single_tokens_read_the_same_window(target, monkeypatch):
    """One long portion through worked-out keys and values, and the same rows through the latents."""
    g = torch.Generator().manual_seed(1)
    H, D, Dv, C, window = 5, 32, 24, 64, 50
    w = dev(bf16_values((H * (D + Dv), C), g, C ** -0.5), target)
    b, _, rows = ragged([100, 130], [30, 0], target[0], windows=[window])
    q, cache = dev(bf16_values((230, H, D), g), target), dev(bf16_values((rows, 1, C), g), target)
    a = M.latent_attention(q, cache, w, Dv, b, 0.5, window)
    monkeypatch.setattr(M, "SHORT_PORTION", 1000)
    z = M.latent_attention(q, cache, w, Dv, b, 0.5, window)
    assert (a - z).abs().max() < (1e-5 if target[1] == torch.float32 else 0.05)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("nq,nc", [(40, 48), (18, 30), (1536, 512), (7, 21)])
def test_latents_are_normed_and_cached(nq, nc, target):
    g = torch.Generator().manual_seed(nq)
    b, _, rows = ragged([1, 20], [33, 7], target[0])
    x, wq, wc = bf16_values((21, nq + nc), g, 3.0), bf16_values((nq,), g), bf16_values((nc,), g)
    cache = torch.full((rows, 1, nc), 9.0, dtype=target[1], device=target[0])
    b.slots[3] = -1                                    # a padding row leaves the cache alone
    cq = M.latent_norm_append(dev(x, target), f32(wq, target), f32(wc, target), 1e-3, b, cache).double().cpu()
    want_q, want_c = plain.plain_norm(x[:, :nq], wq, 1e-3), plain.plain_norm(x[:, nq:], wc, 1e-3)
    tol = 1e-5 if target[1] == torch.float32 else 0.02
    assert (cq - want_q).abs().max() < tol * want_q.abs().max()
    at, keep = b.slots.long().cpu(), [i for i in range(21) if i != 3]
    assert (cache.double().cpu()[at[keep], 0] - want_c[keep]).abs().max() < tol * want_c.abs().max()
    assert (cache == 9.0).all(-1).sum() == rows - 20


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("R,H,N,K", [(3, 5, 16, 24), (130, 3, 512, 72), (300, 2, 256, 128), (64, 33, 40, 136), (4, 3, 7, 9), (129, 4, 128, 64)])
def test_every_head_has_its_own_product(R, H, N, K, target):
    g = torch.Generator().manual_seed(R + N)
    x, w = bf16_values((R, H, K), g), bf16_values((H, N, K), g, K ** -0.5)
    want = torch.einsum("rhk,hnk->rhn", x, w)
    tol = 1e-5 if target[1] == torch.float32 else 0.02
    got = M.head_linear(dev(x, target), dev(w, target))
    assert (got.double().cpu() - want).abs().max() < tol * want.abs().max()
    got = M.head_linear(dev(x, target), dev(w.transpose(1, 2).contiguous(), target), w_kn=True)
    assert (got.double().cpu() - want).abs().max() < tol * want.abs().max()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H", [64, 60, 42, 2048, 5120])
def test_norm_behind_a_sublayer(H, target):
    g = torch.Generator().manual_seed(H)
    R, k, E = 6, 2, 4
    h, resid, w, w2 = bf16_values((R, H), g, 3.0), torch.randn(R, H, generator=g, dtype=torch.float64), bf16_values((H,), g), bf16_values((H,), g)
    tol = 1e-5 if target[1] == torch.float32 else 0.02

    def check(src, dense, mult, offset, nxt, off_next):
        r = f32(resid, target).contiguous()
        x = M.post_norm(src, f32(w, target), r, 1e-3, mult, offset, None if nxt is None else f32(nxt, target), off_next)
        want_r = resid.float().double() + mult * plain.plain_norm(dense, offset + w, 1e-3)
        assert (r.double().cpu() - want_r).abs().max() < 1e-5 * want_r.abs().max()      # the residual sum is 32-bit whatever the activations are
        want = want_r if nxt is None else plain.plain_norm(want_r, off_next + nxt, 1e-3)
        assert x.dtype == target[1] and (x.double().cpu() - want).abs().max() < tol * want.abs().max()
    check(dev(h, target), h, 0.3, 1.0, None, 0.0)
    check(dev(h, target), h, 1.0, 0.0, w2, 1.0)
    wide = torch.cat([h, h], 1)
    check(dev(wide, target)[:, :H], h, 0.5, 1.0, None, 0.0)                             # rows of a wider product
    # experts: rows in expert order, each token's k of them summed, a shared output added
    rt = OF.moe_route(torch.randn(R, E, generator=g).to(target[0]), k, sigmoid=True, norm=False, want_host=False)
    y = bf16_values((R * k, H), g)
    inv = rt.inv.long().cpu().view(R, k)
    check(M.ExpertSum(dev(y, target), rt, dev(h, target)), y[inv].sum(1) + h, 0.5, 1.0, w2, 1.0)
    check(M.ExpertSum(dev(y, target), rt, None), y[inv].sum(1), 0.5, 1.0, None, 0.0)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H", [64, 42])
def test_token_and_position_vectors_are_added(H, target):
    g = torch.Generator().manual_seed(H)
    table, pos_table = bf16_values((9, H), g), bf16_values((30, H), g)
    ids, pos = torch.tensor([3, 0, 8, 3]), torch.tensor([0, 1, 29, 17])
    for pt in (pos_table, None):
        r, x = M.embed_rows(ids.int().to(target[0]), dev(table, target), pos.int().to(target[0]), None if pt is None else dev(pt, target))
        want = table[ids] + (0 if pt is None else pt[pos])
        assert r.dtype == torch.float32 and torch.equal(r.double().cpu(), want.float().double())       # not rounded to the activations' type
        assert x.dtype == target[1] and torch.equal(x.cpu(), want.float().to(target[1]))


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("C", [48, 25])
def test_activations(C, target):
    g = torch.Generator().manual_seed(3)
    tol = 1e-5 if target[1] == torch.float32 else 0.02
    z = bf16_values((7, 2 * C), g, 3.0)
    got = M.gelu_erf(dev(z, target)).double().cpu()
    assert (got - plain.gelu_erf(z)).abs().max() < tol * z.abs().max()
    ids, table = torch.tensor([3, 0, 7, 7, 1, 2, 3]), bf16_values((8, 3 * C), g)
    got = M.side_gate(dev(z, target)[:, :C], ids.int().to(target[0]), dev(table, target), C).double().cpu()
    want = plain.gelu_tanh(z[:, :C]) * table[ids, C:2 * C]
    assert (got - want).abs().max() < tol * want.abs().max()

    def units(g_, u, limit):
        g_, u = g_.clamp(max=limit), u.clamp(-limit, limit)
        return g_ * plain.sigmoid(1.702 * g_) * (u + 1)
    got = M.glu_clamped(dev(z, target), 1.5, 1.702).double().cpu()
    assert (got - units(z[:, :C], z[:, C:], 1.5)).abs().max() < tol * 4
    rt = OF.moe_route(torch.randn(7, 5, generator=g).to(target[0]), 1, sigmoid=True, norm=False, want_host=False)
    w = rt.topw.reshape(-1)[rt.order.long()].double().cpu()[:, None] * torch.ones(1)
    got = M.glu_clamped(dev(z, target), 0.8, 1.702, rt).double().cpu()
    assert (got - units(w * z[:, :C], w * z[:, C:], 0.8)).abs().max() < tol * 4


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name,layer", [("mixed", 1), ("mixed", 3), ("odd", 0), ("wide", 1), ("rank512", 0)])
def test_experts_are_weighted_at_their_input(name, layer, target):
    from areal_b200.models.mixers import InputWeightedMLP

    cfg = CONFIGS[name]
    W, mlp, p = make_weights(cfg, seed=7), cfg["layers"][layer]["mlp"], f"l{layer}.mlp."
    block = make_model(cfg, W, target).layers[layer].mlp
    assert isinstance(block, InputWeightedMLP)
    x = bf16_values((40, cfg["width"]), torch.Generator().manual_seed(8))
    margins = [torch.ones(40)]
    want = plain.feed_forward(W, p, x, mlp, margins)
    with torch.no_grad():
        got = block(dev(x, target)).dense().double().cpu()
    assert_close(got, want, target[1], "experts", torch.stack([m.double() for m in margins]).amin(0) > 0.02)
    # weighting the output instead is something else
    chosen, s = plain.route(x, W[p + "router"], mlp["router"]["top"])
    out = torch.stack([sum(w * plain.expert(W, f"{p}e{e}.", x[t], mlp["expert"]["limit"]) for e, w in zip(chosen[t].tolist(), s[t])) for t in range(40)])
    if mlp.get("shared"):
        out = out + plain.expert(W, p + "shared.", x, mlp["shared"]["limit"])
    assert (out - want).pow(2).mean().sqrt() > 0.05 * want.pow(2).mean().sqrt()


# ----------------------------------------------------------------------------- engine
def greedy(W, cfg, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(plain.forward(W, cfg, t)[0][-1].argmax()))
    return t[len(prompt):]


@pytest.mark.parametrize("target", TARGETS)
def test_greedy_generation_through_the_engine(target):
    """More requests than slots, prompts absorbed in portions of at most 24 tokens beside decoding ones."""
    cfg = config((mixer(size=20), dense()), (mixer(size=31), moe()), vocab=40)
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
        assert (best - mine).max() < (1e-3 if target[1] == torch.float32 else 0.4)
        assert (mine - torch.tensor(r.output_logprobs, dtype=torch.float64)).abs().max() < (1e-3 if target[1] == torch.float32 else 0.4)
        if target[1] == torch.float32:
            assert r.output_tokens == greedy(W, cfg, p, 12)
    assert eng.stats["prefill_tokens"] > 0 and len(eng.cache.free) == eng.cache.num_pages and len(eng.cache.free_slots) == 2
    eng.destroy()


def test_generation_survives_a_short_pool_and_ends_with_the_positions():
    cfg = config((mixer(size=0), None), (mixer(size=30), None), vocab=40, positions=64)
    W = make_weights(cfg, seed=3)
    prompts = [tokens(20, cfg["vocab"], 40 + i) for i in range(3)]
    alone = [greedy(W, cfg, p, 30) for p in prompts]
    eng = make_engine(cfg, W, ("cpu", torch.float32), pages=6, page_size=16, slots=4, loop=True)
    res = generate(eng, prompts, 30)                   # three sequences of 50 tokens need 12 pages: someone is pre-empted
    assert [r.output_tokens for r in res] == alone and eng.stats["preempted"] > 0
    (r,) = generate(eng, prompts[:1], 100)             # every position has a learned vector: there are 64 of them
    assert r.stop_reason == "length" and len(r.output_tokens) == 64 - 20 and r.output_tokens[:30] == alone[0]
    with pytest.raises(ValueError):
        generate(eng, [tokens(65, cfg["vocab"], 1)], 4)
    c = eng.cache.open()
    eng.cache.grow(c, 65)
    with pytest.raises(ValueError):
        eng.runner.step([Entry(c, [1] * 65, [])])
    eng.destroy()


# ----------------------------------------------------------------------------- configuration, checkpoints, trace runner
def test_config_round_trip_and_errors(tmp_path):
    for name in ("tiny-vogilix", "vogilix-8b-layers"):
        mc = preset(name)
        mc.save_pretrained(str(tmp_path))
        back = ModelConfig.from_pretrained(str(tmp_path))
        assert back == mc and back.is_mixer_stack and back.num_params() > 0
    d = preset("tiny-vogilix").to_hf_dict()
    layer = d["layers"][1]
    bad_layer = (dict(layer, type="conv"), dict(layer, mlp=dict(layer["mlp"], kind="other")), dict(layer, mixer=dict(layer["mixer"], kv_rank=0)),
                 dict(layer, mlp=dict(layer["mlp"], router=dict(experts=4, top=5))))
    for bad in [dict(d, architecture="vogilix"), *(dict(d, layers=[b]) for b in bad_layer)]:
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(bad)


def test_checkpoint_round_trip(tmp_path):
    mc = preset("tiny-vogilix")
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


def test_two_designs_share_one_cache_rule():
    """Chunks and windows in one stack: a page goes back when the last layer that could see it cannot."""
    from areal_b200.engine.state_cache import StateCache
    from areal_b200.models.mixers import ChunkAttention, LatentAttention

    mc = preset("tiny-vogilix")
    chunked = ChunkAttention(mc, dict(heads=2, kv_heads=1, dim=8, vdim=8, scale=1.0, mask=dict(size=48)), torch.float32, "cpu")
    latent = LatentAttention(mc, mixer(size=20), torch.float32, "cpu")
    cache = StateCache([chunked, latent], 12, 16, 2, "cpu", torch.float32)
    assert cache.first_visible(60) == 41 and cache.first_visible(90) == 48 and cache.span == 48 and cache.windows == {20}
    c = cache.open()
    cache.grow(c, 100)
    cache.advance(c, 60)
    assert c.first_page == 41 // 16
    cache.advance(c, 40)
    assert c.first_page == 81 // 16 and len(c.pages) == 7 - 5
    cache.close(c)
    assert len(cache.free) == 12
    assert StateCache.bytes_per_page([chunked, latent], 16, 2) == (8 + 8 + 48) * 16 * 2


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
