"""Mixer stacks (Kagolix) against the plain statement in ``plain_stack.py``: every mechanism alone, whole prompts,
portions, single tokens, mixed batches on reused pages and slots, and greedy generation through the rollout engine.

Every case runs on the CPU ops, and on a GPU in 32-bit and bf16 (weights and inputs are bf16 values, so the oracle sees
the same numbers)."""
import asyncio
import json
import random

import pytest
import torch

from areal_b200.api.cli_args import GenerationHyperparameters, InferenceEngineConfig, NativeInferConfig
from areal_b200.api.io_struct import ModelRequest
from areal_b200.engine.infer_engine import NativeInferenceEngine
from areal_b200.engine.ragged_step import Entry
from areal_b200.models import hf_io
from areal_b200.models.config import ModelConfig, preset
from areal_b200.models.decoder import build_model
from areal_b200.ops import mixer_ops as M

from . import plain_stack as plain

TARGETS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda", torch.float32), id="cuda-f32", marks=pytest.mark.gpu),
           pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu)]


@pytest.fixture(autouse=True)
def _one_thread():
    """The oracle is made of very small operations: threads only cost time."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


TOL = {torch.float32: 2e-4, torch.bfloat16: 0.06}        # rms difference over rms


def attention(heads=4, kv=2, dim=32, vdim=32, size=48, softcap=20.0, scale=0.25):
    return "attention", dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, softcap=softcap, mask=dict(size=size))


def rglru(width=96, blocks=3, conv=4):
    return "rglru", dict(width=width, blocks=blocks, conv=conv)


def mamba2(heads=4, vdim=32, state=16, groups=2, norm_groups=2, conv=4):
    return "mamba2", dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv)


def dense(ff=80):
    return dict(kind="dense", ff=ff)


def moe(experts=6, top=2, ff=48):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def config(*layers, vocab=104, width=64, groups=2, cap=12.0, eps=1e-5):
    return dict(architecture="Kagolix", vocab=vocab, width=width, norm=dict(eps=eps, groups=groups), logit_softcap=cap,
                layers=[dict(type=t, mixer=m, mlp=f) for (t, m), f in layers])


CONFIGS = {
    "mixed": config((attention(), dense()), (mamba2(), moe()), (rglru(), moe()), (attention(size=72, kv=4, softcap=9.0), None)),
    # sizes that no vector width divides, one head group, experts of odd size, no grouping
    "odd": config((rglru(width=42, blocks=3, conv=2), moe(experts=5, top=3, ff=20)), (attention(heads=3, kv=1, dim=20, vdim=12, size=33), dense(36)),
                  (mamba2(heads=3, vdim=10, state=7, groups=1, norm_groups=3, conv=3), dense(33)), vocab=101, width=60, groups=3),
    # chunks longer than a page and than a query tile, several heads per group, wide values, states of two lane rows
    "wide": config((attention(heads=8, kv=2, dim=64, vdim=96, size=320), dense(96)), (mamba2(heads=2, vdim=64, state=64, groups=1, norm_groups=1), None),
                   (rglru(width=128, blocks=1, conv=1), dense(128)), width=128, groups=1, vocab=96),
    "dim128": config((attention(heads=2, kv=2, dim=128, vdim=128, size=200), dense(64)), (mamba2(heads=2, vdim=16, state=128, groups=2, norm_groups=4), None),
                     width=64, groups=4),
    "edges": config((attention(heads=2, kv=1, dim=96, vdim=64, size=64), dense()), (attention(heads=2, kv=1, dim=16, vdim=112, size=17), None)),
}


def bf16_values(shape, gen, std=1.0, mean=0.0):
    return (torch.randn(shape, generator=gen, dtype=torch.float64) * std + mean).bfloat16().double()


def make_weights(cfg, seed=0):
    """Random weights under the checkpoint's names (float64 holding bf16 values)."""
    g = torch.Generator().manual_seed(seed)
    H, V = cfg["width"], cfg["vocab"]
    W = {"embed": bf16_values((V, H), g), "head": bf16_values((V, H), g, 2 * H ** -0.5), "final.norm": bf16_values((H,), g, 0.2, 1.0)}

    def mat(name, *shape):
        W[name] = bf16_values(shape, g, shape[-1] ** -0.5)

    def vec(name, n, std=0.2, mean=1.0):
        W[name] = bf16_values(n if isinstance(n, tuple) else (n,), g, std, mean)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            vec(f"l{i}.{n}", H)
        if layer["type"] == "attention":
            q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            mat(p + "q", q, H), mat(p + "k", k, H), mat(p + "v", v, H), mat(p + "o", H, m["heads"] * m["vdim"])
            vec(p + "q.norm", q), vec(p + "k.norm", k)
            W[p + "r1"] = bf16_values((m["heads"],), g).abs()
            W[p + "r2"] = bf16_values((m["heads"],), g, 0.3).abs()
        elif layer["type"] == "rglru":
            n, w = m["blocks"], m["width"]
            mat(p + "y", w, H), mat(p + "x", w, H), mat(p + "o", H, w)
            mat(p + "ra", n, w // n, w // n), mat(p + "ri", n, w // n, w // n)
            for b in ("y.b", "x.b", "conv.b"):
                vec(p + b, w, 0.3, 0.0)
            vec(p + "ra.b", (n, w // n), 0.3, 0.0), vec(p + "ri.b", (n, w // n), 0.3, 0.0)
            W[p + "conv"] = bf16_values((w, m["conv"]), g, 0.5)
            vec(p + "lam", w, 1.5, -3.0)
        else:
            inner, bc = m["heads"] * m["vdim"], 2 * m["groups"] * m["state"]
            mat(p + "in", 2 * inner + bc + m["heads"], H), mat(p + "o", H, inner)
            W[p + "conv"] = bf16_values((inner + bc, m["conv"]), g, 0.5)
            vec(p + "conv.b", inner + bc, 0.2, 0.0), vec(p + "dt_bias", m["heads"], 1.0, -3.0), vec(p + "A_log", m["heads"], 1.0, -0.5)
            vec(p + "D", m["heads"]), vec(p + "norm", inner)
        f, p = layer["mlp"], f"l{i}.mlp."
        if f and f["kind"] == "dense":
            mat(p + "up", f["ff"], H), mat(p + "down", H, f["ff"])
            vec(p + "act", 2, 0.5, 0.3)
        elif f:
            E, I = f["router"]["experts"], f["expert"]["ff"]
            W[p + "router"] = bf16_values((E, H), g, 3 * H ** -0.5)
            vec(p + "correction", E, 0.2, 0.0)
            for e in range(E):
                mat(f"{p}e{e}.gate", I, H), mat(f"{p}e{e}.up", I, H), mat(f"{p}e{e}.down", H, I)
    return W


def make_model(cfg, W, target):
    device, dtype = target
    mc = ModelConfig.from_hf_dict(json.loads(json.dumps(cfg)))
    model = build_model(mc, dtype=dtype, device=device, seed=0)
    hf_io.load_hf_tensors_into(mc, {n: p.data for n, p in model.named_parameters()}, ((n, t.float()) for n, t in W.items()))
    return model


def make_engine(cfg, W, target, pages=24, page_size=64, slots=4, loop=False, **kw):
    ic = NativeInferConfig(page_size=page_size, num_pages=pages, max_running_requests=slots, context_length=4096, **kw)
    return NativeInferenceEngine(InferenceEngineConfig(), ic, model=make_model(cfg, W, target)).initialize(
        device=target[0], start_executor=False, start_loop=loop)


class Driver:
    """Steps requests through an engine's runner and collects every position's logits."""

    def __init__(self, eng):
        self.eng, self.live, self.out = eng, {}, {}

    def step(self, portions, end=()):
        entries = []
        for rid, toks in portions:
            c = self.live.setdefault(rid, None) or self.eng.cache.open()
            self.live[rid] = c
            assert self.eng.cache.grow(c, c.length + len(toks)), "pool exhausted"
            entries.append(Entry(c, list(toks), list(range(len(toks)))))
        logits = self.eng.runner.step(entries).double().cpu()
        at = 0
        for rid, toks in portions:
            self.out.setdefault(rid, []).append(logits[at:at + len(toks)])
            at += len(toks)
        for rid in end:
            self.eng.cache.close(self.live.pop(rid))

    def logits(self, rid):
        return torch.cat(self.out[rid])


def tokens(n, vocab, seed):
    r = random.Random(seed)
    return [r.randrange(vocab) for _ in range(n)]


def assert_close(got, want, dtype, what="", sure=None):
    """``sure``: rows whose choice of experts is clear (bf16 rounding may turn a close one, which is another result)."""
    scale = want.pow(2).mean().sqrt()
    err = (got - want).pow(2).mean(-1).sqrt() / scale
    if sure is not None and dtype == torch.bfloat16:
        assert len(sure) < 20 or sure.double().mean() > 0.6
        err = err * sure
    assert torch.isfinite(got).all() and err.max() < TOL[dtype], f"{what}: row {int(err.argmax())} off by {float(err.max()):.2e}"


_ORACLE: dict = {}


def oracle(name, n, seed):
    """Tokens, logits and rows with a clear choice of experts of a random prompt under a named configuration (cached:
    shared by the targets and the schedules)."""
    if (name, n, seed) not in _ORACLE:
        cfg = CONFIGS[name]
        t = tokens(n, cfg["vocab"], seed)
        margins = [torch.ones(n)]
        logits = plain.forward(make_weights(cfg), cfg, t, margins)[0]
        _ORACLE[name, n, seed] = (t, logits, torch.stack([m.double() for m in margins]).amin(0) > 0.02)
    return _ORACLE[name, n, seed]


# ----------------------------------------------------------------------------- schedules
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_portions_and_single_tokens_agree(name, target):
    cfg = CONFIGS[name]
    eng = make_engine(cfg, make_weights(cfg), target)
    n = 150
    t, want, sure = oracle(name, n, 1)
    cuts = {"whole": [n], "decoded": [100] + [1] * 50, "pairs": [2] * 35 + [80], "ragged": [1, 2, 61, 3, 64, 2, 1, 16]}
    for what, sizes in cuts.items():
        d, at = Driver(eng), 0
        assert sum(sizes) == n
        for s in sizes:
            d.step([("a", t[at:at + s])], end=["a"] if at + s == n else [])
            at += s
        assert_close(d.logits("a"), want, target[1], f"{name} {what}", sure)
    assert len(eng.cache.free) == eng.cache.num_pages and len(eng.cache.free_slots) == eng.cache.num_slots


@pytest.mark.parametrize("target", TARGETS)
def test_long_prompt_and_long_decoding_cross_many_chunks(target):
    name = "wide"
    cfg = CONFIGS[name]
    n = 700
    t, want, sure = oracle(name, n, 2)
    eng = make_engine(cfg, make_weights(cfg), target)
    d = Driver(eng)
    d.step([("a", t)], end=["a"])
    assert_close(d.logits("a"), want, target[1], "whole", sure)
    d = Driver(eng)
    d.step([("a", t[:300])])
    for i in range(300, 345):                      # decoding walks over the chunk border at 320
        d.step([("a", t[i:i + 1])])
    assert d.live["a"].first_page == 320 // 64     # nothing before the border can be seen any more
    d.step([("a", t[345:637])])
    for i in range(637, n):                        # and the next one at 640
        d.step([("a", t[i:i + 1])], end=["a"] if i == n - 1 else [])
    assert_close(d.logits("a"), want, target[1], "decoded", sure)


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
        assert_close(d.logits(rid), ref[rid][1], target[1], rid, ref[rid][2])
    assert len(eng.cache.free) == eng.cache.num_pages


@pytest.mark.parametrize("target", TARGETS)
def test_layer_outputs_match(target):
    cfg = CONFIGS["mixed"]
    W = make_weights(cfg)
    t = tokens(70, cfg["vocab"], 5)
    _, states = plain.forward(W, cfg, t)
    eng = make_engine(cfg, W, target)
    c, seen = eng.cache.open(), []
    eng.cache.grow(c, 70)
    eng.runner.step([Entry(c, t, [69])], on_layer=lambda i, r: seen.append(r.double().cpu().clone()))
    for i, (a, b) in enumerate(zip(seen, states)):
        assert_close(a, b, target[1], f"layer {i}")


# ----------------------------------------------------------------------------- mechanisms
def ragged(lens, starts, device, page_size=16, seed=0, windows=()):
    """A RaggedBatch of entries with scattered pages; single-token entries come first. ``windows``: sliding windows of
    latent layers, whose page lists the batch gets."""
    import numpy as np

    from areal_b200.engine.ragged_step import RaggedRunner
    from areal_b200.engine.state_cache import Carried

    total = sum(-(-(s + n) // page_size) for n, s in zip(lens, starts))
    order = list(range(total))
    random.Random(seed).shuffle(order)
    entries = []
    for i, (n, s) in enumerate(zip(lens, starts)):
        pages = [order.pop() for _ in range(-(-(s + n) // page_size))]
        entries.append(Entry(Carried(slot=len(lens) - 1 - i, pages=pages, length=s), [0] * n, []))
    runner = RaggedRunner.__new__(RaggedRunner)
    runner.device = torch.device(device)
    runner.cache = type("C", (), dict(page_size=page_size, has_kv=True, windows=windows))
    b, _ = RaggedRunner._layout(runner, entries)
    assert np.all(np.diff([len(e.tokens) != 1 for e in entries]) >= 0)
    return b, entries, total * page_size


def dev(x, target):
    return x.to(target[0]).to(target[1])


def f32(x, target):
    return x.to(target[0]).float()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("D,Dv,Hq,Hkv,chunk,cap", [(32, 32, 4, 2, 48, 5.0), (96, 64, 6, 2, 112, 24.0), (64, 128, 2, 1, 0, 0.0), (20, 12, 3, 1, 33, 8.0),
                                                  (128, 128, 16, 1, 200, 15.0), (8, 40, 2, 2, 1, 3.0), (128, 72, 2, 2, 512, 0.0)])
def test_chunk_attention(D, Dv, Hq, Hkv, chunk, cap, target):
    """Portions and single tokens against all earlier keys. One key per chunk edge, page edge and far end is made to stand
    out for the queries that must (or must not) see it."""
    g = torch.Generator().manual_seed(D + Dv)
    lens, starts = [1, 1, 1, 130, 300, 2], [0, 47, 333, 0, 70, 118]
    b, entries, rows = ragged(lens, starts, target[0])
    kc = torch.zeros(rows, Hkv, D, dtype=target[1], device=target[0])
    vc = torch.zeros(rows, Hkv, Dv, dtype=target[1], device=target[0])
    r1, r2 = torch.rand(Hq, generator=g).double(), torch.rand(Hq, generator=g).double()
    r1[0] = 0.02
    qs, ks, vs = [], [], []
    for n, s in zip(lens, starts):
        L = n + s
        q, k, v = bf16_values((L, Hq, D), g), bf16_values((L, Hkv, D), g), bf16_values((L, Hkv, Dv), g)
        base = bf16_values((D,), g)
        edges = {0, 1, 15, 16, L - 1} | {c * chunk + o for c in range(1, L // max(chunk, 20) + 1) for o in (-1, 0) if chunk > 20}
        for j in edges:
            if 0 <= j < L:
                k[j] = base                          # scores of these keys stand out for the queries below
        q[-2:] = base * 1.5
        q[chunk - 1:chunk + 2] = base * 1.5
        qs.append(q), ks.append(k), vs.append(v)
    for e, ent in enumerate(entries):
        L = lens[e] + starts[e]
        j = torch.arange(L)
        at = (torch.tensor(ent.carry.pages)[j // 16] * 16 + j % 16).to(target[0])
        kc[at], vc[at] = dev(ks[e], target), dev(vs[e], target)
    q_rows = torch.cat([q[s:] for q, s in zip(qs, starts)])
    scale = 0.7 * D ** -0.5
    got = M.chunk_attention(dev(q_rows, target).contiguous(), kc, vc, b, scale, cap, f32(r1, target), f32(r2, target), chunk).double().cpu()
    at = 0
    for e, (n, s) in enumerate(zip(lens, starts)):
        want = plain.attend(qs[e], ks[e], vs[e], scale, cap, r1.float().double(), r2.float().double(), chunk)[s:]
        err = (got[at:at + n] - want).abs().amax()
        assert err < (1e-4 if target[1] == torch.float32 else 0.03), (e, float(err))
        at += n


def test_chunk_attention_without_distance_bias_or_cap_is_softmax_attention():
    g = torch.Generator().manual_seed(1)
    b, entries, rows = ragged([40], [0], "cpu")
    k, v, q = torch.randn(40, 2, 16, generator=g), torch.randn(40, 2, 8, generator=g), torch.randn(40, 4, 16, generator=g)
    kc, vc = torch.zeros(rows, 2, 16), torch.zeros(rows, 2, 8)
    kc[b.slots.long()], vc[b.slots.long()] = k, v
    got = M.chunk_attention(q, kc, vc, b, 0.25)
    want = torch.nn.functional.scaled_dot_product_attention(q.transpose(0, 1), k.transpose(0, 1).repeat_interleave(2, 0),
                                                            v.transpose(0, 1).repeat_interleave(2, 0), is_causal=True, scale=0.25)
    assert torch.allclose(got, want.transpose(0, 1), atol=1e-5)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,groups", [(64, 1), (64, 4), (96, 12), (60, 3), (42, 1), (2048, 2), (5120, 20)])
def test_grouped_norms(H, groups, target):
    g = torch.Generator().manual_seed(H)
    h, resid = bf16_values((5, H), g, 3.0), torch.randn(5, H, generator=g, dtype=torch.float64)
    w1, w2, z = bf16_values((H,), g), bf16_values((H,), g), bf16_values((5, H), g)
    ids, table = torch.tensor([3, 0, 7, 7, 1]), bf16_values((8, H), g)
    tol = 1e-5 if target[1] == torch.float32 else 0.02
    r = f32(resid, target).contiguous()
    x = M.sandwich_norm(dev(h, target), f32(w1, target), r, f32(w2, target), groups, 1e-3)
    want_r = resid.float().double() + plain.root_mean_square_norm(h, w1, 1e-3, groups)
    assert (r.double().cpu() - want_r).abs().max() < 1e-5          # the residual sum is 32-bit whatever the activations are
    want = plain.root_mean_square_norm(want_r, w2, 1e-3, groups)
    assert (x.double().cpu() - want).abs().max() < tol * want.abs().max()
    r, x = M.embed_norm(ids.to(target[0]).int(), dev(table, target), f32(w2, target), groups, 1e-3)
    assert torch.equal(r.double().cpu(), table[ids])
    want = plain.root_mean_square_norm(table[ids], w2, 1e-3, groups)
    assert (x.double().cpu() - want).abs().max() < tol * want.abs().max()
    y = torch.randn(5, H, generator=g, dtype=torch.float64).float().double()
    got = M.gated_group_norm(f32(y, target), dev(z, target), f32(w1, target), groups, 1e-3).double().cpu()
    want = plain.root_mean_square_norm(y * plain.silu(z), w1, 1e-3, groups)
    assert (got - want).abs().max() < tol * want.abs().max()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("C,K,silu", [(48, 4, True), (33, 3, False), (130, 1, True), (64, 2, False), (20, 6, False)])
def test_causal_conv_carries_its_tail(C, K, silu, target):
    g = torch.Generator().manual_seed(C)
    L = 150
    x, bin_ = bf16_values((L, C), g), bf16_values((C,), g)
    w, bias = bf16_values((C, K), g), bf16_values((C,), g)
    want = plain.causal_conv(x + bin_, w, bias)
    want = plain.silu(want) if silu else want
    for sizes in ([L], [1] * 5 + [2, 1, 2, 70, 70], [149, 1]):
        tail = torch.full((1, C, K - 1), 7.0, device=target[0])      # what the slot's last user left
        at, got = 0, []
        for n in sizes:
            b, _, _ = ragged([n], [at], target[0])
            wide = dev(torch.cat([x[at:at + n], x[at:at + n]], 1), target)[:, C:]          # rows of a wider product
            got.append(M.causal_conv(wide, f32(bin_, target), f32(w, target), f32(bias, target), silu, b, tail).double().cpu())
            at += n
            if at == L:
                break
        got = torch.cat(got)
        assert (got - want[:at]).abs().max() < (1e-4 if target[1] == torch.float32 else 0.05)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("n,bs", [(3, 32), (5, 72), (1, 21), (2, 64)])
def test_rglru_state_follows_the_sequence(n, bs, target):
    g = torch.Generator().manual_seed(bs)
    W, L = n * bs, 140
    u, y = bf16_values((L, W), g), bf16_values((L, W), g)
    p = {k: bf16_values(s, g, std, mean) for k, s, std, mean in (("yb", (W,), 0.3, 0), ("gw", (2, n, bs, bs), bs ** -0.5, 0),
                                                                ("gb", (2, n, bs), 0.5, 0), ("lam", (W,), 1.5, -3.0))}
    ub = u.view(L, n, bs)
    r, i = (plain.sigmoid(torch.einsum("lnk,nok->lno", ub, p["gw"][k]) + p["gb"][k]).reshape(L, W) for k in (0, 1))
    la = -8 * r * plain.softplus(p["lam"])
    h, want = torch.zeros(W, dtype=torch.float64), []
    for t in range(L):
        h = torch.exp(la[t]) * h + torch.sqrt(1 - torch.exp(2 * la[t])) * i[t] * u[t]
        want.append(h * plain.gelu_tanh(y[t] + p["yb"]))
    want = torch.stack(want)
    for sizes in ([L], [1, 2, 1, 66, 70], [3, 136, 1]):
        S, at, got = torch.full((1, W), 5.0, device=target[0]), 0, []
        for m in sizes:
            b, _, _ = ragged([m], [at], target[0])
            got.append(M.rglru(dev(u[at:at + m], target).contiguous(), dev(y[at:at + m], target), f32(p["yb"], target), dev(p["gw"], target).contiguous(),
                               f32(p["gb"], target).contiguous(), f32(p["lam"], target), b, S).double().cpu())
            at += m
        assert (torch.cat(got) - want).abs().max() < (1e-4 if target[1] == torch.float32 else 0.03)
        assert (S[0].double().cpu() - h).abs().max() < 1e-4           # gates and state are 32-bit also beside bf16 activations


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,P,N,G", [(4, 32, 16, 2), (2, 64, 128, 1), (3, 10, 7, 1), (6, 40, 32, 3), (2, 16, 64, 2)])
def test_mamba2_state_follows_the_sequence(H, P, N, G, target):
    g = torch.Generator().manual_seed(P * N)
    L, I = 200, H * P
    xbc, dt = bf16_values((L, I + 2 * G * N), g), bf16_values((L, H), g)
    dtb, Al, D = bf16_values((H,), g, 1.0, -3.0), bf16_values((H,), g, 1.0, -0.5), bf16_values((H,), g)
    x, B, C = xbc[:, :I].view(L, H, P), xbc[:, I:I + G * N].view(L, G, N), xbc[:, I + G * N:].view(L, G, N)
    step = plain.softplus(dt + dtb)
    S, want = torch.zeros(H, P, N, dtype=torch.float64), []
    for t in range(L):
        rep = [hd // (H // G) for hd in range(H)]
        S = torch.exp(-torch.exp(Al) * step[t])[:, None, None] * S + step[t][:, None, None] * x[t][:, :, None] * B[t][rep][:, None, :]
        want.append(((S * C[t][rep][:, None, :]).sum(-1) + D[:, None] * x[t]).reshape(-1))
    want = torch.stack(want)
    for sizes in ([L], [1, 2, 1, 66, 130], [3, 196, 1]):
        state, at, got = torch.full((1, H, P, N), 3.0, device=target[0]), 0, []
        for m in sizes:
            b, _, _ = ragged([m], [at], target[0])
            got.append(M.mamba2_scan(dev(xbc[at:at + m], target).contiguous(), dev(dt[at:at + m], target).contiguous(), f32(dtb, target), f32(Al, target),
                                     f32(D, target), H, P, N, G, b, state).double().cpu())
            at += m
        scale = want.abs().max()
        assert (torch.cat(got) - want).abs().max() < 2e-4 * scale
        assert (state[0].double().cpu() - S).abs().max() < 2e-4 * S.abs().max()


@pytest.mark.parametrize("target", TARGETS)
def test_feed_forward_pieces(target):
    g = torch.Generator().manual_seed(3)
    tol = 1e-5 if target[1] == torch.float32 else 0.02
    z, pq = bf16_values((7, 50), g, 3.0), bf16_values((2,), g)
    got = M.xielu(dev(z, target), f32(pq, target)).double().cpu()
    assert (got - plain.xielu(z, *pq)).abs().max() < tol * plain.xielu(z, *pq).abs().max()
    got = M.glu_silu(dev(z, target)).double().cpu()
    assert (got - plain.silu(z[:, :25]) * z[:, 25:]).abs().max() < tol * 20
    logits = torch.randn(7, 33, generator=g, dtype=torch.float64) * 9
    got = M.softcap_(f32(logits, target).clone(), 5.0).double().cpu()
    assert (got - 5 * torch.tanh(logits / 5)).abs().max() < 1e-5


@pytest.mark.parametrize("target", TARGETS)
def test_router_chooses_with_the_correction_and_weighs_without(target):
    """An expert that the scores put last is chosen because of its correction, with its small score as weight; the weights
    of a token do not add up to one."""
    from areal_b200.models.mixers import RoutedMLP

    cfg = CONFIGS["mixed"]
    W = make_weights(cfg, seed=7)
    layer = 1
    p = f"l{layer}.mlp."
    W[p + "correction"] = torch.tensor([0.0, 0.0, 3.0, 0.0, -3.0, 0.0], dtype=torch.float64)
    model = make_model(cfg, W, target)
    mlp = model.layers[layer].mlp
    assert isinstance(mlp, RoutedMLP)
    x = bf16_values((40, cfg["width"]), torch.Generator().manual_seed(8))
    chosen, weight = plain.route(x, W[p + "router"], W[p + "correction"], 2)
    assert (chosen == 2).any(-1).all() and not (chosen == 4).any() and (weight.sum(-1) < 0.999).any()
    want = plain.feed_forward(W, p, x, cfg["layers"][layer]["mlp"])
    with torch.no_grad():
        got = mlp(dev(x, target)).double().cpu()
    assert_close(got, want, target[1], "experts")


# ----------------------------------------------------------------------------- engine
def greedy(W, cfg, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(plain.forward(W, cfg, t)[0][-1].argmax()))
    return t[len(prompt):]


def generate(eng, prompts, n, **kw):
    g = GenerationHyperparameters(max_new_tokens=n, max_tokens=2000, greedy=True, ignore_eos=True, **kw)

    async def run():
        return await asyncio.gather(*[eng.agenerate(ModelRequest(rid=f"q{i}", input_ids=list(p), gconfig=g)) for i, p in enumerate(prompts)])
    return asyncio.run(run())


@pytest.mark.parametrize("target", TARGETS)
def test_greedy_generation_through_the_engine(target):
    """More requests than slots, prompts absorbed in portions of at most 24 tokens beside decoding ones."""
    cfg = config((attention(size=20), dense()), (mamba2(), moe()), (rglru(), None), vocab=40)
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
        assert (best - mine).max() < (1e-3 if target[1] == torch.float32 else 0.3)
        assert (mine - torch.tensor(r.output_logprobs, dtype=torch.float64)).abs().max() < (1e-3 if target[1] == torch.float32 else 0.3)
        if target[1] == torch.float32:
            assert r.output_tokens == greedy(W, cfg, p, 12)
    assert eng.stats["prefill_tokens"] > 0 and len(eng.cache.free) == eng.cache.num_pages and len(eng.cache.free_slots) == 2
    eng.destroy()


def test_generation_survives_a_short_pool_and_a_pause():
    cfg = config((attention(size=500), None), (rglru(), None), vocab=40)
    W = make_weights(cfg, seed=3)
    prompts = [tokens(20, cfg["vocab"], 40 + i) for i in range(3)]
    alone = [greedy(W, cfg, p, 30) for p in prompts]
    eng = make_engine(cfg, W, ("cpu", torch.float32), pages=6, page_size=16, slots=4, loop=True)
    res = generate(eng, prompts, 30)                   # three sequences of 50 tokens need 12 pages: someone is pre-empted
    assert [r.output_tokens for r in res] == alone and eng.stats["preempted"] > 0
    eng.pause_generation()
    eng.offload()
    assert eng.cache is None
    eng.onload()
    assert [r.output_tokens for r in generate(eng, prompts[:1], 30)] == alone[:1]
    eng.destroy()


def test_weight_update_reaches_the_served_model():
    cfg = config((attention(), dense()), vocab=40)
    eng = make_engine(cfg, make_weights(cfg, 0), ("cpu", torch.float32), loop=True)
    W = make_weights(cfg, 1)
    fresh = make_model(cfg, W, ("cpu", torch.float32))
    eng.update_weights_from_tensors({n: p.detach() for n, p in fresh.named_parameters()}).result()
    p = tokens(9, 40, 1)
    assert generate(eng, [p], 6)[0].output_tokens == greedy(W, cfg, p, 6)
    eng.destroy()


# ----------------------------------------------------------------------------- configuration, checkpoints, trace runner
def test_config_round_trip_and_errors(tmp_path):
    mc = preset("tiny-kagolix")
    mc.save_pretrained(str(tmp_path))
    back = ModelConfig.from_pretrained(str(tmp_path))
    assert back == mc and back.is_mixer_stack and back.num_params() > 0
    d = mc.to_hf_dict()
    for bad in (dict(d, architecture="Other"), dict(d, layers=[dict(type="conv", mixer={}, mlp=None)]), dict(d, norm=dict(eps=1e-6, groups=7)),
                dict(d, layers=[dict(type="rglru", mixer=dict(width=10, blocks=3, conv=2), mlp=None)])):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(bad)


def test_checkpoint_round_trip(tmp_path):
    mc = preset("tiny-kagolix")
    a, b = (build_model(mc, dtype=torch.float32, seed=s) for s in (1, 2))
    hf_io.save_model_hf(a, str(tmp_path))
    hf_io.load_model_hf(b, str(tmp_path))
    for (n, p), (_, q) in zip(a.named_parameters(), b.named_parameters()):
        assert torch.equal(p, q), n
    with pytest.raises(NotImplementedError):
        a(torch.tensor([1, 2]), torch.tensor([0, 2], dtype=torch.int32))


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
    ta, wa, sure = oracle(name, 97, 12)
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
    assert_close(got[0], wa[[3, 89]], target[1], sure=sure[[3, 89]])
    assert_close(got[2], torch.stack([wa[96], wa[92], wb[1]]), target[1])
    assert_close(got[3], wb[[6]], target[1])
    assert len(eng.cache.free) == 4 and len(eng.cache.free_slots) == 4
