"""Serving throughput of a mixer stack beside the framework's closest existing models at equal layer sizes, and the time of
every kernel against its roofline (``bench.py --workload mixer-serve``). Random weights, synthetic tokens, one GPU.

Kernel times are CUDA events around one launch with the L2 flushed in between (a 256 MB buffer is written); step times
are CUDA events around whole steps of the serving path, whose weights alone exceed L2."""
from __future__ import annotations

import json
import math
import os
import time

import torch
import torch.nn.functional as F

from ..ops import functional as OF
from ..ops import lib as oplib
from ..ops import mixer_ops as M

ROOT = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))


def peaks() -> tuple[float, float, str]:
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12, "measured"
    except (OSError, KeyError, ValueError):
        return 6.65e12, 1.59e15, "fallback"


def timed(fn, iters: int = 10, warmup: int = 3, flush=None) -> float:
    """Median seconds of one call."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    ts = []
    for _ in range(iters):
        if flush is not None:
            flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        b.synchronize()
        ts.append(a.elapsed_time(b) * 1e-3)
    return sorted(ts)[len(ts) // 2]


def _batch(lens, starts, dev, page_size=64, windows=()):
    """A ragged batch over consecutive pages; single-token entries first. Returns (batch, cache rows)."""
    from ..engine.ragged_step import Entry, RaggedRunner
    from ..engine.state_cache import Carried

    ents, at = [], 0
    for i, (n, s) in enumerate(zip(lens, starts)):
        k = -(-(n + s) // page_size)
        ents.append(Entry(Carried(slot=i, pages=list(range(at, at + k)), length=s), [1] * n, []))
        at += k
    r = RaggedRunner.__new__(RaggedRunner)
    r.device = torch.device(dev)
    r.cache = type("C", (), dict(page_size=page_size, has_kv=True, windows=windows))
    return RaggedRunner._layout(r, ents)[0], at * page_size


def kernel_table(cfg, prefill=(4, 2048), decode=(64, 960), dev="cuda") -> list[dict]:
    """Time, roofline time and fraction of the new design's kernels, each beside the like kernel of the existing models.
    ``prefill`` = (sequences, tokens each), ``decode`` = (sequences, cached tokens each)."""
    bw, fl, _ = peaks()
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    bf = dict(device=dev, dtype=torch.bfloat16)
    f32 = dict(device=dev, dtype=torch.float32)
    rows = []

    def add(name, fn, nbytes=0.0, flops=0.0, like=None):
        t = timed(fn, flush=flush)
        roof = max(nbytes / bw, flops / fl)
        rows.append(dict(kernel=name, us=round(t * 1e6, 1), roofline_us=round(roof * 1e6, 1), fraction=round(roof / t, 3), like=like))

    H = cfg.hidden_size
    spec = {e["type"]: e["mixer"] for e in cfg.mixer_layers}
    at, m2, lr = spec["attention"], spec["mamba2"], spec["rglru"]
    B, L = prefill
    T = B * L
    pb, prow = _batch([L] * B, [0] * B, dev)
    nB, ctx = decode
    db, drow = _batch([1] * nB, [ctx] * nB, dev)
    w = torch.ones(H, **f32)
    for tag, R in (("prefill", T), ("decode", nB)):
        h, res = torch.randn(R, H, **bf), torch.randn(R, H, **f32)
        add(f"sandwich_norm {tag}", lambda: M.sandwich_norm(h, w, res, w, cfg.norm_groups, 1e-6), R * H * 12, like=f"rmsnorm {tag}")
        r16, w16 = res.bfloat16(), w.bfloat16()
        with torch.no_grad():
            add(f"rmsnorm {tag}", lambda: OF.rmsnorm(h, w16, 1e-6, r16), R * H * 8)
    # attention
    nq, nk, D, Dv = at["heads"], at["kv_heads"], at["dim"], at["vdim"]
    chunk = at["mask"]["size"]
    r1, r2 = torch.rand(nq, **f32), torch.rand(nq, **f32)
    for tag, b, R, rows_ in (("prefill", pb, T, prow), ("decode", db, nB, drow)):
        kc, vc, q = torch.randn(rows_, nk, D, **bf), torch.randn(rows_, nk, Dv, **bf), torch.randn(R, nq, D, **bf)
        qkv = torch.randn(R, nq * D + nk * (D + Dv), **bf)
        wq, wk = torch.ones(nq * D, **f32), torch.ones(nk * D, **f32)
        add(f"qk_norm_append {tag}", lambda: M.qk_norm_append(qkv, wq, wk, 1e-6, b, kc, vc, nq), qkv.numel() * 4)
        if tag == "prefill":
            pairs = B * sum(p % chunk + 1 for p in range(L))
            fn = lambda: M.chunk_attention(q, kc, vc, b, D ** -0.5, at["softcap"], r1, r2, chunk)      # noqa: E731
            add("chunk_attention prefill", fn, (q.numel() * 2 + (nk * (D + Dv)) * T) * 2, 2.0 * nq * (D + Dv) * pairs, like="attn_fwd prefill")
            if D == Dv and D in (64, 128):
                k, v = torch.randn(T, nk, D, **bf), torch.randn(T, nk, D, **bf)
                cu = torch.arange(0, T + 1, L, device=dev, dtype=torch.int32)
                ti = OF.attn_tile_table(cu, T)
                add("attn_fwd prefill", lambda: OF.attention_fwd(q, k, v, cu, True, D ** -0.5, ti), 0, 4.0 * nq * D * B * L * (L + 1) / 2)
        else:
            see = ctx % chunk + 1
            add("chunk_attention decode", lambda: M.chunk_attention(q, kc, vc, b, D ** -0.5, at["softcap"], r1, r2, chunk), nB * see * nk * (D + Dv) * 2,
                like="paged_decode decode")
            if D == Dv and D in (64, 128):
                lens = torch.full((nB,), ctx + 1, device=dev, dtype=torch.int32)
                po, ml = torch.empty(nB * nq * 4 * D, **f32), torch.empty(nB * nq * 8, **f32)
                o = torch.empty_like(q)

                def paged():
                    oplib.check(oplib.get_lib().ab2_paged_decode_strided(
                        q.data_ptr(), kc.data_ptr(), vc.data_ptr(), b.pages.data_ptr(), lens.data_ptr(), po.data_ptr(), ml.data_ptr(), o.data_ptr(), nB, nq,
                        nk, D, 64, b.pages.shape[1], 4, D ** -0.5, q.stride(0), oplib.stream_ptr()), "paged_decode")
                add("paged_decode decode", paged, nB * (ctx + 1) * nk * 2 * D * 2)
    # recurrences
    Hm, P, N, G = m2["heads"], m2["vdim"], m2["state"], m2["groups"]
    I, C = Hm * P, Hm * P + 2 * G * N
    dtb, Al, Dd = torch.randn(Hm, **f32) - 4, torch.rand(Hm, **f32), torch.ones(Hm, **f32)
    W, nb_ = lr["width"], lr["blocks"]
    gw, gb, lam = torch.randn(2, nb_, W // nb_, W // nb_, **bf) * 0.05, torch.zeros(2, nb_, W // nb_, **f32), torch.full((W,), -3.0, **f32)
    for tag, b, R, ne in (("prefill", pb, T, B), ("decode", db, nB, nB)):
        x, taps = torch.randn(R, I + C + Hm, **bf), m2["conv"]
        cw, cb, tail = torch.randn(C, taps, **f32), torch.randn(C, **f32), torch.zeros(ne, C, taps - 1, **f32)
        add(f"causal_conv {tag}", lambda: M.causal_conv(x[:, I:I + C], None, cw, cb, True, b, tail), R * C * 4 + (ne * C * (taps - 1) * 8))
        xbc, S = torch.randn(R, C, **bf), torch.zeros(ne, Hm, P, N, **f32)
        add(f"mamba2_scan {tag}", lambda: M.mamba2_scan(xbc, x[:, I + C:], dtb, Al, Dd, Hm, P, N, G, b, S), R * (C * 2 + I * 4) + 2 * S.numel() * 4, 0,
            like=f"gated_delta_rule {tag}")
        y, nw = torch.randn(R, I, **f32), torch.ones(I, **f32)
        add(f"gated_group_norm {tag}", lambda: M.gated_group_norm(y, x[:, :I], nw, m2["norm_groups"], 1e-6), R * I * 8)
        yx, SL, yb = torch.randn(R, 2 * W, **bf), torch.zeros(ne, W, **f32), torch.zeros(W, **f32)
        u = torch.randn(R, W, **bf)
        add(f"rglru {tag}", lambda: M.rglru(u, yx[:, :W], yb, gw, gb, lam, b, SL), R * W * 6 + gw.numel() * 2 + 2 * SL.numel() * 4,
            4.0 * R * W * (W // nb_), like=f"gated_delta_rule {tag}")
        # the existing linear-attention rule at the same state size (heads x 128 x 64 / 128)
        from ..models.hybrid import gated_delta_rule_chunked, gated_delta_rule_recurrent

        shp = (ne, R // ne, Hm)
        q_, k_ = torch.randn(*shp, N, **f32), F.normalize(torch.randn(*shp, N, **f32), dim=-1)
        v_, g_, be = torch.randn(*shp, P, **f32), -torch.rand(*shp, **f32), torch.rand(*shp, **f32)
        rule = gated_delta_rule_chunked if tag == "prefill" else gated_delta_rule_recurrent
        S0 = torch.zeros(ne, Hm, N, P, **f32)
        add(f"gated_delta_rule {tag}", lambda: rule(q_, k_, v_, g_, be, state=S0), R * Hm * (2 * N + 2 * P) * 2 + 2 * S0.numel() * 4)
    # feed-forward pieces
    ff = max([e["mlp"]["ff"] for e in cfg.mixer_layers if e["mlp"] and e["mlp"]["kind"] == "dense"], default=4 * H)
    pq = torch.ones(2, **f32)
    for tag, R in (("prefill", T), ("decode", nB)):
        x = torch.randn(R, ff, **bf)
        add(f"xielu {tag}", lambda: M.xielu(x, pq), R * ff * 4, like=f"swiglu {tag}")
        gu = torch.randn(R, 2 * ff, **bf)
        add(f"glu_silu {tag}", lambda: M.glu_silu(gu), R * ff * 6, like=f"swiglu {tag}")
        with torch.no_grad():
            add(f"swiglu {tag}", lambda: OF.swiglu(gu), R * ff * 6)
        lg = torch.randn(min(R, 256), cfg.vocab_size, **f32)
        add(f"softcap {tag}", lambda: M.softcap_(lg, 30.0), lg.numel() * 8)
        moe = next((e["mlp"] for e in cfg.mixer_layers if e["mlp"] and e["mlp"]["kind"] == "moe"), None)
        if moe:
            E, k, If = moe["router"]["experts"], moe["router"]["top"], moe["expert"]["ff"]
            rt = OF.moe_route(torch.randn(R, E, **f32), k, norm=False, want_probs=False, want_host=False)
            ys, wgu, wd = torch.randn(R * k, H, **bf), torch.randn(E, 2 * If, H, **bf), torch.randn(E, H, If, **bf)
            hh = torch.randn(R * k, If, **bf)
            live = min(E, R * k)
            add(f"expert_linear up {tag}", lambda: M.expert_linear(ys, wgu, rt), (live * 2 * If * H + R * k * (H + 2 * If)) * 2, 4.0 * R * k * H * If)
            add(f"expert_linear down {tag}", lambda: M.expert_linear(hh, wd, rt), (live * If * H + R * k * (H + If)) * 2, 2.0 * R * k * H * If)
            add(f"expert_combine {tag}", lambda: M.expert_combine(ys, rt, rt.topw), R * (k + 1) * H * 2, like=f"gather and sum {tag}")
            add(f"gather and sum {tag}", lambda: (ys.index_select(0, rt.inv).view(R, k, H) * rt.topw.to(ys.dtype).unsqueeze(-1)).sum(1), R * (k + 1) * H * 2)
    return rows


def latent_kernel_table(cfg, prefill=(4, 2048), decode=(64, 960), dev="cuda") -> list[dict]:
    """As :func:`kernel_table`, for a stack of latent attention (Vogilix)."""
    bw, fl, _ = peaks()
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    bf = dict(device=dev, dtype=torch.bfloat16)
    f32 = dict(device=dev, dtype=torch.float32)
    rows = []

    def add(name, fn, nbytes=0.0, flops=0.0, like=None):
        t = timed(fn, flush=flush)
        roof = max(nbytes / bw, flops / fl)
        rows.append(dict(kernel=name, us=round(t * 1e6, 1), roofline_us=round(roof * 1e6, 1), fraction=round(roof / t, 3), like=like))

    Hd, V = cfg.hidden_size, cfg.vocab_size
    at = cfg.mixer_layers[0]["mixer"]
    nq, D, Dv, rq, C, scale = at["heads"], at["dim"], at["vdim"], at["q_rank"], at["kv_rank"], at["scale"]
    windows = sorted({e["mixer"]["mask"]["size"] for e in cfg.mixer_layers})
    dense = next(e["mlp"] for e in cfg.mixer_layers if e["mlp"] and e["mlp"]["kind"] == "dense")
    moe = next(e["mlp"] for e in cfg.mixer_layers if e["mlp"] and e["mlp"]["kind"] == "moe")
    E, k, If, Is = moe["router"]["experts"], moe["router"]["top"], moe["expert"]["ff"], moe["shared"]["ff"]
    (B, L), (nB, ctx) = prefill, decode
    pb, prow = _batch([L] * B, [0] * B, dev, windows=windows)
    db, drow = _batch([1] * nB, [ctx] * nB, dev, windows=windows)
    w, wrq, wc = torch.zeros(Hd, **f32), torch.ones(rq, **f32), torch.ones(C, **f32)
    w_kv = torch.randn(nq * (D + Dv), C, **bf) * C ** -0.5
    w_k, w_v = w_kv[:nq * D].view(nq, D, C), w_kv[nq * D:].view(nq, Dv, C)
    table, ptab = torch.randn(V, Hd, **bf), torch.randn(cfg.max_position_embeddings, Hd, **bf)
    side, sd = torch.randn(V, cfg.num_layers * cfg.token_side_dim, **bf), cfg.token_side_dim
    for tag, b, R, rows_ in (("prefill", pb, B * L, prow), ("decode", db, nB, drow)):
        # norms, embedding
        h, res = torch.randn(R, Hd, **bf), torch.randn(R, Hd, **f32)
        ids = torch.randint(0, V, (R,), device=dev, dtype=torch.int32)
        add(f"embed_rows {tag}", lambda: M.embed_rows(ids, table, b.pos, ptab), R * Hd * 10, like=f"embedding {tag}")
        with torch.no_grad():
            add(f"embedding {tag}", lambda: OF.embedding(ids.long(), table), R * Hd * 4)
        add(f"post_norm {tag}", lambda: M.post_norm(h, w, res, 1e-6, 0.5, 1.0), R * Hd * 12, like=f"rmsnorm {tag}")
        r16, w16 = res.bfloat16(), w.bfloat16()
        with torch.no_grad():
            add(f"rmsnorm {tag}", lambda: OF.rmsnorm(h, w16, 1e-6, r16), R * Hd * 8)
        # attention
        x, cache = torch.randn(R, rq + C, **bf), torch.randn(rows_, 1, C, **bf)
        add(f"latent_norm_append {tag}", lambda: M.latent_norm_append(x, wrq, wc, 1e-6, b, cache), x.numel() * 4, like=f"qk_norm_append {tag}")
        kc, vc, wq_ = torch.randn(rows_, 1, 128, **bf), torch.randn(rows_, 1, 128, **bf), torch.ones(rq + C - 256, **f32)
        add(f"qk_norm_append {tag}", lambda: M.qk_norm_append(x, wq_, wc[:128], 1e-6, b, kc, vc, (rq + C - 256) // 128), x.numel() * 4)
        q = torch.randn(R, nq, D, **bf)
        if tag == "prefill":
            seen = pb.seen[windows[-1]]
            add("latents gathered prefill", lambda: cache.view(-1, 64 * C).index_select(0, seen.pages), R * C * 4)
            rows_c = cache.view(-1, C)[:R]
            add("keys and values prefill (GEMM)", lambda: M.linear(rows_c, w_kv), (R * C + w_kv.numel() + R * nq * (D + Dv)) * 2, 2.0 * R * C * nq * (D + Dv))
            for win in windows:
                pairs = B * sum(min(p + 1, win) for p in range(L))
                flops = 2.0 * nq * (D + Dv) * pairs
                kv, out = M.linear(rows_c, w_kv), torch.empty(R, nq, Dv, **bf)
                sn = pb.seen[win]

                def attn():
                    M._call("ab2_chunk_prefill", q.data_ptr(), pb.cu.data_ptr(), pb.start.data_ptr(), pb.tiles.data_ptr(), pb.tiles.shape[0], out.data_ptr(), R,
                            kv.shape[0], kv.stride(0), kv.stride(0), kv.data_ptr(), kv[:, nq * D:].data_ptr(), sn.table.data_ptr(), sn.base.data_ptr(),
                            sn.table.shape[1], 64, nq, nq, D, Dv, scale, 0.0, None, None, 0, win, None)
                add(f"window attention {win} prefill", attn, (q.numel() + out.numel() + kv.numel()) * 2, flops, like="attn_fwd prefill")
                add(f"latent_attention {win} prefill (all of it)", lambda: M.latent_attention(q, cache, w_kv, Dv, pb, scale, win),
                    (q.numel() * 2 + R * C) * 2, flops + 2.0 * R * C * nq * (D + Dv))
            if D == Dv and D in (64, 128):
                k_, v_ = torch.randn(R, nq, D, **bf), torch.randn(R, nq, D, **bf)
                cu = torch.arange(0, R + 1, L, device=dev, dtype=torch.int32)
                ti = OF.attn_tile_table(cu, R)
                add("attn_fwd prefill", lambda: OF.attention_fwd(q, k_, v_, cu, True, D ** -0.5, ti), q.numel() * 8, 4.0 * nq * D * B * L * (L + 1) / 2)
        else:
            qc, oc = torch.randn(R, nq, C, **bf), torch.empty(R, nq, C, **bf)
            add("head_linear of the queries decode", lambda: M.head_linear(q, w_k, w_kn=True), (q.numel() + qc.numel() + w_k.numel()) * 2, 2.0 * R * nq * D * C,
                like="linear of the same weight bytes decode")
            add("head_linear of the values decode", lambda: M.head_linear(qc, w_v), (q.numel() + qc.numel() + w_v.numel()) * 2, 2.0 * R * nq * Dv * C,
                like="linear of the same weight bytes decode")
            xl, wl = torch.randn(R, C, **bf), torch.randn(nq * D, C, **bf)
            add("linear of the same weight bytes decode", lambda: M.linear(xl, wl), (xl.numel() + wl.numel() + R * nq * D) * 2, 2.0 * R * nq * D * C)
            for win in windows:
                see = min(ctx + 1, win)

                def dec():
                    M._call("ab2_latent_decode", qc.data_ptr(), b.pos.data_ptr(), b.slots.data_ptr(), b.row_entry.data_ptr(), oc.data_ptr(), R,
                            cache.data_ptr(), cache.shape[0], b.pages.data_ptr(), b.page_base.data_ptr(), b.pages.shape[1], 64, nq, C, scale, win, None)
                add(f"latent_decode {win} decode", dec, (R * see * C + 2 * qc.numel()) * 2, 4.0 * R * see * nq * C, like="paged_decode decode")
            # as many bytes as the paged kernel below reads: four times the sequences
            b4, rows4 = _batch([1] * (4 * nB), [ctx] * (4 * nB), dev, windows=windows)
            cache4, qc4 = torch.randn(rows4, 1, C, **bf), torch.randn(4 * nB, nq, C, **bf)
            oc4, see = torch.empty_like(qc4), min(ctx + 1, windows[-1])

            def dec4():
                M._call("ab2_latent_decode", qc4.data_ptr(), b4.pos.data_ptr(), b4.slots.data_ptr(), b4.row_entry.data_ptr(), oc4.data_ptr(), 4 * nB,
                        cache4.data_ptr(), cache4.shape[0], b4.pages.data_ptr(), b4.page_base.data_ptr(), b4.pages.shape[1], 64, nq, C, scale, windows[-1],
                        None)
            add(f"latent_decode {windows[-1]} decode, {4 * nB} sequences", dec4, (4 * nB * see * C + 2 * qc4.numel()) * 2, 16.0 * nB * see * nq * C,
                like="paged_decode decode")
            nk = max(1, nq // 4)
            kc, vc = torch.randn(rows_, nk, 128, **bf), torch.randn(rows_, nk, 128, **bf)
            q2 = torch.randn(R, nq, 128, **bf)
            lens = torch.full((nB,), ctx + 1, device=dev, dtype=torch.int32)
            po, ml, o = torch.empty(nB * nq * 4 * 128, **f32), torch.empty(nB * nq * 8, **f32), torch.empty_like(q2)

            def paged():
                oplib.check(oplib.get_lib().ab2_paged_decode_strided(
                    q2.data_ptr(), kc.data_ptr(), vc.data_ptr(), b.pages.data_ptr(), lens.data_ptr(), po.data_ptr(), ml.data_ptr(), o.data_ptr(), nB, nq, nk,
                    128, 64, b.pages.shape[1], 4, 128 ** -0.5, q2.stride(0), oplib.stream_ptr()), "paged_decode")
            add("paged_decode decode", paged, nB * (ctx + 1) * nk * 256 * 2)
        # feed-forwards and the token input
        ff = dense["ff"]
        z, gu = torch.randn(R, ff, **bf), torch.randn(R, 2 * ff, **bf)
        add(f"gelu_erf {tag}", lambda: M.gelu_erf(z), R * ff * 4, like=f"swiglu {tag}")
        with torch.no_grad():
            add(f"swiglu {tag}", lambda: OF.swiglu(gu), R * ff * 6)
        rw, x16 = torch.randn(E, Hd, **bf), torch.randn(R, Hd, **bf)
        add(f"router_logits {tag}", lambda: M.router_logits(x16, rw), (R * Hd + E * Hd) * 2 + R * E * 4, 2.0 * R * E * Hd, like=f"router in the routed decoder {tag}")
        add(f"router in the routed decoder {tag}", lambda: F.linear(x16.float(), rw.float()), (R * Hd + E * Hd) * 2 + R * E * 4, 2.0 * R * E * Hd)
        rt = OF.moe_route(torch.randn(R, E, **f32), k, sigmoid=True, norm=False, want_probs=False, want_host=False)
        eg = torch.randn(R * k, 2 * If, **bf)
        add(f"glu_clamped experts {tag}", lambda: M.glu_clamped(eg, 6.0, 1.702, rt), R * k * If * 6, like=f"swiglu {tag}")
        sg = torch.randn(R, 2 * Is, **bf)
        add(f"glu_clamped shared {tag}", lambda: M.glu_clamped(sg, 7.0, 1.702), R * Is * 6, like=f"swiglu {tag}")
        y, sh = torch.randn(R * k, Hd, **bf), torch.randn(R, Hd, **bf)
        add(f"post_norm of experts {tag}", lambda: M.post_norm(M.ExpertSum(y, rt, sh), w, res, 1e-6, 0.5, 1.0), R * Hd * (2 * k + 12), like=f"gather and sum {tag}")
        add(f"gather and sum {tag}", lambda: (y.index_select(0, rt.inv).view(R, k, Hd) * rt.topw.to(y.dtype).unsqueeze(-1)).sum(1), R * (k + 1) * Hd * 2)
        g = torch.randn(R, sd, **bf)
        add(f"side_gate {tag}", lambda: M.side_gate(g, ids, side, 0), R * sd * 6, like=f"swiglu {tag}")
    return rows


def looped_kernel_table(cfg, prefill=(4, 2048), decode=(64, 960), dev="cuda") -> list[dict]:
    """As :func:`kernel_table`, for a stack of parallel branches and latent attention with positions (Bumotar), each kernel beside
    the like one of the other mixer stacks at the same sizes."""
    bw, fl, _ = peaks()
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    bf = dict(device=dev, dtype=torch.bfloat16)
    f32 = dict(device=dev, dtype=torch.float32)
    rows = []

    def add(name, fn, nbytes=0.0, flops=0.0, like=None):
        t = timed(fn, flush=flush)
        roof = max(nbytes / bw, flops / fl)
        rows.append(dict(kernel=name, us=round(t * 1e6, 1), roofline_us=round(roof * 1e6, 1), fraction=round(roof / t, 3), like=like))

    Hd, V = cfg.hidden_size, cfg.vocab_size
    p = next(e["mixer"] for e in cfg.mixer_layers if e["type"] == "parallel")
    at = next(e["mixer"] for e in cfg.mixer_layers if e["type"] == "latent_attention")
    moe = next(e["mlp"] for e in cfg.mixer_layers if e["mlp"])
    lf, rt_ = p["left"], p["right"]
    nq, nk, D, Dv, win, cap = lf["heads"], lf["kv_heads"], lf["dim"], lf["vdim"], lf["mask"]["size"], lf["softcap"]
    Hr, N, P = rt_["heads"], rt_["dim"], rt_["vdim"]
    nl, Dl, r, Dvl, C, scale = at["heads"], at["dim"], at["rot_dim"], at["vdim"], at["kv_rank"], at["scale"]
    E, k, If, Is = moe["router"]["experts"], moe["router"]["top"], moe["expert"]["ff"], moe["shared"]["ff"]
    (B, L), (nB, ctx) = prefill, decode
    pb, prow = _batch([L] * B, [0] * B, dev, windows=(0,))
    db, drow = _batch([1] * nB, [ctx] * nB, dev, windows=(0,))
    w, wc, wh = torch.ones(Hd, **f32), torch.ones(C, **f32), torch.ones(D, **f32)
    half, hl, hr = lf["rot"]["dims"] // 2, r // 2, rt_["rot"]["dims"] // 2
    freq, mult = torch.rand(half + hl + hr, device=dev, dtype=torch.float64), torch.ones(half + hl + hr, **f32)
    w_kv = torch.randn(nl * (Dl + Dvl), C, **bf) * C ** -0.5
    w_k, w_v = w_kv[:nl * Dl].view(nl, Dl, C), w_kv[nl * Dl:].view(nl, Dvl, C)
    sink, decay = torch.randn(nl, **f32), torch.tensor(rt_["decay"], **f32)
    table = torch.randn(V, Hd, **bf)
    for tag, b, R, rows_, ne in (("prefill", pb, B * L, prow, B), ("decode", db, nB, drow, nB)):
        ids = torch.randint(0, V, (R,), device=dev, dtype=torch.int32)
        both = torch.empty(R, 2 * Hd, **bf)
        add(f"embed_rows into both halves {tag}", lambda: M.embed_rows(ids, table, b.pos, None, both[:, Hd:], both[:, :Hd]), R * Hd * 10, like=f"embed_rows {tag}")
        add(f"embed_rows {tag}", lambda: M.embed_rows(ids, table, b.pos), R * Hd * 8)
        add(f"rotary_table {tag}", lambda: M.rotary_table(b.pos, freq, mult), R * (4 + 8 * freq.numel()), like=f"embed_rows {tag}")
        cs = M.rotary_table(b.pos, freq, mult)
        # residual sums and norms
        h, res, res2 = torch.randn(R, Hd, **bf), torch.randn(R, Hd, **f32), torch.randn(R, Hd, **f32)
        add(f"residual_norm {tag}", lambda: M.residual_norm(h, res, w, 1e-6, torch.bfloat16), R * Hd * 12, like=f"post_norm {tag}")
        add(f"post_norm {tag}", lambda: M.post_norm(h, w, res2, 1e-6, 0.5, 1.0), R * Hd * 12)
        rt = OF.moe_route(torch.randn(R, E, **f32), k, want_probs=False, want_host=False)
        y, sh, lg = torch.randn(R * k, Hd, **bf), torch.randn(R, Hd, **bf), torch.randn(R, E + 8, **f32)
        add(f"residual_norm of experts {tag}", lambda: M.residual_norm(M.ExpertSum(y, rt, sh, rt.topw, lg[:, E]), res, w, 1e-6, torch.bfloat16),
            R * Hd * (2 * k + 12), like=f"post_norm of experts {tag}")
        add(f"post_norm of experts {tag}", lambda: M.post_norm(M.ExpertSum(y, rt, sh), w, res2, 1e-6, 0.5, 1.0), R * Hd * (2 * k + 12))
        eg = torch.randn(R * k, 2 * If, **bf)
        add(f"glu_silu experts {tag}", lambda: M.glu_silu(eg), R * k * If * 6, like=f"glu_clamped experts {tag}")
        add(f"glu_clamped experts {tag}", lambda: M.glu_clamped(eg, 6.0, 1.702, rt), R * k * If * 6)
        sg = torch.randn(R, 2 * Is, **bf)
        add(f"glu_silu shared {tag}", lambda: M.glu_silu(sg), R * Is * 6, like=f"glu_clamped shared {tag}")
        add(f"glu_clamped shared {tag}", lambda: M.glu_clamped(sg, 7.0, 1.702), R * Is * 6)
        # windowed attention, beside the chunked one that sees the same number of keys, with its distance bias
        nin = nq * D + nk * (D + Dv) + nq * Dv
        z = torch.randn(R, nin, **bf)
        kc, vc = torch.randn(rows_, nk, D, **bf), torch.randn(rows_, nk, Dv, **bf)
        add(f"qk_head_norm_append {tag}", lambda: M.qk_head_norm_append(z, wh, wh, 1e-6, cs[:, :half], False, b, kc, vc, nq), R * (nin - nq * Dv) * 4 + R * half * 8,
            like=f"qk_norm_append {tag}")
        wq, wk = torch.ones(nq * D, **f32), torch.ones(nk * D, **f32)
        add(f"qk_norm_append {tag}", lambda: M.qk_norm_append(z, wq, wk, 1e-6, b, kc, vc, nq), R * (nin - nq * Dv) * 4)
        q, o = torch.randn(R, nq, D, **bf), torch.empty(R, nq * Dv + Hr * P, **bf)
        gate, r1, r2 = z[:, nin - nq * Dv:], torch.rand(nq, **f32), torch.rand(nq, **f32)
        pairs = B * sum(min(x + 1, win) for x in range(L)) if tag == "prefill" else nB * min(ctx + 1, win)
        kv_bytes = (nk * (D + Dv)) * 2 * (R if tag == "prefill" else pairs)
        flops = 2.0 * nq * (D + Dv) * pairs
        add(f"window attention {tag}", lambda: M.chunk_attention(q, kc, vc, b, D ** -0.5, cap, window=win, sink=0.0, gate=gate, out_scale=0.7, out=o[:, :nq * Dv]),
            q.numel() * 2 + R * nq * Dv * 4 + kv_bytes, flops, like=f"chunk_attention {tag}")
        seen = B * sum(x % win + 1 for x in range(L)) if tag == "prefill" else nB * (ctx % win + 1)
        add(f"chunk_attention {tag}", lambda: M.chunk_attention(q, kc, vc, b, D ** -0.5, cap, r1, r2, win), q.numel() * 2 + R * nq * Dv * 2 +
            (nk * (D + Dv)) * 2 * (R if tag == "prefill" else seen), 2.0 * nq * (D + Dv) * seen)
        # retention, beside the Mamba-2 recurrence of the same state, and its norm
        zr, S = torch.randn(R, Hr * (2 * N + 2 * P), **bf), torch.zeros(ne, Hr, P, N, **f32)
        ro = o[:, nq * Dv:]
        log2 = torch.log2(decay)
        rot_r = cs[:, half + hl:]
        # (its output is bf16 and gated; 32-bit rows between its two kernels in prompts)
        add(f"retention {tag}", lambda: M.retention(zr, decay, log2, rot_r, 1e-6, 0.4, ro, Hr, N, P, b, S),
            zr.numel() * 2 + R * Hr * P * (10 if tag == "prefill" else 2) + R * hr * 8 + 2 * S.numel() * 4, like=f"mamba2_scan and norm {tag}")
        Cm = Hr * P + 2 * Hr * N
        xbc, dtr, dd = torch.randn(R, Cm, **bf), torch.randn(R, Hr, **bf), torch.ones(Hr, **f32)
        zg, nw = torch.randn(R, Hr * P, **bf), torch.ones(Hr * P, **f32)
        add(f"mamba2_scan and norm {tag}", lambda: M.gated_group_norm(M.mamba2_scan(xbc, dtr, dd, dd, dd, Hr, P, N, Hr, b, S), zg, nw, Hr, 1e-6),
            (xbc.numel() + dtr.numel()) * 2 + R * Hr * P * 12 + 2 * S.numel() * 4)
        if tag == "prefill":
            yr = torch.empty(R, Hr * P, **f32)

            def blocks():
                M._call("ab2_retention_portions", zr.data_ptr(), zr.stride(0), rot_r.data_ptr(), rot_r.stride(0) // 2, hr, decay.data_ptr(), log2.data_ptr(),
                        N ** -0.5, b.cu.data_ptr(), b.start.data_ptr(), b.state.data_ptr(), 0, B, S.data_ptr(), yr.data_ptr(), Hr, N, P, 1, 0)
            add("retention_blocks prefill", blocks, R * Hr * (2 * N + P) * 2 + yr.numel() * 4 + 2 * S.numel() * 4, like="mamba2_scan prefill")
            add("mamba2_scan prefill", lambda: M.mamba2_scan(xbc, dtr, dd, dd, dd, Hr, P, N, Hr, b, S), (xbc.numel() + dtr.numel()) * 2 + R * Hr * P * 4 + 2 * S.numel() * 4)
        # latent attention, beside the one without positions
        ld = nl * (Dl + r) + C + r + nl
        zl, cache, cache0 = torch.randn(R, ld, **bf), torch.randn(rows_, 1, C + r, **bf), torch.randn(rows_, 1, C, **bf)
        add(f"latent_rope_append {tag}", lambda: M.latent_rope_append(zl, wc, 1e-6, cs[:, half:half + hl], True, b, cache, nl, Dl),
            R * (2 * nl * r + 2 * (C + r)) * 2 + R * hl * 8, like=f"latent_norm_append {tag}")
        wql = torch.ones(1536, **f32)
        xl = torch.randn(R, 1536 + C, **bf)
        add(f"latent_norm_append {tag}", lambda: M.latent_norm_append(xl, wql, wc, 1e-6, b, cache0), xl.numel() * 4)
        ql, q0 = zl[:, :nl * (Dl + r)].unflatten(1, (nl, Dl + r)), torch.randn(R, nl, Dl, **bf)
        gl = zl[:, ld - nl:]
        if tag == "prefill":
            pairs = B * L * (L + 1) // 2
            out = torch.empty(R, nl, Dvl, **bf)
            sn = pb.seen[0]
            rows_c = cache.view(-1, C + r)
            kv = M.linear(rows_c[:, :C], w_kv)
            x = M._extra(sink, gl, True, ldq=ld, hsq=Dl + r, q2=ql[:, :, Dl:].data_ptr(), ldq2=ld, hsq2=Dl + r, D2=r, k2=rows_c[:, C:].data_ptr(), ldk2=C + r)

            def tiles(q_, extra):
                M._call("ab2_chunk_prefill", q_.data_ptr(), pb.cu.data_ptr(), pb.start.data_ptr(), pb.tiles.data_ptr(), pb.tiles.shape[0], out.data_ptr(), R,
                        kv.shape[0], kv.stride(0), kv.stride(0), kv.data_ptr(), kv[:, nl * Dl:].data_ptr(), sn.table.data_ptr(), sn.base.data_ptr(),
                        sn.table.shape[1], 64, nl, nl, Dl, Dvl, scale, 0.0, None, None, 0, 0, extra)
            add("attention with shared key part prefill", lambda: tiles(ql, M.ctypes.byref(x)), 0, 2.0 * nl * (Dl + r + Dvl) * pairs, like="attention prefill")
            add("attention prefill", lambda: tiles(q0, None), 0, 2.0 * nl * (Dl + Dvl) * pairs)
            wb = 2.0 * R * C * nl * (Dl + Dvl)
            add("latent attention with positions prefill (all of it)", lambda: M.latent_attention(ql, cache, w_kv, Dvl, b, scale, 0, r, sink, gl), 0,
                2.0 * nl * (Dl + r + Dvl) * pairs + wb, like="latent_attention prefill (all of it)")
            add("latent_attention prefill (all of it)", lambda: M.latent_attention(q0, cache0, w_kv, Dvl, b, scale, 0), 0, 2.0 * nl * (Dl + Dvl) * pairs + wb)
        else:
            for n, (bb, rw) in ((nB, (db, drow)), (4 * nB, _batch([1] * (4 * nB), [ctx] * (4 * nB), dev, windows=(0,)))):
                qc, oc = torch.randn(n, nl, C, **bf), torch.empty(n, nl, C, **bf)
                zz = torch.randn(n, ld, **bf)
                qq, ca, ca0 = zz[:, :nl * (Dl + r)].unflatten(1, (nl, Dl + r)), torch.randn(rw, 1, C + r, **bf), torch.randn(rw, 1, C, **bf)
                xd = M._extra(sink, zz[:, ld - nl:], True, ldk=C + r, q2=qq[:, :, Dl:].data_ptr(), ldq2=ld, hsq2=Dl + r, D2=r, k2=ca[:, :, C:].data_ptr(), ldk2=C + r)

                def dec(c_, extra):
                    M._call("ab2_latent_decode", qc.data_ptr(), bb.pos.data_ptr(), bb.slots.data_ptr(), bb.row_entry.data_ptr(), oc.data_ptr(), n, c_.data_ptr(),
                            c_.shape[0], bb.pages.data_ptr(), bb.page_base.data_ptr(), bb.pages.shape[1], 64, nl, C, scale, 0, extra)
                t = "" if n == nB else f", {n} sequences"
                add(f"latent_decode with positions{t}", lambda: dec(ca, M.ctypes.byref(xd)), (n * (ctx + 1) * (C + r) + 2 * qc.numel() + n * nl * r) * 2,
                    2.0 * n * (ctx + 1) * nl * (2 * C + r), like=f"latent_decode{t}")
                add(f"latent_decode{t}", lambda: dec(ca0, None), (n * (ctx + 1) * C + 2 * qc.numel()) * 2, 4.0 * n * (ctx + 1) * nl * C)
            add("head_linear of strided queries decode", lambda: M.head_linear(ql[:, :, :Dl], w_k, w_kn=True), (R * nl * (Dl + C) + w_k.numel()) * 2, 2.0 * R * nl * Dl * C,
                like="head_linear of the queries decode")
            add("head_linear of the queries decode", lambda: M.head_linear(q0, w_k, w_kn=True), (R * nl * (Dl + C) + w_k.numel()) * 2, 2.0 * R * nl * Dl * C)
        wl = torch.randn(Hd, 2 * Hd, **bf)
        add(f"entrance of a pass {tag} (GEMM, 32-bit sums)", lambda: M.linear(both, wl, fp32_out=True), (both.numel() + wl.numel()) * 2 + R * Hd * 4,
            4.0 * R * Hd * Hd, like=f"the same product, bf16 {tag}")
        add(f"the same product, bf16 {tag}", lambda: M.linear(both, wl), (both.numel() + wl.numel()) * 2 + R * Hd * 2, 4.0 * R * Hd * Hd)
        rw_, x16 = torch.randn(-(-(E + 1) // 8) * 8, Hd, **bf), torch.randn(R, Hd, **bf)
        add(f"router_logits and gate {tag}", lambda: M.router_logits(x16, rw_), (R * Hd + E * Hd) * 2 + R * E * 4, 2.0 * R * E * Hd, like=f"router_logits {tag}")
        rw0 = rw_[:E]
        add(f"router_logits {tag}", lambda: M.router_logits(x16, rw0), (R * Hd + E * Hd) * 2 + R * E * 4, 2.0 * R * E * Hd)
    return rows


def shifted_kernel_table(cfg, prefill=(4, 2048), decode=(64, 960), dev="cuda") -> list[dict]:
    """As :func:`kernel_table`, for a stack with a token shift, rotated attention and attention beside minGRU (Goganex), each kernel
    beside the like one of the other stacks and decoders at the same sizes."""
    bw, fl, _ = peaks()
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    bf = dict(device=dev, dtype=torch.bfloat16)
    f32 = dict(device=dev, dtype=torch.float32)
    rows = []

    def add(name, fn, nbytes=0.0, flops=0.0, like=None):
        t = timed(fn, flush=flush)
        roof = max(nbytes / bw, flops / fl)
        rows.append(dict(kernel=name, us=round(t * 1e6, 1), roofline_us=round(roof * 1e6, 1), fraction=round(roof / t, 3), like=like))

    Hd, V, ff = cfg.hidden_size, cfg.vocab_size, cfg.intermediate_size
    at = next(e["mixer"] for e in cfg.mixer_layers if e["type"] == "attention")
    p = next(e["mixer"] for e in cfg.mixer_layers if e["type"] == "parallel")
    nq, nk, D, Dv = at["heads"], at["kv_heads"], at["dim"], at["vdim"]
    lq, lk, Dl, W = p["left"]["heads"], p["left"]["kv_heads"], p["left"]["dim"], p["right"]["width"]
    half, blocks = at["rot"]["dims"] // 2, W // 256
    (B, L), (nB, ctx) = prefill, decode
    pb, prow = _batch([L] * B, [0] * B, dev)
    db, drow = _batch([1] * nB, [ctx] * nB, dev)
    w, share, table, dt = torch.ones(Hd, **f32), torch.rand(Hd, **f32), torch.randn(V, Hd, **bf), torch.bfloat16
    freq, mult, temp = torch.rand(half, device=dev, dtype=torch.float64), torch.ones(half, **f32), torch.ones(nq, **f32)
    for tag, b, R, rows_, ne in (("prefill", pb, B * L, prow, B), ("decode", db, nB, drow, nB)):
        one = tag == "decode"
        # the stream: sums, norms, shift (a portion's stream goes from one buffer to another)
        ids = torch.randint(0, V, (R,), device=dev, dtype=torch.int32)
        h, h2, res, S = torch.randn(R, Hd, **bf), torch.randn(R, Hd, **bf), torch.randn(R, Hd, **f32), torch.zeros(ne, Hd, **f32)
        slot = 2 * ne * Hd * 4
        add(f"embedding, norm, shift {tag}", lambda: M.stream_norm(M.EmbeddingRows(ids, table, 4.0), None, w, 1e-6, dt, None, share, b, S), R * Hd * 8 + slot,
            like=f"embed_rows {tag}")
        add(f"embed_rows {tag}", lambda: M.embed_rows(ids, table, b.pos), R * Hd * 8)
        add(f"residual sum, norm, shift {tag}", lambda: M.stream_norm(h, res, w, 1e-6, dt, None, share, b, S), R * Hd * 12 + slot, like=f"residual_norm {tag}")
        add(f"residual_norm {tag}", lambda: M.residual_norm(h, res, w, 1e-6, dt), R * Hd * 12)
        pair = M.BranchSum(h, h2, w, w, 0.5, 1e-6)
        add(f"normed branches, norm, shift {tag}", lambda: M.stream_norm(pair, res, w, 1e-6, dt, None, share, b, S), R * Hd * 14 + slot, like=f"sandwich_norm {tag}")
        add(f"normed branches, norm {tag}", lambda: M.residual_norm(pair, res, w, 1e-6, dt), R * Hd * 14, like=f"sandwich_norm {tag}")
        add(f"sandwich_norm {tag}", lambda: M.sandwich_norm(h, w, res, w, 1, 1e-6), R * Hd * 12)
        # queries and keys
        cs = M.rotary_table(b.pos, freq, mult)
        z, wh = torch.randn(R, nq * D + nk * (D + Dv), **bf), torch.ones(D, **f32)
        kc, vc = torch.randn(rows_, nk, D, **bf), torch.randn(rows_, nk, Dv, **bf)
        add(f"turn, unit norm, append {tag}", lambda: M.qk_head_norm_append(z, None, None, 1e-6, cs, True, b, kc, vc, nq, unit=True, q_factor=temp),
            z.numel() * 4 + R * half * 8, like=f"qk_head_norm_append {tag}")
        add(f"qk_head_norm_append {tag}", lambda: M.qk_head_norm_append(z, wh, wh, 1e-6, cs, False, b, kc, vc, nq), z.numel() * 4 + R * half * 8)
        zl, kl, kf = torch.randn(R, (lq + lk) * Dl, **bf), torch.randn(rows_, lk, Dl, **bf), torch.rand(rows_, lk, **f32)
        add(f"unit norm, keys as they are {tag}", lambda: M.qk_head_norm_append(zl, None, None, 1e-6, None, False, b, kl, None, lq, unit=True, key_factor=kf),
            zl.numel() * 4 + R * lk * 4, like=f"qk_head_norm_append {tag}")
        # attention over everything before, beside the chunked one (capped, biased) whose chunk is as long, and the decoders'
        q, ql = torch.randn(R, nq, D, **bf), torch.randn(R, lq, Dl, **bf)
        pairs = nB * (ctx + 1) if one else B * L * (L + 1) // 2
        keys = pairs if one else R

        def cost(hq, hk, d, dv, per_key):
            return R * hq * (d + dv) * 2 + keys * per_key, 2.0 * hq * (d + dv) * pairs
        add(f"attention with a sink {tag}", lambda: M.chunk_attention(q, kc, vc, b, D ** -0.5, sink=0.0), *cost(nq, nk, D, Dv, nk * (D + Dv) * 2),
            like=f"chunk_attention {tag}")
        add(f"attention, keys as values {tag}", lambda: M.chunk_attention(ql, kl, None, b, Dl ** -0.5, key_factor=kf), *cost(lq, lk, Dl, Dl, lk * (Dl * 2 + 4)),
            like=f"chunk_attention {tag}")
        r1, r2 = torch.rand(nq, **f32), torch.rand(nq, **f32)
        add(f"chunk_attention {tag}", lambda: M.chunk_attention(q, kc, vc, b, D ** -0.5, 30.0, r1, r2, 4096), *cost(nq, nk, D, Dv, nk * (D + Dv) * 2))
        if D == Dv and D in (64, 128):
            if one:
                lens = torch.full((nB,), ctx + 1, device=dev, dtype=torch.int32)
                po, ml, o = torch.empty(nB * nq * 4 * D, **f32), torch.empty(nB * nq * 8, **f32), torch.empty_like(q)

                def paged():
                    oplib.check(oplib.get_lib().ab2_paged_decode_strided(
                        q.data_ptr(), kc.data_ptr(), vc.data_ptr(), b.pages.data_ptr(), lens.data_ptr(), po.data_ptr(), ml.data_ptr(), o.data_ptr(), nB, nq, nk, D,
                        64, b.pages.shape[1], 4, D ** -0.5, q.stride(0), oplib.stream_ptr()), "paged_decode")
                add("paged_decode decode", paged, *cost(nq, nk, D, Dv, nk * (D + Dv) * 2))
            else:
                k, v = torch.randn(R, nk, D, **bf), torch.randn(R, nk, D, **bf)
                cu = torch.arange(0, R + 1, L, device=dev, dtype=torch.int32)
                ti = OF.attn_tile_table(cu, R)
                add("attn_fwd prefill", lambda: OF.attention_fwd(q, k, v, cu, True, D ** -0.5, ti), *cost(nq, nk, D, Dv, nk * (D + Dv) * 2))
        # recurrence, beside the RG-LRU of the same width (whose gates are products of their own)
        zug, bias, St = torch.randn(R, 3 * W, **bf), torch.zeros(2 * W, **f32), torch.zeros(ne, W, **f32)
        add(f"min_gru {tag}", lambda: M.min_gru(zug, bias, b, St), R * W * 8 + 2 * St.numel() * 4, like=f"rglru {tag}")
        n = W // blocks
        gw, gb, lam, yb = torch.randn(2, blocks, n, n, **bf) * 0.05, torch.zeros(2, blocks, n, **f32), torch.full((W,), -3.0, **f32), torch.zeros(W, **f32)
        u, yx = torch.randn(R, W, **bf), torch.randn(R, 2 * W, **bf)
        add(f"rglru {tag}", lambda: M.rglru(u, yx[:, :W], yb, gw, gb, lam, b, St), R * W * 6 + gw.numel() * 2 + 2 * St.numel() * 4, 4.0 * R * W * n)
        # feed-forward
        gu = torch.randn(R, 2 * ff, **bf)
        add(f"glu_clamped {tag}", lambda: M.glu_clamped(gu, 7.0, 1.702), R * ff * 6, like=f"swiglu {tag}")
        with torch.no_grad():
            add(f"swiglu {tag}", lambda: OF.swiglu(gu), R * ff * 6)
    return rows


# ----------------------------------------------------------------------------- whole steps
def _engine(cfg, seqs, total, prefill_tokens):
    from ..api.cli_args import InferenceEngineConfig, NativeInferConfig
    from ..engine.infer_engine import NativeInferenceEngine
    from ..models.decoder import build_model

    ic = NativeInferConfig(page_size=64, num_pages=seqs * (total // 64 + 2), max_running_requests=seqs, context_length=total + 64,
                           max_prefill_tokens=prefill_tokens)
    model = build_model(cfg, dtype=torch.bfloat16, device="cuda", seed=1)
    return NativeInferenceEngine(InferenceEngineConfig(), ic, model=model).initialize(device="cuda", start_executor=False, start_loop=False)


def mixer_steps(cfg, prefill, decode) -> dict:
    from ..engine.ragged_step import Entry

    (B, L), (nB, ctx) = prefill, decode
    eng = _engine(cfg, max(B, nB), max(L, ctx + 64), B * L)
    toks = torch.randint(0, cfg.vocab_size, (L,)).tolist()

    def fill(n, length):
        cs = []
        for _ in range(n):
            c = eng.cache.open()
            assert eng.cache.grow(c, length)
            cs.append(c)
        return cs

    def prompt():
        cs = fill(B, L)
        eng.runner.step([Entry(c, toks, [L - 1]) for c in cs])
        for c in cs:
            eng.cache.close(c)
    with torch.cuda.stream(eng.stream):
        tp = timed(prompt, iters=5, warmup=2)
        cs = fill(nB, ctx)
        for c in cs:
            eng.runner.step([Entry(c, (toks * (ctx // L + 1))[:ctx], [])])

        def one():
            for c in cs:
                eng.cache.grow(c, c.length + 1)
            eng.runner.step([Entry(c, [7], [0]) for c in cs])
        td = timed(one, iters=20, warmup=4)
        n0, t0 = oplib.launch_count(), time.perf_counter()
        for _ in range(10):
            one()
        torch.cuda.synchronize()
        wall, n = (time.perf_counter() - t0) / 10, (oplib.launch_count() - n0) // 10
    out = dict(prefill_tokens_per_s=round(B * L / tp), prefill_ms=round(tp * 1e3, 3), decode_tokens_per_s=round(nB / td), decode_ms=round(td * 1e3, 3),
               decode_wall_ms=round(wall * 1e3, 3), decode_launches=n, params_m=round(sum(p.numel() for p in eng.model.parameters()) / 1e6, 1))
    eng.destroy()
    return out


def decoder_steps(cfg, prefill, decode) -> dict:
    """A dense / routed decoder of the framework: packed prefill and graph-captured paged decode of the rollout engine."""
    from ..engine.infer_engine import _Seq

    (B, L), (nB, ctx) = prefill, decode
    eng = _engine(cfg, max(B, nB), max(L, ctx + 64), max(B * L, ctx * 8))

    def seq(i, n):
        return _Seq(rid=str(i), tokens=torch.randint(0, cfg.vocab_size, (n,)).tolist(), prompt_len=n, max_new=1 << 20, min_new=0, temperature=1.0, greedy=True,
                    stop_ids=set(), ignore_eos=True, seed=1)

    def prompt():
        ss = [seq(i, L) for i in range(B)]
        for s in ss:
            s.pages = eng.cache.alloc(eng.cache.pages_needed(L + 1))
        eng._prefill(ss, [])
        for s in ss:
            eng.cache.release(s.pages)
    with torch.cuda.stream(eng.stream), torch.no_grad():
        tp = timed(prompt, iters=5, warmup=2)
        run = [seq(i, ctx) for i in range(nB)]
        for i in range(0, nB, 8):
            for s in run[i:i + 8]:
                s.pages = eng.cache.alloc(eng.cache.pages_needed(ctx + 64))
            eng._prefill(run[i:i + 8], [])
        for s in run:
            eng._assign_row(s)
        td = timed(lambda: eng._decode(run, []), iters=20, warmup=4)
    out = dict(prefill_tokens_per_s=round(B * L / tp), prefill_ms=round(tp * 1e3, 3), decode_tokens_per_s=round(nB / td), decode_ms=round(td * 1e3, 3),
               params_m=round(sum(p.numel() for p in eng.model.parameters()) / 1e6, 1))
    eng.destroy()
    return out


def hybrid_steps(cfg, prefill, decode) -> dict:
    """The framework's linear / full attention stack (carried state outside pages and graphs)."""
    from ..models.decoder import build_model
    from ..models.hybrid import decode_states, prefill_states

    (B, L), (nB, ctx) = prefill, decode
    model = build_model(cfg, dtype=torch.bfloat16, device="cuda", seed=1).eval()
    with torch.no_grad():
        ids = torch.randint(0, cfg.vocab_size, (B * L,), device="cuda")
        cu = torch.arange(0, B * L + 1, L, device="cuda", dtype=torch.int32)
        tp = timed(lambda: model.logits(prefill_states(model, ids, cu, L)[0][(cu[1:] - 1).long()]), iters=3, warmup=1)
        states = []
        for _ in range(0, nB, 8):
            n = min(8, nB)
            c2 = torch.arange(0, n * ctx + 1, ctx, device="cuda", dtype=torch.int32)
            states += prefill_states(model, torch.randint(0, cfg.vocab_size, (n * ctx,), device="cuda"), c2, ctx)[1]
        t1 = torch.randint(0, cfg.vocab_size, (nB,), device="cuda")
        td = timed(lambda: model.logits(decode_states(model, t1, states[:nB])), iters=5, warmup=2)
    return dict(prefill_tokens_per_s=round(B * L / tp), prefill_ms=round(tp * 1e3, 3), decode_tokens_per_s=round(nB / td), decode_ms=round(td * 1e3, 3),
                params_m=round(sum(p.numel() for p in model.parameters()) / 1e6, 1))


def like_sized(cfg):
    """The closest existing models with the same width, heads, feed-forward and vocabulary: (hybrid stack, dense decoder,
    routed decoder), as many layers as ``cfg`` has."""
    from ..models.config import ModelConfig

    at = next(e["mixer"] for e in cfg.mixer_layers if e["type"] == "attention")
    moe = next(e["mlp"] for e in cfg.mixer_layers if e["mlp"] and e["mlp"]["kind"] == "moe")
    n = cfg.num_layers
    base = dict(vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, num_layers=n, num_heads=at["heads"], num_kv_heads=at["kv_heads"], head_dim=at["dim"],
                intermediate_size=cfg.intermediate_size, tie_word_embeddings=False, attention_bias=False, qk_norm=True)
    hyb = ModelConfig(arch="qwen3_5", **base, layer_types=["full_attention" if i == 0 else "linear_attention" for i in range(n)], linear_key_head_dim=128,
                      linear_value_head_dim=128, linear_num_key_heads=cfg.hidden_size // 256, linear_num_value_heads=cfg.hidden_size // 128,
                      partial_rotary_factor=0.25, attn_output_gate=True, rms_norm_offset=True)
    routed = ModelConfig(arch="qwen3_moe", **base, num_experts=moe["router"]["experts"], num_experts_per_tok=moe["router"]["top"],
                         moe_intermediate_size=moe["expert"]["ff"])
    return hyb, ModelConfig(arch="qwen3", **base), routed


def latent_like_sized(cfg):
    """The closest existing models with the same width, heads, feed-forwards, experts and vocabulary as a latent stack: the
    mixer stack with grouped-query attention in chunks as long as the windows (a key head per four query heads), the dense
    and the routed decoder."""
    from ..models.config import ModelConfig

    at = cfg.mixer_layers[0]["mixer"]
    nk = max(1, at["heads"] // 4)
    layers = []
    for e in cfg.mixer_layers:
        m = dict(heads=at["heads"], kv_heads=nk, dim=at["dim"], vdim=at["vdim"], scale=at["scale"], softcap=30.0, mask=dict(e["mixer"]["mask"]))
        layers.append(dict(type="attention", mixer=m, mlp=e["mlp"]))
    stack = ModelConfig.from_hf_dict(dict(architecture="Kagolix", vocab=cfg.vocab_size, width=cfg.hidden_size, norm=dict(eps=1e-6, groups=1),
                                          logit_softcap=0.0, layers=layers))
    base = dict(vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, num_layers=cfg.num_layers, num_heads=at["heads"], num_kv_heads=nk,
                head_dim=at["dim"], intermediate_size=cfg.intermediate_size, tie_word_embeddings=False, attention_bias=False, qk_norm=True)
    routed = ModelConfig(arch="qwen3_moe", **base, num_experts=cfg.num_experts, num_experts_per_tok=cfg.num_experts_per_tok,
                         moe_intermediate_size=cfg.moe_intermediate_size)
    return stack, ModelConfig(arch="qwen3", **base), routed


def looped_like_sized(cfg):
    """The closest existing models with the same width, experts and vocabulary as a looped stack, one layer per layer run:
    the other latent stack (windows of a whole prompt), the stack with Mamba-2 and chunked attention in place of the parallel
    branches and of the latents, the routed decoder."""
    from ..models.config import ModelConfig
    from ..models.mixers import MixerStackLM

    runs = MixerStackLM.layer_runs.fget(type("S", (), dict(cfg=cfg)))
    par = next(e["mixer"] for e in cfg.mixer_layers if e["type"] == "parallel")
    at = next(e["mixer"] for e in cfg.mixer_layers if e["type"] == "latent_attention")
    moe = next(e["mlp"] for e in cfg.mixer_layers if e["mlp"])
    lf, rt = par["left"], par["right"]
    lat = dict(heads=at["heads"], dim=at["dim"], vdim=at["vdim"], q_rank=1536, kv_rank=at["kv_rank"], scale=at["scale"], mask=dict(size=4096))
    experts = dict(moe, expert=dict(moe["expert"], limit=6.0), shared=dict(moe["shared"], limit=7.0))
    vog = ModelConfig.from_hf_dict(dict(architecture="Vogilix", vocab=cfg.vocab_size, width=cfg.hidden_size, max_positions=8192, norm=dict(eps=1e-6), residual_mult=0.5,
                                        token_side=None, layers=[dict(type="latent_attention", mixer=lat, mlp=experts) for _ in runs]))
    att = dict(heads=lf["heads"], kv_heads=lf["kv_heads"], dim=lf["dim"], vdim=lf["vdim"], scale=lf["scale"], softcap=lf["softcap"], mask=dict(lf["mask"]))
    ssm = dict(heads=2 * rt["heads"], vdim=rt["vdim"], state=rt["dim"], groups=rt["heads"], norm_groups=rt["heads"], conv=4)
    stack = ModelConfig.from_hf_dict(dict(
        architecture="Kagolix", vocab=cfg.vocab_size, width=cfg.hidden_size, norm=dict(eps=1e-6, groups=1), logit_softcap=0.0,
        layers=[dict(type="attention" if n % 2 else "mamba2", mixer=att if n % 2 else ssm, mlp=dict(moe, shared=None)) for n in range(len(runs))]))
    base = dict(vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, num_layers=len(runs), num_heads=lf["heads"], num_kv_heads=lf["kv_heads"],
                head_dim=lf["dim"], intermediate_size=0, tie_word_embeddings=False, attention_bias=False, qk_norm=True)
    routed = ModelConfig(arch="qwen3_moe", **base, num_experts=cfg.num_experts, num_experts_per_tok=cfg.num_experts_per_tok,
                         moe_intermediate_size=cfg.moe_intermediate_size)
    return vog, stack, routed


def shifted_like_sized(cfg):
    """The closest existing models with the same width, heads and vocabulary as a shifted stack, one layer per layer run: the stack
    that alternates chunked attention (chunks longer than the prompts) and RG-LRU, its dense feed-forwards (two matrices) one and a
    half times as wide for the same weights; the dense decoder."""
    from ..models.config import ModelConfig
    from ..models.mixers import MixerStackLM

    runs = MixerStackLM.layer_runs.fget(type("S", (), dict(cfg=cfg)))
    at = next(e["mixer"] for e in cfg.mixer_layers if e["type"] == "attention")
    W, ff = next(e["mixer"] for e in cfg.mixer_layers if e["type"] == "parallel")["right"]["width"], cfg.intermediate_size
    att = dict(heads=at["heads"], kv_heads=at["kv_heads"], dim=at["dim"], vdim=at["vdim"], scale=at["scale"], softcap=30.0, mask=dict(size=4096))
    lru = dict(width=W, blocks=W // 256, conv=4)
    stack = ModelConfig.from_hf_dict(dict(
        architecture="Kagolix", vocab=cfg.vocab_size, width=cfg.hidden_size, norm=dict(eps=1e-6, groups=1), logit_softcap=0.0,
        layers=[dict(type="rglru" if n % 2 else "attention", mixer=lru if n % 2 else att, mlp=dict(kind="dense", ff=3 * ff // 2)) for n in range(len(runs))]))
    dense = ModelConfig(arch="qwen3", vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, num_layers=len(runs), num_heads=at["heads"],
                        num_kv_heads=at["kv_heads"], head_dim=at["dim"], intermediate_size=ff, tie_word_embeddings=False, attention_bias=False, qk_norm=True)
    return stack, dense


def run(steps=True, kernels=True, design="kagolix", sizes=None) -> dict:
    from ..models.config import preset

    torch.manual_seed(0)
    bw, fl, src = peaks()
    out = dict(workload="mixer-serve", dtype="bf16", data="synthetic tokens, random weights", roofline=f"{src}: {bw / 1e9:.0f} GB/s, {fl / 1e12:.0f} TFLOP/s",
               sizes={})
    for name in sizes or (f"{design}-8b-layers", f"{design}-2b-layers"):
        cfg = preset(name)
        prefill, decode = (4, 2048), (64, 960)
        r = dict(prefill=f"{prefill[0]} x {prefill[1]} tokens", decode=f"{decode[0]} sequences at {decode[1]} tokens")
        if steps and design == "vogilix":
            stack, dense, routed = latent_like_sized(cfg)
            for key, fn, c in (("vogilix", mixer_steps, cfg), ("mixer_stack_attention", mixer_steps, stack), ("decoder_dense", decoder_steps, dense),
                               ("decoder_routed", decoder_steps, routed)):
                r[key] = fn(c, prefill, decode)
                torch.cuda.empty_cache()
        elif steps and design == "bumotar":
            latent, stack, routed = looped_like_sized(cfg)
            for key, fn, c in (("bumotar", mixer_steps, cfg), ("vogilix", mixer_steps, latent), ("mixer_stack", mixer_steps, stack), ("decoder_routed", decoder_steps, routed)):
                r[key] = fn(c, prefill, decode)
                torch.cuda.empty_cache()
        elif steps and design == "goganex":
            stack, dense = shifted_like_sized(cfg)
            for key, fn, c in (("goganex", mixer_steps, cfg), ("mixer_stack", mixer_steps, stack), ("decoder_dense", decoder_steps, dense)):
                r[key] = fn(c, prefill, decode)
                torch.cuda.empty_cache()
        elif steps:
            hyb, dense, routed = like_sized(cfg)
            r["mixer_stack"] = mixer_steps(cfg, prefill, decode)
            torch.cuda.empty_cache()
            for key, fn, c in (("decoder_dense", decoder_steps, dense), ("decoder_routed", decoder_steps, routed), ("hybrid", hybrid_steps, hyb)):
                r[key] = fn(c, prefill, decode)
                torch.cuda.empty_cache()
        if kernels:
            r["kernels"] = {"vogilix": latent_kernel_table, "bumotar": looped_kernel_table, "goganex": shifted_kernel_table,
                            "kagolix": kernel_table}[design](cfg, prefill, decode)
        out["sizes"][name] = r
    return out
