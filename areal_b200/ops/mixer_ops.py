"""Ops of mixer stacks: grouped sandwich norms on a 32-bit residual stream, chunked attention with capped scores and
a logarithmic distance bias over a paged cache, causal convolutions, RG-LRU and Mamba-2 recurrences on slot states,
xIELU, expert combine and capped logits.

Every op works on a :class:`RaggedBatch`: the rows of several requests, each bringing any number of its next tokens,
continuing from the cache pages and state slots that earlier steps left. The first ``n_dec`` entries bring one row
each, so that single tokens take the decode kernels and longer portions the prefill kernels.

As in :mod:`.functional`, CUDA tensors run the sm_100a kernels (activations bf16 or fp32), CPU tensors a PyTorch
statement of the same op. Vectors (norm weights, biases, decay parameters, convolution taps), states and the residual
stream are fp32 everywhere.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from . import functional as OF
from . import lib as _lib
from .functional import EPI_F32, Routing, gemm, grouped_gemm_rt

SCAN_BLOCK = 64          # rows per block of the blocked recurrences
ATTN_TILE = 256          # query rows per tile of the prefill attention kernel

_V, _I, _F = _lib.c_void_p, _lib.c_int, _lib.c_float


def _p(t):
    return None if t is None else t.data_ptr()


def _dt(t) -> int:
    if t.dtype == torch.bfloat16:
        return 0
    if t.dtype == torch.float32:
        return 1
    raise TypeError(f"mixer ops take bf16 or fp32 activations, not {t.dtype}")


def _call(name: str, *args):
    _lib.check(getattr(_lib.get_lib(), name)(*args, _lib.stream_ptr()), name)


@dataclass
class RaggedBatch:
    """Rows of one step (all tensors int32 on the model's device)."""

    tokens: torch.Tensor         # [R] token ids
    pos: torch.Tensor            # [R] position in its sequence
    slots: torch.Tensor          # [R] cache row of the token (page * page_size + offset); -1: padding row
    row_entry: torch.Tensor      # [R] entry of the row
    cu: torch.Tensor             # [E + 1] first row of every entry
    start: torch.Tensor          # [E] tokens absorbed before this step (0: a new sequence, its state counts as zero)
    state: torch.Tensor          # [E] state slot; -1: padding entry
    pages: torch.Tensor          # [E, P] pages held, from page number ``page_base`` of the sequence on
    page_base: torch.Tensor      # [E]
    blocks: Optional[torch.Tensor]   # [NB, 4] (entry, first row, rows, 1 if first of its entry), rows of entries >= n_dec
    tiles: Optional[torch.Tensor]    # [NT, 2] (entry, first row) query tiles of entries >= n_dec
    n_dec: int                   # leading entries with one row
    page_size: int

    @property
    def n_rows(self) -> int:
        return self.tokens.shape[0]

    @property
    def n_entries(self) -> int:
        return self.start.shape[0]


def _segments(b: RaggedBatch):
    """(entry, first row, end row, start position, state slot) per entry that is not padding (CPU ops)."""
    cu, st, sl = b.cu.tolist(), b.start.tolist(), b.state.tolist()
    return [(e, cu[e], cu[e + 1], st[e], sl[e]) for e in range(b.n_entries) if sl[e] >= 0]


# ----------------------------------------------------------------------------- matrix products
def linear(x: torch.Tensor, w: torch.Tensor, fp32_out: bool = False) -> torch.Tensor:
    """``x @ w^T`` without autograd, output in x's dtype (or fp32). bf16 products with aligned rows take the tcgen05
    GEMM, 32-bit ones and odd row lengths the library product."""
    if x.is_cuda and x.dtype == torch.bfloat16 and x.shape[1] % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0:
        N = w.shape[0]
        if OF.DECODE_SPLITK and not fp32_out and x.shape[0] <= OF.DECODE_GEMM_MAX_ROWS and N % 8 == 0:
            return OF.gemm_decode(x, w)
        ld = -(-N // 8) * 8
        out = torch.empty(x.shape[0], ld, device=x.device, dtype=torch.float32 if fp32_out else torch.bfloat16)
        gemm(x, w, out=out[:, :N], epi=EPI_F32 if fp32_out else 0)
        return out[:, :N]
    if fp32_out and x.dtype != torch.float32:
        return F.linear(x.float(), w.float())
    return F.linear(x, w)


def router_logits(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """32-bit router logits from (possibly bf16) activations and weights."""
    return F.linear(x.float(), w.float())


# ----------------------------------------------------------------------------- norms
def group_norm_ref(x, w, groups, eps):
    xf = x.float()
    p = xf.reshape(*xf.shape[:-1], groups, -1)
    p = p * torch.rsqrt(p.pow(2).mean(-1, keepdim=True) + eps)
    return p.reshape(xf.shape) * w


def embed_norm(ids, table, w, groups: int, eps: float):
    """``(residual fp32, groupnorm(residual) * w)`` for the embedding rows of ``ids``."""
    H = table.shape[1]
    if not table.is_cuda:
        resid = table[ids.long()].float()
        return resid, group_norm_ref(resid, w, groups, eps).to(table.dtype)
    resid = torch.empty(ids.shape[0], H, device=table.device, dtype=torch.float32)
    x = torch.empty(ids.shape[0], H, device=table.device, dtype=table.dtype)
    _call("ab2_sandwich_norm", _p(ids), _p(table), table.shape[0], None, 0, None, _p(resid), _p(w), _p(x), ids.shape[0], H, groups, eps, _dt(table))
    return resid, x


def sandwich_norm(h, w_post, resid, w_next, groups: int, eps: float):
    """``resid += groupnorm(h) * w_post`` (in place, fp32), returns ``groupnorm(resid) * w_next`` in h's dtype."""
    if not h.is_cuda:
        resid += group_norm_ref(h, w_post, groups, eps)
        return group_norm_ref(resid, w_next, groups, eps).to(h.dtype)
    T, H = h.shape
    assert h.stride(1) == 1
    x = torch.empty(T, H, device=h.device, dtype=h.dtype)
    _call("ab2_sandwich_norm", None, None, 0, _p(h), h.stride(0), _p(w_post), _p(resid), _p(w_next), _p(x), T, H, groups, eps, _dt(h))
    return x


# ----------------------------------------------------------------------------- attention
def qk_norm_append(qkv, wq, wk, eps: float, b: RaggedBatch, kc, vc, Hq: int):
    """Whole-projection RMS norms of q and k, then k and v into the cache rows of ``b.slots``; returns q [R, Hq, D].
    ``qkv`` rows are q | k | v; ``kc`` [S, Hkv, D], ``vc`` [S, Hkv, Dv]."""
    Hkv, D, Dv = kc.shape[1], kc.shape[2], vc.shape[2]
    nq, nk, nv = Hq * D, Hkv * D, Hkv * Dv
    R = qkv.shape[0]
    if not qkv.is_cuda:
        q = group_norm_ref(qkv[:, :nq], wq, 1, eps).to(qkv.dtype)
        k = group_norm_ref(qkv[:, nq:nq + nk], wk, 1, eps).to(qkv.dtype)
        ok = b.slots >= 0
        kc[b.slots[ok].long()] = k[ok].view(-1, Hkv, D)
        vc[b.slots[ok].long()] = qkv[ok, nq + nk:].reshape(-1, Hkv, Dv)
        return q.view(R, Hq, D)
    q = torch.empty(R, Hq, D, device=qkv.device, dtype=qkv.dtype)
    _call("ab2_qk_norm_append", _p(qkv), qkv.stride(0), _p(wq), _p(wk), _p(b.slots), _p(q), _p(kc), _p(vc), R, nq, nk, nv, eps, _dt(qkv))
    return q


def chunk_attention_ref(q, kc, vc, b: RaggedBatch, scale, softcap, r1, r2, chunk):
    R, Hq, D = q.shape
    Hkv, Dv = kc.shape[1], vc.shape[2]
    out = torch.zeros(R, Hq, Dv, dtype=q.dtype)
    rep, ps = Hq // Hkv, b.page_size
    for e, r0, r1_, st, _ in _segments(b):
        end = st + r1_ - r0
        lo = (st // chunk) * chunk if chunk else 0
        j = torch.arange(lo, end)
        rows = b.pages[e][(j // ps - b.page_base[e]).long()].long() * ps + j % ps
        k = kc[rows].float().repeat_interleave(rep, 1)
        v = vc[rows].float().repeat_interleave(rep, 1)
        i = torch.arange(st, end)
        s = torch.einsum("ihd,jhd->hij", q[r0:r1_].float(), k) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        dist = (i[:, None] - j[None, :])
        if r1 is not None:
            s = s - r1[:, None, None] * torch.log1p(r2[:, None, None] * dist.clamp(min=0))
        see = dist >= 0
        if chunk:
            see &= (i // chunk)[:, None] == (j // chunk)[None, :]
        s = s.masked_fill(~see, float("-inf"))
        out[r0:r1_] = torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v).to(q.dtype)
    return out


def chunk_attention(q, kc, vc, b: RaggedBatch, scale: float, softcap: float = 0.0, r1=None, r2=None, chunk: int = 0):
    """Attention of the step's queries over the paged cache (their own keys already appended): ``softcap *
    tanh(q.k * scale / softcap)`` minus ``r1[h] * ln(1 + r2[h] * distance)``, softmax over the earlier positions of
    the query's own chunk of ``chunk`` positions (0: no limit). Returns [R, Hq, Dv]."""
    if not q.is_cuda:
        return chunk_attention_ref(q, kc, vc, b, scale, softcap, r1, r2, chunk)
    R, Hq, D = q.shape
    Hkv, Dv = kc.shape[1], vc.shape[2]
    out = torch.empty(R, Hq, Dv, device=q.device, dtype=q.dtype)
    common = (_p(kc), _p(vc), _p(b.pages), _p(b.page_base), b.pages.shape[1], b.page_size, Hq, Hkv, D, Dv, scale, softcap, _p(r1), _p(r2), chunk)
    fast = q.dtype == torch.bfloat16 and D % 8 == 0 and Dv % 8 == 0 and D <= 128 and Dv <= 128
    nd = b.n_dec
    if nd:
        if fast and Hq // Hkv <= 16:
            _call("ab2_chunk_decode", _p(q), _p(b.pos), _p(b.slots), _p(out), nd, *common)
        else:
            _call("ab2_chunk_attn_plain", _p(q), _p(b.pos), _p(b.slots), _p(b.row_entry), _p(out), nd, *common, _dt(q))
    if R > nd:
        if fast and b.page_size in (16, 32, 64, 128) and b.tiles is not None:
            _call("ab2_chunk_prefill", _p(q), _p(b.cu), _p(b.start), _p(b.tiles), b.tiles.shape[0], _p(out), R, kc.shape[0], *common)
        else:
            _call("ab2_chunk_attn_plain", _p(q[nd:]), _p(b.pos[nd:]), _p(b.slots[nd:]), _p(b.row_entry[nd:]), _p(out[nd:]), R - nd, *common, _dt(q))
    return out


# ----------------------------------------------------------------------------- causal convolution with carried tails
def causal_conv(x, bias_in, w, bias, silu: bool, b: RaggedBatch, tail):
    """Per-channel causal convolution of ``x (+ bias_in)`` over every entry's rows, continuing from (and updating) the
    last ``taps - 1`` inputs of its slot. x [R, C] (rows may be strided), w [C, taps] (last tap on the current token),
    tail [slots, C, taps - 1]. Returns bias + convolution, through silu when asked, in x's dtype."""
    C, K = w.shape
    if not x.is_cuda:
        out = torch.zeros(x.shape, dtype=x.dtype)
        for e, r0, r1, st, sl in _segments(b):
            seg = x[r0:r1].float() + (bias_in if bias_in is not None else 0.0)
            old = tail[sl].t() if st > 0 else torch.zeros(K - 1, C)
            full = torch.cat([old, seg], 0)
            y = bias + sum(full[j:j + r1 - r0] * w[:, j] for j in range(K))
            out[r0:r1] = (F.silu(y) if silu else y).to(x.dtype)
            if K > 1:
                tail[sl] = full[-(K - 1):].t()
        return out
    R = x.shape[0]
    out = torch.empty(R, C, device=x.device, dtype=x.dtype)
    nb = 0 if b.blocks is None else b.blocks.shape[0]
    _call("ab2_causal_conv", _p(x), x.stride(0), _p(bias_in), _p(w), _p(bias), int(silu), _p(b.cu), _p(b.start), _p(b.state), _p(b.blocks), nb,
          b.n_dec, b.n_entries, _p(tail), _p(out), C, K, _dt(x))
    return out


# ----------------------------------------------------------------------------- RG-LRU
def rglru(u, y, y_bias, gate_w, gate_b, lam, b: RaggedBatch, S):
    """``S_t = a S_(t-1) + sqrt(1 - a^2) i u`` with ``a = exp(-8 r softplus(lam))`` and the block-diagonal gates r, i of
    u; returns ``S * gelu_tanh(y + y_bias)`` in u's dtype and leaves the last state of every entry in its slot.
    u [R, W]; y [R, W] (rows may be strided); gate_w [2, blocks, W / blocks, W / blocks] (r, i); S [slots, W]."""
    R, W = u.shape
    n, bs = gate_w.shape[1], gate_w.shape[2]
    if not u.is_cuda:
        ub = u.float().view(R, n, bs)
        r, i = (torch.sigmoid(torch.einsum("rnk,nok->rno", ub, gate_w[g].float()) + gate_b[g]).reshape(R, W) for g in (0, 1))
        log_a = -8.0 * r * F.softplus(lam)
        a, x = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * i * u.float()
        gate = F.gelu(y.float() + y_bias, approximate="tanh")
        out = torch.zeros(R, W, dtype=u.dtype)
        for e, r0, r1, st, sl in _segments(b):
            h = S[sl].clone() if st > 0 else torch.zeros(W)
            for t in range(r0, r1):
                h = a[t] * h + x[t]
                out[t] = (h * gate[t]).to(u.dtype)
            S[sl] = h
        return out
    out = torch.empty(R, W, device=u.device, dtype=u.dtype)
    nd, nb = b.n_dec, 0 if b.blocks is None else b.blocks.shape[0]
    if nd:
        _call("ab2_rglru_decode", _p(u), _p(y), y.stride(0), _p(y_bias), _p(gate_w), _p(gate_b), _p(lam), _p(b.start), _p(b.state), _p(S), _p(out),
              nd, n, bs, _dt(u))
    if nb:
        f32 = dict(device=u.device, dtype=torch.float32)
        a, x = torch.empty(R - nd, W, **f32), torch.empty(R - nd, W, **f32)
        carry = torch.empty(2, nb, W, **f32)
        _call("ab2_rglru_prefill", _p(u[nd:]), _p(y[nd:]), y.stride(0), _p(y_bias), _p(gate_w), _p(gate_b), _p(lam), _p(b.blocks), nb, nd, R - nd,
              _p(b.start), _p(b.state), _p(S), _p(a), _p(x), _p(carry), _p(out[nd:]), n, bs, _dt(u))
    return out


# ----------------------------------------------------------------------------- Mamba-2
def mamba2_scan(xbc, dt_raw, dt_bias, A_log, D, heads: int, vdim: int, state: int, groups: int, b: RaggedBatch, S):
    """``S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T``, ``y_t = S_t^T C_t + D x_t`` per head, from the convolved
    rows x | B | C and ``dt = softplus(dt_raw + dt_bias)``. Returns y [R, heads * vdim] (fp32); S [slots, heads, vdim,
    state] is left at every entry's last token."""
    R = xbc.shape[0]
    inner = heads * vdim
    if not xbc.is_cuda:
        x = xbc[:, :inner].float().view(R, heads, vdim)
        B, C = (t.float().view(R, groups, state).repeat_interleave(heads // groups, 1)
                for t in (xbc[:, inner:inner + groups * state], xbc[:, inner + groups * state:]))
        dt = F.softplus(dt_raw.float() + dt_bias)
        decay = torch.exp(-torch.exp(A_log) * dt)
        y = torch.zeros(R, heads, vdim)
        for e, r0, r1, st, sl in _segments(b):
            h = S[sl].clone() if st > 0 else torch.zeros(heads, vdim, state)
            for t in range(r0, r1):
                h = decay[t][:, None, None] * h + (dt[t][:, None] * x[t])[:, :, None] * B[t][:, None, :]
                y[t] = (h * C[t][:, None, :]).sum(-1) + D[:, None] * x[t]
            S[sl] = h
        return y.reshape(R, inner)
    y = torch.empty(R, inner, device=xbc.device, dtype=torch.float32)
    args = (_p(xbc), xbc.stride(0), _p(dt_raw), dt_raw.stride(0), _p(dt_bias), _p(A_log), _p(D), _p(b.cu), _p(b.start), _p(b.state))
    E, nd = b.n_entries, b.n_dec
    if E > nd and xbc.dtype == torch.bfloat16 and vdim % 8 == 0 and state % 8 == 0 and state <= 128 and xbc.stride(0) % 8 == 0:
        # portions in blocks on the tensor cores, single tokens with one pass over their state
        _call("ab2_mamba2_ssd", *args, nd, E, _p(S), _p(y), heads, vdim, state, groups)
        E = nd
    if E:
        _call("ab2_mamba2_scan", *args, E, _p(S), _p(y), heads, vdim, state, groups, _dt(xbc))
    return y


def gated_group_norm(y, z, w, groups: int, eps: float):
    """``groupnorm(y * silu(z)) * w`` in z's dtype; y fp32 [R, C], z [R, C] (rows may be strided)."""
    if not z.is_cuda:
        return group_norm_ref(y * F.silu(z.float()), w, groups, eps).to(z.dtype)
    R, C = y.shape
    out = torch.empty(R, C, device=z.device, dtype=z.dtype)
    _call("ab2_gated_group_norm", _p(y), _p(z), z.stride(0), _p(w), _p(out), R, C, groups, eps, _dt(z))
    return out


# ----------------------------------------------------------------------------- feed-forward pieces
def xielu(x, pq):
    """``softplus(p) z^2 + z / 2`` above zero, ``(1/2 + softplus(q)) (exp(z) - 1 - z) + z / 2`` below; pq fp32 [2]."""
    if not x.is_cuda:
        z, s = x.float(), F.softplus(pq)
        n = z.clamp(max=0)
        return torch.where(z > 0, s[0] * z * z, (0.5 + s[1]) * (torch.expm1(n) - n)).add(z / 2).to(x.dtype)
    out = torch.empty(x.shape, device=x.device, dtype=x.dtype)
    _call("ab2_xielu", _p(x), x.stride(0), _p(pq), _p(out), x.shape[0], x.shape[1], _dt(x))
    return out


def glu_silu(gu):
    """``silu(g) * u`` for rows g | u."""
    I = gu.shape[1] // 2
    if not gu.is_cuda:
        return (F.silu(gu[:, :I].float()) * gu[:, I:].float()).to(gu.dtype)
    out = torch.empty(gu.shape[0], I, device=gu.device, dtype=gu.dtype)
    _call("ab2_glu_silu", _p(gu), gu.stride(0), _p(out), gu.shape[0], I, _dt(gu))
    return out


def expert_linear(x, w, routing: Routing):
    """Rows of ``x`` sorted by expert times ``w[e]^T``: the grouped tcgen05 GEMM for bf16 with aligned sizes, a plain
    grouped kernel in 32-bit and for odd sizes."""
    N, K = w.shape[1], w.shape[2]
    if not x.is_cuda or (x.dtype == torch.bfloat16 and N % 8 == 0 and K % 8 == 0):
        return grouped_gemm_rt(x, w, routing)
    out = torch.empty(x.shape[0], N, device=x.device, dtype=x.dtype)
    _call("ab2_grouped_plain", _p(x), _p(w), _p(out), _p(routing.row_tiles), _p(routing.num_row_tiles), routing.row_tiles.shape[0], N, K, _dt(x))
    return out


def expert_combine(y, routing: Routing, topw):
    """``sum_s topw[t, s] * y[row of (t, s)]`` with fp32 weights and sum; y holds the expert-sorted rows."""
    T, k = topw.shape
    if not y.is_cuda:
        return (y.index_select(0, routing.inv).view(T, k, -1).float() * topw[..., None]).sum(1).to(y.dtype)
    out = torch.empty(T, y.shape[1], device=y.device, dtype=y.dtype)
    _call("ab2_expert_combine", _p(y), _p(routing.inv), _p(topw), _p(out), T, k, y.shape[1], _dt(y))
    return out


# ----------------------------------------------------------------------------- output
def softcap_(logits, cap: float):
    """``cap * tanh(logits / cap)`` in place on fp32 logits."""
    if cap <= 0:
        return logits
    if not logits.is_cuda:
        return logits.copy_(cap * torch.tanh(logits / cap))
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    _call("ab2_softcap", _p(logits), logits.stride(0), logits.shape[0], logits.shape[1], cap)
    return logits


for _n, _a in {
    "ab2_sandwich_norm": [_V, _V, _I, _V, _lib.c_ll, _V, _V, _V, _V, _I, _I, _I, _F, _I],
    "ab2_qk_norm_append": [_V, _lib.c_ll, _V, _V, _V, _V, _V, _V, _I, _I, _I, _I, _F, _I],
    "ab2_chunk_attn_plain": [_V] * 5 + [_I] + [_V] * 4 + [_I] * 6 + [_F, _F, _V, _V, _I, _I],
    "ab2_chunk_decode": [_V] * 4 + [_I] + [_V] * 4 + [_I] * 6 + [_F, _F, _V, _V, _I],
    "ab2_chunk_prefill": [_V] * 4 + [_I, _V, _I, _I] + [_V] * 4 + [_I] * 6 + [_F, _F, _V, _V, _I],
    "ab2_causal_conv": [_V, _lib.c_ll, _V, _V, _V, _I] + [_V] * 4 + [_I] * 3 + [_V, _V, _I, _I, _I],
    "ab2_rglru_decode": [_V, _V, _lib.c_ll] + [_V] * 8 + [_I] * 4,
    "ab2_rglru_prefill": [_V, _V, _lib.c_ll] + [_V] * 5 + [_I] * 3 + [_V] * 7 + [_I] * 3,
    "ab2_mamba2_scan": [_V, _lib.c_ll, _V, _lib.c_ll] + [_V] * 6 + [_I] + [_V] * 2 + [_I] * 5,
    "ab2_mamba2_ssd": [_V, _lib.c_ll, _V, _lib.c_ll] + [_V] * 6 + [_I, _I] + [_V] * 2 + [_I] * 4,
    "ab2_gated_group_norm": [_V, _V, _lib.c_ll, _V, _V, _I, _I, _I, _F, _I],
    "ab2_xielu": [_V, _lib.c_ll, _V, _V, _I, _I, _I],
    "ab2_glu_silu": [_V, _lib.c_ll, _V, _I, _I, _I],
    "ab2_grouped_plain": [_V] * 5 + [_I] * 4,
    "ab2_expert_combine": [_V] * 4 + [_I] * 4,
    "ab2_softcap": [_V, _lib.c_ll, _I, _I, _F],
}.items():
    _lib.declare(_n, _a + [_V])
