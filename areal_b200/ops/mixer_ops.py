"""Ops of mixer stacks: norms around (grouped), behind or before the sublayers on a 32-bit residual stream, rotated
positions, attention over a paged cache (chunks or sliding windows, capped scores, a logarithmic distance bias, sinks, gated
outputs, keys that are the values too), attention on cached latents, causal convolutions, token shifts, RG-LRU, minGRU, Mamba-2 and
retention recurrences on slot states, activations, expert combine, per-layer token inputs and capped logits.

Every op works on a :class:`RaggedBatch`: the rows of several requests, each bringing any number of its next tokens,
continuing from the cache pages and state slots that earlier steps left. The first ``n_dec`` entries bring one row
each, so that single tokens take the decode kernels and longer portions the prefill kernels.

As in :mod:`.functional`, CUDA tensors run the sm_100a kernels (activations bf16 or fp32), CPU tensors a PyTorch
statement of the same op. Vectors (norm weights, biases, decay parameters, convolution taps), states and the residual
stream are fp32 everywhere.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass, field
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
class PageList:
    """Cache pages that a step's portions see, in one list, and every entry's place in it."""

    pages: torch.Tensor          # [NP] pages of the cache
    table: torch.Tensor          # [E, P'] numbers in ``pages`` of the entry's pages, from page number ``base`` of its sequence on
    base: torch.Tensor           # [E]


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
    seen: dict = field(default_factory=dict)     # sliding window -> PageList of the entries >= n_dec (latent attention)
    rot: Optional[torch.Tensor] = None           # [R, P, 2] (cos, sin) of the step's rows, made by the model (rotary_table)

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
        if OF.DECODE_SPLITK and x.shape[0] <= OF.DECODE_GEMM_MAX_ROWS and N % 8 == 0:
            return OF.gemm_decode(x, w, fp32_out=fp32_out)
        ld = -(-N // 8) * 8
        out = torch.empty(x.shape[0], ld, device=x.device, dtype=torch.float32 if fp32_out else torch.bfloat16)
        gemm(x, w, out=out[:, :N], epi=EPI_F32 if fp32_out else 0)
        return out[:, :N]
    if fp32_out and x.dtype != torch.float32:
        return F.linear(x.float(), w.float())
    return F.linear(x, w)


def head_linear(x: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None, w_kn: bool = False) -> torch.Tensor:
    """Every head's own product: ``out[r, h] = w[h] x[r, h]``; x [R, H, K] (rows and heads may be strided), w [H, N, K] (``w_kn``:
    [H, K, N]). One tcgen05 launch for bf16 with aligned sizes, the library's batched product in 32-bit and for odd sizes."""
    R, H, K = x.shape
    N = w.shape[2] if w_kn else w.shape[1]
    if out is None:
        out = torch.empty(R, H, N, device=x.device, dtype=x.dtype)
    lda, hsa = x.stride(0), max(x.stride(1), K)          # (a single head has no stride to speak of)
    if x.is_cuda and x.dtype == torch.bfloat16 and K % 8 == 0 and N % 8 == 0 and lda % 8 == 0 and hsa % 8 == 0 and x.data_ptr() % 16 == 0:
        assert x.stride(2) == 1 and w.is_contiguous() and out.is_contiguous()
        bn = 256 if N % 256 == 0 and R > 128 else 128
        _call("ab2_gemm_heads", _p(x), _p(w), _p(out), R, H, N, K, max(lda, hsa * (H - 1) + K), hsa, int(w_kn), bn)
        return out
    out.copy_(torch.bmm(x.transpose(0, 1), w if w_kn else w.transpose(1, 2)).transpose(0, 1))
    return out


def router_logits(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """32-bit router logits from (possibly bf16) activations and weights: exact products, 32-bit sums."""
    return linear(x, w, fp32_out=True)


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


@dataclass
class ExpertSum:
    """A feed-forward output that is still in pieces: the expert-sorted rows ``y``, to be summed per token (weighted when
    ``weights`` are given), and what is added to them (times ``sigmoid(shared_logit)`` when that is given). The residual sum or
    the norm behind the sublayer reads the pieces."""

    y: torch.Tensor                      # [T * k, H]
    routing: Routing
    shared: Optional[torch.Tensor]       # [T, H]
    weights: Optional[torch.Tensor] = None        # [T, k]
    shared_logit: Optional[torch.Tensor] = None   # [T] fp32, may be strided

    def dense(self) -> torch.Tensor:
        k = self.routing.k
        h = self.y.index_select(0, self.routing.inv).view(-1, k, self.y.shape[1]).float()
        h = (h if self.weights is None else h * self.weights[..., None]).sum(1)
        if self.shared is None:
            return h
        return h + (self.shared.float() if self.shared_logit is None else self.shared.float() * torch.sigmoid(self.shared_logit)[:, None])


@dataclass
class BranchSum:
    """A mixer output that is still in two pieces: ``factor`` times the sum of both, each first RMS-normed with its weight. The
    residual sum behind the mixer reads the pieces."""

    left: torch.Tensor                   # [T, H], rows may be strided
    right: torch.Tensor
    w_left: torch.Tensor                 # [H] fp32
    w_right: torch.Tensor
    factor: float
    eps: float

    def dense(self) -> torch.Tensor:
        return self.factor * (group_norm_ref(self.left, self.w_left, 1, self.eps) + group_norm_ref(self.right, self.w_right, 1, self.eps))


@dataclass
class EmbeddingRows:
    """What begins a residual stream: ``scale`` times the rows of ``ids``."""

    ids: torch.Tensor
    table: torch.Tensor
    scale: float = 1.0

    def dense(self) -> torch.Tensor:
        return self.table[self.ids.long()].float() * self.scale


def embed_rows(ids, table, pos, pos_table=None, out=None, out2=None):
    """``(residual fp32, residual in the table's dtype)``: the embedding rows of ``ids``, plus the rows of ``pos`` in
    ``pos_table`` when there is one. ``out`` / ``out2``: where the second one goes (rows may be strided, both alike)."""
    if not table.is_cuda:
        resid = table[ids.long()].float()
        if pos_table is not None:
            resid = resid + pos_table[pos.long().clamp(0, pos_table.shape[0] - 1)].float()
        x = resid.to(table.dtype)
        for o in (out, out2):
            if o is not None:
                o.copy_(x)
        return resid, x if out is None else out
    T, H = ids.shape[0], table.shape[1]
    resid = torch.empty(T, H, device=table.device, dtype=torch.float32)
    x = torch.empty(T, H, device=table.device, dtype=table.dtype) if out is None else out
    assert out2 is None or out2.stride(0) == x.stride(0)
    _call("ab2_embed_rows", _p(ids), _p(table), table.shape[0], _p(pos), _p(pos_table), 0 if pos_table is None else pos_table.shape[0], _p(resid), _p(x),
          _p(out2), x.stride(0), T, H, _dt(table))
    return resid, x


def post_norm(h, w, resid, eps: float, mult: float = 1.0, offset: float = 0.0, w_next=None, offset_next: float = 0.0):
    """``resid += mult * rmsnorm(h) * (offset + w)`` (in place, fp32); returns resid in h's dtype, or with ``w_next``
    ``rmsnorm(resid) * (offset_next + w_next)``. ``h`` is [R, H] or an :class:`ExpertSum`."""
    parts = isinstance(h, ExpertSum)
    src = h.y if parts else h
    assert not (parts and (h.weights is not None or h.shared_logit is not None)), "expert rows summed as they are"
    if not src.is_cuda:
        resid += mult * group_norm_ref(h.dense() if parts else h, offset + w, 1, eps)
        out = resid if w_next is None else group_norm_ref(resid, offset_next + w_next, 1, eps)
        return out.to(src.dtype)
    T, H = resid.shape
    assert src.stride(1) == 1
    x = torch.empty(T, H, device=src.device, dtype=src.dtype)
    base = h.shared if parts else h
    ld = 0 if base is None else base.stride(0)
    y, inv, k, n = (_p(h.y), _p(h.routing.inv), h.routing.k, h.y.shape[0]) if parts else (None, None, 0, 0)
    _call("ab2_post_norm", _p(base), ld, y, inv, k, n, _p(w), offset, mult, _p(resid), _p(w_next), offset_next, _p(x), T, H, eps, _dt(src))
    return x


def residual_norm(h, resid, w_next, eps: float, dtype, vec=None, mult: float = 1.0, out=None):
    """``resid += h + vec`` (in place, fp32; ``h`` is [R, H], an :class:`ExpertSum`, a :class:`BranchSum` or None, ``vec`` [H] or None);
    returns ``mult * rmsnorm(resid) * w_next`` in ``dtype``, or resid itself without ``w_next``. ``out``: where it goes (rows may be
    strided)."""
    if isinstance(h, BranchSum) and resid.is_cuda:
        assert w_next is not None, "branches are summed on the way into a norm"
        return _stream_norm(h, resid, resid, w_next, eps, dtype, vec, mult, out)
    parts = isinstance(h, ExpertSum)
    R, H = resid.shape
    if not resid.is_cuda:
        if h is not None:
            resid += h.float() if torch.is_tensor(h) else h.dense()
        if vec is not None:
            resid += vec
        x = (resid if w_next is None else mult * group_norm_ref(resid, w_next, 1, eps)).to(dtype)
        return x if out is None else out.copy_(x)
    x = torch.empty(R, H, device=resid.device, dtype=dtype) if out is None else out
    base = h.shared if parts else h
    lg = h.shared_logit if parts else None
    assert resid.is_contiguous() and x.dtype == dtype and (base is None or (base.stride(1) == 1 and base.dtype == dtype))
    y, inv, tw, k, n = (_p(h.y), _p(h.routing.inv), _p(h.weights), h.routing.k, h.y.shape[0]) if parts else (None, None, None, 0, 0)
    _call("ab2_residual_norm", _p(base), 0 if base is None else base.stride(0), _p(lg), 0 if lg is None else lg.stride(0), y, inv, tw, k, n, _p(vec), _p(resid),
          _p(w_next), mult, _p(x), x.stride(0), R, H, eps, _dt(x))
    return x


def _stretch(rows: int, blocks: Optional[int]) -> int:
    """Rows that a CTA of the stream kernel walks: few of them make more CTAs, many read less twice (``blocks``: 64-row blocks of the
    portions when rows are shifted, else None)."""
    if blocks is None:
        return 4 if rows >= 2048 else 1
    return 7 if blocks >= 16 else 3


def _stream_norm(src, resid, new, w, eps, dtype, vec=None, mult=1.0, out=None, shift=None):
    """The kernel behind :func:`stream_norm`; ``shift`` = (share, batch, slot states)."""
    R, H = new.shape
    x = torch.empty(R, H, device=new.device, dtype=dtype) if out is None else out
    ids = table = a = c = wa = wb = None
    scale = 1.0
    if isinstance(src, EmbeddingRows):
        ids, table, scale = src.ids, src.table, src.scale
        assert table.is_contiguous() and table.dtype == dtype
    elif isinstance(src, BranchSum):
        a, c, wa, wb, scale = src.left, src.right, src.w_left, src.w_right, src.factor
        assert src.eps == eps
    else:
        a = src
    assert new.is_contiguous() and (resid is None or resid.is_contiguous()) and x.dtype == dtype and x.stride(1) == 1
    assert all(t is None or (t.dtype == dtype and t.stride(1) == 1 and t.shape == (R, H)) for t in (a, c))
    share, b, S = shift or (None, None, None)
    nb = 0 if b is None or b.blocks is None else b.blocks.shape[0]
    batch = (None,) * 4 + (0, 0) if b is None else (_p(b.cu), _p(b.start), _p(b.state), _p(b.blocks), nb, b.n_dec)
    _call("ab2_stream_norm", _p(ids), _p(table), 0 if table is None else table.shape[0], _p(a), 0 if a is None else a.stride(0), _p(c),
          0 if c is None else c.stride(0), _p(wa), _p(wb), scale, _p(vec), _p(resid), _p(new), _p(w), mult, _p(share), _p(x), x.stride(0), *batch,
          _stretch(R, None if b is None else nb),
          _p(S), R, H, eps, _dt(x))
    return x


def stream_norm(src, resid, w, eps: float, dtype, vec=None, share=None, b: Optional[RaggedBatch] = None, S=None):
    """What a mixer reads: ``(stream, x)`` with stream = ``resid`` + ``src`` + ``vec`` in fp32 (``src``: [R, H], an :class:`EmbeddingRows`, which
    begins the stream, a :class:`BranchSum`, an :class:`ExpertSum` or None) and x = h = ``rmsnorm(stream) * w`` in ``dtype``. With a
    token shift (``share`` [H]) x = ``h + (h' - h) * share``, h' being the h of the sequence's previous token: the row before, or what
    the entry's slot in S [slots, H] holds (zeros when the sequence is new); S is left at every entry's last h. ``resid`` may be
    overwritten."""
    if isinstance(src, ExpertSum):
        residual_norm(src, resid, None, eps, dtype)
        src = None
    like = src.ids if isinstance(src, EmbeddingRows) else resid
    if like.is_cuda:
        R = like.shape[0]
        new = resid if share is None and resid is not None else torch.empty(R, w.shape[0], device=like.device, dtype=torch.float32)
        return new, _stream_norm(src, resid, new, w, eps, dtype, vec, shift=None if share is None else (share, b, S))
    add = 0.0 if src is None else (src.float() if torch.is_tensor(src) else src.dense())
    stream = (0.0 if resid is None else resid) + add + (0.0 if vec is None else vec)
    h = group_norm_ref(stream, w, 1, eps)
    if share is None:
        return stream, h.to(dtype)
    x = torch.zeros_like(h)
    for _, r0, r1, st, sl in _segments(b):
        old = S[sl] if st > 0 else torch.zeros_like(h[0])
        before = torch.cat([old[None], h[r0:r1 - 1]])
        x[r0:r1] = h[r0:r1] + (before - h[r0:r1]) * share
        S[sl] = h[r1 - 1]
    return stream, x.to(dtype)


# ----------------------------------------------------------------------------- rotated positions
def rotary_table(pos, freq, mult):
    """``(cos, sin)`` of the rows' angles times ``mult``: pos [R], freq [P] double in turns per position, mult [P] fp32. Returns
    [R, P, 2] fp32."""
    if not pos.is_cuda:
        turns = pos.double()[:, None] * freq
        a = ((turns - turns.round()) * (2 * math.pi)).float()
        return torch.stack([torch.cos(a) * mult, torch.sin(a) * mult], -1)
    out = torch.empty(pos.shape[0], freq.shape[0], 2, device=pos.device, dtype=torch.float32)
    _call("ab2_rotary_table", _p(pos), _p(freq), _p(mult), _p(out), pos.shape[0], freq.shape[0])
    return out


def rotate_ref(x, cs, interleaved: bool):
    """x [R, ..., D] in fp32 with its first pairs turned; cs [R, half, 2]."""
    half = cs.shape[1]
    x = x.float().clone()
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    c, s = cs[..., 0].reshape(shape), cs[..., 1].reshape(shape)
    a, b = (slice(0, 2 * half, 2), slice(1, 2 * half, 2)) if interleaved else (slice(0, half), slice(half, 2 * half))
    u, v = x[..., a].clone(), x[..., b].clone()
    x[..., a], x[..., b] = u * c - v * s, v * c + u * s
    return x


def _rot(rot):
    """Arguments of a stretch [R, half, 2] of a step's table."""
    return _p(rot), rot.stride(0) // 2, rot.shape[1]


def qk_head_norm_append(z, wq, wk, eps: float, rot, interleaved: bool, b: RaggedBatch, kc, vc, Hq: int, unit: bool = False, q_factor=None,
                        key_factor=None):
    """Per-head RMS norms of q and k (weights [D] shared by the heads; None: no norm, or with ``unit`` one without weights), rotation
    of the first ``2 * rot.shape[1]`` numbers of every head (rot None: none), q times ``q_factor`` [Hq], then k and v into the cache rows of
    ``b.slots``; returns q [R, Hq, D]. ``z`` rows begin with q | k | v. A norm without weights may as well follow the rotation, which keeps a
    head's length. With ``key_factor`` [S, Hkv] (fp32) keys are cached as they are, the numbers that norm them go there, and there is no v."""
    Hkv, D = kc.shape[1], kc.shape[2]
    Dv = 0 if vc is None else vc.shape[2]
    R, nq, nk = z.shape[0], Hq * D, Hkv * D
    if not z.is_cuda:
        ones = torch.ones(D)

        def turn(x, w):
            w = ones if w is None and unit else w
            x = x.float() if w is None else group_norm_ref(x, w, 1, eps)
            return x if rot is None else rotate_ref(x, rot, interleaved)
        ok = b.slots >= 0
        at, k = b.slots[ok].long(), z[:, nq:nq + nk].reshape(R, Hkv, D)
        if key_factor is None:
            kc[at] = turn(k, wk).to(z.dtype)[ok]
        else:
            kc[at] = k[ok]
            key_factor[at] = torch.rsqrt(k.float().pow(2).mean(-1) + eps)[ok]
        if vc is not None:
            vc[at] = z[ok, nq + nk:nq + nk + Hkv * Dv].reshape(-1, Hkv, Dv)
        q = turn(z[:, :nq].reshape(R, Hq, D), wq)
        return (q if q_factor is None else q * q_factor[:, None]).to(z.dtype)
    q = torch.empty(R, Hq, D, device=z.device, dtype=z.dtype)
    turned = (None, 0, 0) if rot is None else _rot(rot)
    _call("ab2_qk_head_norm_append", _p(z), z.stride(0), _p(wq), _p(wk), *turned, int(interleaved), _p(b.slots), _p(q), _p(kc), _p(vc), R, Hq, Hkv, D,
          Hkv * Dv, eps, int(unit), _p(q_factor), _p(key_factor), _dt(z))
    return q


# ----------------------------------------------------------------------------- attention
class AttnExtra(ctypes.Structure):
    """Optional inputs of the attention kernels (the struct of the same name in csrc/mixer_common.cuh)."""

    _fields_ = ([(n, ctypes.c_void_p) for n in ("q2", "k2", "gate", "sink", "kf")] +
                [(n, ctypes.c_longlong) for n in ("ldq", "hsq", "ldq2", "hsq2", "ldk", "ldv", "ldk2", "ldo", "ldg")] +
                [(n, ctypes.c_int) for n in ("D2", "gate_per_head")] + [(n, ctypes.c_float) for n in ("sink_const", "out_scale")])


def _extra(sink=None, gate=None, gate_per_head=False, out_scale=1.0, **strides) -> AttnExtra:
    x = AttnExtra(sink_const=-math.inf if sink is None or torch.is_tensor(sink) else sink, out_scale=out_scale, gate_per_head=int(gate_per_head), **strides)
    if torch.is_tensor(sink):
        x.sink = _p(sink)
    if gate is not None:
        x.gate, x.ldg = _p(gate), gate.stride(0)
    return x


def softmax_with_sink(s, sink):
    """Softmax of s [H, i, j] with ``exp(sink)`` added to the denominator (a number or one per head; None: nothing)."""
    if sink is None:
        return torch.softmax(s, -1)
    sink = (sink if torch.is_tensor(sink) else torch.full((s.shape[0],), float(sink))).float()[:, None, None].expand(-1, s.shape[1], 1)
    return torch.softmax(torch.cat([s, sink], -1), -1)[..., :-1]


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


def chunk_attention_ref(q, kc, vc, b: RaggedBatch, scale, softcap, r1, r2, chunk, window=0, sink=None, key_factor=None):
    R, Hq, D = q.shape
    Hkv, Dv = kc.shape[1], vc.shape[2]
    out = torch.zeros(R, Hq, Dv, dtype=q.dtype)
    rep, ps = Hq // Hkv, b.page_size
    for e, r0, r1_, st, _ in _segments(b):
        end = st + r1_ - r0
        lo = (st // chunk) * chunk if chunk else (max(0, st - window + 1) if window else 0)
        j = torch.arange(lo, end)
        rows = b.pages[e][(j // ps - b.page_base[e]).long()].long() * ps + j % ps
        k = kc[rows].float() if key_factor is None else kc[rows].float() * key_factor[rows][..., None]
        k = k.repeat_interleave(rep, 1)
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
        if window:
            see &= dist < window
        s = s.masked_fill(~see, float("-inf"))
        out[r0:r1_] = torch.einsum("hij,jhd->ihd", softmax_with_sink(s, sink), v).to(q.dtype)
    return out


def chunk_attention(q, kc, vc, b: RaggedBatch, scale: float, softcap: float = 0.0, r1=None, r2=None, chunk: int = 0, window: int = 0, sink=None, gate=None,
                    out_scale: float = 1.0, out=None, key_factor=None):
    """Attention of the step's queries over the paged cache (their own keys already appended): ``softcap *
    tanh(q.k * scale / softcap)`` minus ``r1[h] * ln(1 + r2[h] * distance)``, softmax over the earlier positions of
    the query's own chunk of ``chunk`` positions, or over itself and the ``window - 1`` before it (0: no limit), with
    ``exp(sink)`` more in the denominator; then times ``sigmoid(gate)`` (gate [R, Hq * Dv], rows may be strided) and ``out_scale``.
    Without ``vc`` the keys are the values; ``key_factor`` [S, Hkv] (fp32) multiplies every key's scores, not its value.
    Returns [R, Hq, Dv], in ``out`` [R, Hq * Dv] (rows may be strided) when that is given."""
    R, Hq, D = q.shape
    vc = kc if vc is None else vc
    Hkv, Dv = kc.shape[1], vc.shape[2]
    if not q.is_cuda:
        o = chunk_attention_ref(q, kc, vc, b, scale, softcap, r1, r2, chunk, window, sink, key_factor)
        if gate is not None or out_scale != 1.0:
            o = (o.float() * (1.0 if gate is None else torch.sigmoid(gate.float()).view(R, Hq, Dv)) * out_scale).to(q.dtype)
        return o if out is None else out.copy_(o.view(R, -1))
    if out is None:
        out = torch.empty(R, Hq, Dv, device=q.device, dtype=q.dtype)
    x = _extra(sink, gate, out_scale=out_scale, ldo=out.stride(0), kf=_p(key_factor))
    common = (_p(kc), _p(vc), _p(b.pages), _p(b.page_base), b.pages.shape[1], b.page_size, Hq, Hkv, D, Dv, scale, softcap, _p(r1), _p(r2), chunk, window,
              ctypes.byref(x))
    fast = q.dtype == torch.bfloat16 and D % 8 == 0 and Dv % 8 == 0 and D <= 128 and Dv <= 128
    tiles = fast and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0 and (gate is None or (gate.stride(0) % 8 == 0 and gate.data_ptr() % 16 == 0))
    tiles = tiles and (key_factor is None or (softcap == 0.0 and r1 is None))
    nd = b.n_dec
    if nd:
        if fast and Hq // Hkv <= 16:
            _call("ab2_chunk_decode", _p(q), _p(b.pos), _p(b.slots), _p(out), nd, *common)
        else:
            _call("ab2_chunk_attn_plain", _p(q), _p(b.pos), _p(b.slots), _p(b.row_entry), _p(out), nd, *common, _dt(q))
    if R > nd:
        if tiles and b.page_size in (16, 32, 64, 128) and b.tiles is not None:
            _call("ab2_chunk_prefill", _p(q), _p(b.cu), _p(b.start), _p(b.tiles), b.tiles.shape[0], _p(out), R, kc.shape[0], Hkv * D, Hkv * Dv, *common)
        else:
            if gate is not None:
                x.gate = _p(gate[nd:])
            _call("ab2_chunk_attn_plain", _p(q[nd:]), _p(b.pos[nd:]), _p(b.slots[nd:]), _p(b.row_entry[nd:]), _p(out[nd:]), R - nd, *common, _dt(q))
    return out


# ----------------------------------------------------------------------------- attention on cached latents
def latent_norm_append(x, wq, wc, eps: float, b: RaggedBatch, cache):
    """RMS norms of the two parts of ``x`` (query latent | cached latent), the second into the cache rows of ``b.slots``;
    returns the first [R, q_rank]. ``cache`` [S, 1, kv_rank]."""
    nq, nc = wq.shape[0], wc.shape[0]
    R = x.shape[0]
    if not x.is_cuda:
        ok = b.slots >= 0
        cache[b.slots[ok].long(), 0] = group_norm_ref(x[:, nq:], wc, 1, eps).to(x.dtype)[ok]
        return group_norm_ref(x[:, :nq], wq, 1, eps).to(x.dtype)
    cq = torch.empty(R, nq, device=x.device, dtype=x.dtype)
    _call("ab2_qk_norm_append", _p(x), x.stride(0), _p(wq), _p(wc), _p(b.slots), _p(cq), _p(cache), None, R, nq, nc, 0, eps, _dt(x))
    return cq


def latent_rope_append(z, wc, eps: float, rot, interleaved: bool, b: RaggedBatch, cache, H: int, D: int):
    """Rows of ``z``: queries [H, D + r] | latent | key part [r]; r = ``2 * rot.shape[1]``. Turns the last r numbers of every query
    head in place; the RMS-normed latent and the turned key part go into the cache rows of ``b.slots`` (cache [S, 1, C + r])."""
    r = 2 * rot.shape[1]
    C, R, nq = cache.shape[2] - r, z.shape[0], H * (D + r)
    if not z.is_cuda:
        q = z[:, :nq].view(R, H, D + r)
        q[..., D:] = rotate_ref(q[..., D:], rot, interleaved).to(z.dtype)
        ok = b.slots >= 0
        row = torch.cat([group_norm_ref(z[:, nq:nq + C], wc, 1, eps), rotate_ref(z[:, nq + C:nq + C + r], rot, interleaved)], -1)
        cache[b.slots[ok].long(), 0] = row.to(z.dtype)[ok]
        return
    _call("ab2_latent_rope_append", _p(z), z.stride(0), _p(wc), *_rot(rot), int(interleaved), _p(b.slots), _p(cache), R, H, D, C, eps, _dt(z))


def latent_attention_ref(q, cache, w_kv, Dv, b: RaggedBatch, scale, window, rot_dim=0, sink=None):
    R, H, D = q.shape[0], q.shape[1], q.shape[2] - rot_dim
    C, ps = w_kv.shape[1], b.page_size
    out = torch.zeros(R, H, Dv, dtype=q.dtype)
    for e, r0, r1, st, _ in _segments(b):
        i = torch.arange(st, st + r1 - r0)
        j = torch.arange(max(0, st - window + 1) if window else 0, st + r1 - r0)
        rows = b.pages[e][(j // ps - b.page_base[e]).long()].long() * ps + j % ps
        kv = F.linear(cache[rows, 0, :C].float(), w_kv.float())
        k, v = kv[:, :H * D].view(-1, H, D), kv[:, H * D:].view(-1, H, Dv)
        s = torch.einsum("ihd,jhd->hij", q[r0:r1, :, :D].float(), k)
        if rot_dim:
            s = s + torch.einsum("ihd,jd->hij", q[r0:r1, :, D:].float(), cache[rows, 0, C:].float())
        dist = i[:, None] - j[None, :]
        see = (dist >= 0) & (dist < window) if window else dist >= 0
        w = softmax_with_sink((s * scale).masked_fill(~see, float("-inf")), sink)
        out[r0:r1] = torch.einsum("hij,jhd->ihd", w, v).to(q.dtype)
    return out


# portions of up to this many tokens (on average) read the latents as single tokens do: working out keys and values of a
# whole window would cost more than it saves
SHORT_PORTION = 16


def latent_attention(q, cache, w_kv, Dv: int, b: RaggedBatch, scale: float, window: int = 0, rot_dim: int = 0, sink=None, gate=None):
    """Attention of the step's queries q [R, H, D + rot_dim] (rows may be strided) over cached latents (the step's own already
    appended): head h has keys ``w_kv[h D:(h + 1) D] c`` and values ``w_kv[H D + h Dv:...] c``, the last ``rot_dim`` numbers of a
    query meet the part behind the latent, which is every head's key; softmax of ``scale * q.k`` over the position itself and
    the ``window - 1`` before it (0: no limit), with ``exp(sink)`` more in the denominator; every head's output times
    ``sigmoid(gate)`` (gate [R, H], rows may be strided). cache [S, 1, C + rot_dim], w_kv [H (D + Dv), C]. Returns [R, H, Dv]."""
    R, H, D = q.shape[0], q.shape[1], q.shape[2] - rot_dim
    C, ld = w_kv.shape[1], cache.shape[2]
    if not q.is_cuda:
        o = latent_attention_ref(q, cache, w_kv, Dv, b, scale, window, rot_dim, sink)
        return o if gate is None else (o.float() * torch.sigmoid(gate.float())[..., None]).to(o.dtype)
    w_k, w_v = w_kv[:H * D].view(H, D, C), w_kv[H * D:].view(H, Dv, C)
    out = torch.empty(R, H, Dv, device=q.device, dtype=q.dtype)
    nd, bf16 = b.n_dec, q.dtype == torch.bfloat16
    q1, q2, c2 = q[:, :, :D], q[:, :, D:], cache[:, :, C:]
    hs = max(q.stride(1), D + rot_dim)
    paged = bf16 and C % 8 == 0 and b.page_size in (16, 32, 64, 128) and rot_dim % 8 == 0 and rot_dim <= 64
    part2 = not rot_dim or (D % 8 == 0 and q.stride(0) % 8 == 0 and hs % 8 == 0 and q.data_ptr() % 16 == 0)
    fast_rows = paged and part2 and C <= 512
    fast_tiles = paged and part2 and D % 8 == 0 and Dv % 8 == 0 and D <= 128 and Dv <= 128 and q.stride(0) % 8 == 0 and hs % 8 == 0 and q.data_ptr() % 16 == 0
    whole = R > nd and fast_tiles and R - nd > SHORT_PORTION * (b.n_entries - nd)
    n = nd if whole else R
    second = dict(q2=_p(q2), ldq2=q.stride(0), hsq2=hs, D2=rot_dim) if rot_dim else {}
    if n:
        # keys applied to the queries: scores against the latents themselves, the values' part after the sum
        qc = head_linear(q1[:n], w_k, w_kn=True)
        oc = torch.empty_like(qc)
        x = _extra(sink, gate, True, ldk=ld, ldv=ld, **second, **(dict(k2=_p(c2), ldk2=ld) if rot_dim else {}))
        args = (_p(qc), _p(b.pos), _p(b.slots), _p(b.row_entry), _p(oc), n)
        if fast_rows:
            _call("ab2_latent_decode", *args, _p(cache), cache.shape[0], _p(b.pages), _p(b.page_base), b.pages.shape[1], b.page_size, H, C, scale, window,
                  ctypes.byref(x))
        else:
            _call("ab2_chunk_attn_plain", *args, _p(cache), _p(cache), _p(b.pages), _p(b.page_base), b.pages.shape[1], b.page_size, H, 1, C, C, scale, 0.0,
                  None, None, 0, window, ctypes.byref(x), _dt(q))
        head_linear(oc, w_v, out[:n])
    if whole:
        seen, ps = b.seen[window], b.page_size
        rows = cache.view(-1, ps * ld).index_select(0, seen.pages).view(-1, ld)
        kv = linear(rows[:, :C], w_kv)
        x = _extra(sink, gate, True, ldq=q.stride(0), hsq=hs, **second, **(dict(k2=_p(rows[:, C:]), ldk2=ld) if rot_dim else {}))
        _call("ab2_chunk_prefill", _p(q), _p(b.cu), _p(b.start), _p(b.tiles), b.tiles.shape[0], _p(out), R, kv.shape[0], kv.stride(0), kv.stride(0),
              _p(kv), _p(kv[:, H * D:]), _p(seen.table), _p(seen.base), seen.table.shape[1], ps, H, H, D, Dv, scale, 0.0, None, None, 0, window,
              ctypes.byref(x))
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


# ----------------------------------------------------------------------------- minGRU
def min_gru(zug, bias, b: RaggedBatch, S, out=None, cluster: int = 0):
    """Element-wise ``S_t = (1 - z) S_(t-1) + z c`` with ``z = sigmoid(zr + bz)``, ``u = ur + bu`` and c = u + 1/2 where u >= 0, else sigmoid(u);
    returns ``S * silu(g)`` [R, W] in zug's dtype and leaves the last state of every entry in its slot. zug [R, 3 W] rows zr | ur | g (may be
    strided), bias [2 W] bz | bu, S [slots, W]. ``cluster``: CTAs that share a portion (0: by size)."""
    R, W = zug.shape[0], S.shape[1]
    if not zug.is_cuda:
        z, u, g = zug.float().view(R, 3, W).unbind(1)
        z, u = z + bias[:W], u + bias[W:]
        keep, x = torch.sigmoid(-z), torch.sigmoid(z) * torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
        y = torch.zeros(R, W)
        for _, r0, r1, st, sl in _segments(b):
            h = S[sl].clone() if st > 0 else torch.zeros(W)
            for t in range(r0, r1):
                h = keep[t] * h + x[t]
                y[t] = h
            S[sl] = h
        y = (y * F.silu(g)).to(zug.dtype)
        return y if out is None else out.copy_(y)
    out = torch.empty(R, W, device=zug.device, dtype=zug.dtype) if out is None else out
    assert zug.stride(1) == 1 and bias.is_contiguous() and out.stride(1) == 1
    _call("ab2_min_gru", _p(zug), zug.stride(0), _p(bias), _p(b.cu), _p(b.start), _p(b.state), b.n_dec, b.n_entries, 0 if b.blocks is None else b.blocks.shape[0],
          cluster, _p(S), _p(out), out.stride(0), W, _dt(zug))
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


# ----------------------------------------------------------------------------- retention
def retention(z, decay, log2_decay, rot, eps: float, scale: float, out, heads: int, dim: int, vdim: int, b: RaggedBatch, S):
    """Per head ``S_t = decay S_(t-1) + k_t v_t^T`` and ``o_t = S_t^T q_t`` with turned q and k (halves paired) and k times
    ``dim ** -0.5``; every head's o over its root mean square, times ``silu(gate)`` and ``scale``, goes to ``out`` [R, heads * vdim] (rows
    may be strided). ``z`` rows begin with q | k | v | gate; S [slots, heads, vdim, dim] is left at every entry's last token."""
    R, nq, nv = z.shape[0], heads * dim, heads * vdim
    k_scale = dim ** -0.5
    if not z.is_cuda:
        q, k = (rotate_ref(z[:, i * nq:(i + 1) * nq].reshape(R, heads, dim), rot, False) for i in (0, 1))
        k, v = k * k_scale, z[:, 2 * nq:2 * nq + nv].float().view(R, heads, vdim)
        o = torch.zeros(R, heads, vdim)
        for e, r0, r1, st, sl in _segments(b):
            h = S[sl].clone() if st > 0 else torch.zeros(heads, vdim, dim)
            for t in range(r0, r1):
                h = decay[:, None, None] * h + v[t][:, :, None] * k[t][:, None, :]
                o[t] = (h * q[t][:, None, :]).sum(-1)
            S[sl] = h
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)
        out.copy_((o.reshape(R, nv) * F.silu(z[:, 2 * nq + nv:2 * nq + 2 * nv].float()) * scale).to(z.dtype))
        return out
    nd, E, half = b.n_dec, b.n_entries, rot.shape[1]
    if nd:
        _call("ab2_retention_decode", _p(z), z.stride(0), *_rot(rot), _p(decay), k_scale, _p(b.start), _p(b.state), _p(S), _p(out), out.stride(0), nd, heads,
              dim, vdim, eps, scale, _dt(z))
    if E > nd:
        y = torch.empty(R - nd, nv, device=z.device, dtype=torch.float32)
        blocks = z.dtype == torch.bfloat16 and dim <= 128 and dim % 8 == 0 and vdim % 8 == 0 and half % 4 == 0 and z.stride(0) % 8 == 0 and z.data_ptr() % 16 == 0
        _call("ab2_retention_portions", _p(z), z.stride(0), *_rot(rot), _p(decay), _p(log2_decay), k_scale, _p(b.cu), _p(b.start), _p(b.state), nd, E, _p(S),
              _p(y), heads, dim, vdim, int(blocks), _dt(z))
        gate = z[nd:, 2 * nq + nv:]
        _call("ab2_head_norm_gate", _p(y), _p(gate), z.stride(0), _p(out[nd:]), out.stride(0), R - nd, heads, vdim, eps, scale, _dt(z))
    return out


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


def gelu_erf(x):
    """``z (1 + erf(z / sqrt 2)) / 2``."""
    if not x.is_cuda:
        return F.gelu(x.float()).to(x.dtype)
    out = torch.empty(x.shape, device=x.device, dtype=x.dtype)
    _call("ab2_gelu_erf", _p(x), x.stride(0), _p(out), x.shape[0], x.shape[1], _dt(x))
    return out


def glu_clamped(gu, limit: float, alpha: float, routing: Optional[Routing] = None):
    """``g sigmoid(alpha g) (u + 1)`` with ``g = min(w g', limit)`` and ``u = clamp(w u', -limit, limit)`` for rows g' | u'.
    With a routing the rows are its expert-sorted ones and w is each row's gate weight, else 1."""
    I = gu.shape[1] // 2
    if not gu.is_cuda:
        z = gu.float()
        if routing is not None:
            z = z * routing.topw.reshape(-1)[routing.order.long()][:, None]
        g, u = z[:, :I].clamp(max=limit), z[:, I:].clamp(-limit, limit)
        return (g * torch.sigmoid(alpha * g) * (u + 1)).to(gu.dtype)
    out = torch.empty(gu.shape[0], I, device=gu.device, dtype=gu.dtype)
    order, topw = (None, None) if routing is None else (_p(routing.order), _p(routing.topw))
    _call("ab2_glu_clamped", _p(gu), gu.stride(0), order, topw, _p(out), gu.shape[0], I, limit, alpha, _dt(gu))
    return out


def side_gate(g, ids, table, col: int):
    """``gelu_tanh(g) * table[ids, col:col + D]`` for g [R, D]."""
    D = g.shape[1]
    if not g.is_cuda:
        return (F.gelu(g.float(), approximate="tanh") * table[ids.long(), col:col + D].float()).to(g.dtype)
    out = torch.empty(g.shape[0], D, device=g.device, dtype=g.dtype)
    _call("ab2_side_gate", _p(g), g.stride(0), _p(ids), _p(table), table.shape[0], table.stride(0), col, _p(out), g.shape[0], D, _dt(g))
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
    "ab2_embed_rows": [_V, _V, _I, _V, _V, _I, _V, _V, _V, _lib.c_ll, _I, _I, _I],
    "ab2_residual_norm": [_V, _lib.c_ll, _V, _lib.c_ll, _V, _V, _V, _I, _I, _V, _V, _V, _F, _V, _lib.c_ll, _I, _I, _F, _I],
    "ab2_rotary_table": [_V] * 4 + [_I, _I],
    "ab2_qk_head_norm_append": [_V, _lib.c_ll, _V, _V, _V, _I, _I, _I] + [_V] * 4 + [_I] * 5 + [_F, _I, _V, _V, _I],
    "ab2_stream_norm": [_V, _V, _I, _V, _lib.c_ll, _V, _lib.c_ll, _V, _V, _F] + [_V] * 4 + [_F, _V, _V, _lib.c_ll] + [_V] * 4 + [_I] * 3 + [_V, _I, _I, _F, _I],
    "ab2_min_gru": [_V, _lib.c_ll] + [_V] * 4 + [_I] * 4 + [_V, _V, _lib.c_ll, _I, _I],
    "ab2_latent_rope_append": [_V, _lib.c_ll, _V, _V, _I, _I, _I, _V, _V] + [_I] * 4 + [_F, _I],
    "ab2_retention_decode": [_V, _lib.c_ll, _V, _I, _I, _V, _F] + [_V] * 4 + [_lib.c_ll] + [_I] * 4 + [_F, _F, _I],
    "ab2_retention_portions": [_V, _lib.c_ll, _V, _I, _I, _V, _V, _F] + [_V] * 3 + [_I, _I, _V, _V] + [_I] * 5,
    "ab2_head_norm_gate": [_V, _V, _lib.c_ll, _V, _lib.c_ll, _I, _I, _I, _F, _F, _I],
    "ab2_post_norm": [_V, _lib.c_ll, _V, _V, _I, _I, _V, _F, _F, _V, _V, _F, _V, _I, _I, _F, _I],
    "ab2_gemm_heads": [_V] * 3 + [_I] * 8,
    "ab2_chunk_attn_plain": [_V] * 5 + [_I] + [_V] * 4 + [_I] * 6 + [_F, _F, _V, _V, _I, _I, _V, _I],
    "ab2_chunk_decode": [_V] * 4 + [_I] + [_V] * 4 + [_I] * 6 + [_F, _F, _V, _V, _I, _I, _V],
    "ab2_chunk_prefill": [_V] * 4 + [_I, _V, _I, _I, _lib.c_ll, _lib.c_ll] + [_V] * 4 + [_I] * 6 + [_F, _F, _V, _V, _I, _I, _V],
    "ab2_latent_decode": [_V] * 5 + [_I, _V, _I, _V, _V] + [_I] * 4 + [_F, _I, _V],
    "ab2_gelu_erf": [_V, _lib.c_ll, _V, _I, _I, _I],
    "ab2_glu_clamped": [_V, _lib.c_ll, _V, _V, _V, _I, _I, _F, _F, _I],
    "ab2_side_gate": [_V, _lib.c_ll, _V, _V, _I, _lib.c_ll, _I, _V, _I, _I, _I],
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
