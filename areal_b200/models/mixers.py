"""Mixer stacks: decoder models whose layers are listed one by one, each with its own token mixer and feed-forward.

Four designs are built from the parts below (:data:`DESIGNS`):

* Kagolix normalises twice around every sublayer, in groups: ``x += norm_b(f(norm_a(x)))``; its output is capped;
* Vogilix normalises the sublayer's output only, ``x += m * norm(f(x))``, adds a learned vector per position to the
  embedding, and ends every layer with a gated input from the layer's own part of a per-token row;
* Bumotar normalises before every sublayer, ``x += f(norm(x))``, and runs a stretch of its layers several times in a row with
  the same weights, every pass with caches and states of its own and with the embedding mixed in again before it;
* Goganex does so too, with nothing between the passes, scales the embedding, and blends what a mixer reads with the same row of
  the token before (token shift).

The sum x stays in 32 bits in all of them. The mixers

* ``attention``: grouped-query attention inside chunks of positions, whole-projection RMS norms on q and k, no rotation,
  capped scores and a logarithmic distance bias (two numbers per head);
* ``rglru``: a gated branch times a real-gated linear recurrence behind a short causal convolution;
* ``mamba2``: the scalar-decay state-space recurrence, gated and normalised in groups;
* ``latent_attention``: keys and values of all heads from one normed latent per token (the only thing cached), queries from
  a latent of their own, no positions, a sliding window; or (:class:`RotaryLatentAttention`) queries straight from the layer's
  input and beside the latent one rotated key part for all heads, sinks and a gate per head;
* ``parallel``: branches side by side on one input and one output projection: windowed attention with rotated, normed
  queries and keys, capped scores, a sink and gated channels; retention (linear attention with a fixed decay per head); or
  (:class:`NormedParallel`) on output projections of their own whose results are normed before they are added: attention without
  positions whose keys are its values, and minGRU;
* ``attention`` as :class:`RotaryAttention`: rotated queries and keys of unit length, a factor per head, a sink;

and the feed-forwards (dense with xIELU, the exact GELU or clamped gated units; experts behind a softmax or a sigmoid router, weighted at their
output or at their input, with or without a gated shared expert) are built from the ops of :mod:`..ops.mixer_ops`. A forward
pass runs the rows of one step (:class:`~..ops.mixer_ops.RaggedBatch`) from the pages and state slots of
:class:`~..engine.state_cache.StateCache`; whole prompts, portions and single tokens are the same call.

Matrices are stored in the model's dtype, everything that is used in 32 bits (norm weights, biases, taps, decay and bias
parameters) as fp32. Serving only: there is no backward pass.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch
import torch.nn as nn

from ..ops import functional as OF
from ..ops import mixer_ops as M
from .config import ModelConfig
from .decoder import CausalLM


def check_layer_specs(arch: str, layers: list, width: int, norm_groups: int) -> None:
    """Raises ``ValueError`` for a layer list that no kernel could run."""
    design = DESIGNS[arch]
    if width % max(1, norm_groups):
        raise ValueError(f"norm groups {norm_groups} do not divide the width {width}")
    for i, e in enumerate(layers):
        t, m, mlp = e["type"], e["mixer"], e["mlp"]
        if t not in design.mixers:
            raise ValueError(f"layer {i}: unknown mixer '{t}' (have {sorted(design.mixers)})")
        design.mixers[t].check(m, f"layer {i}: ")
        if mlp and mlp["kind"] not in design.mlps:
            raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
        if mlp and mlp["kind"] == "moe" and not 1 <= mlp["router"]["top"] <= mlp["router"]["experts"]:
            raise ValueError(f"layer {i}: {mlp['router']['top']} of {mlp['router']['experts']} experts")


class _Block(nn.Module):
    """Parameter helpers: ``mat`` in the model's dtype, ``vec`` in fp32."""

    def __init__(self, cfg: ModelConfig, dtype, device):
        super().__init__()
        self.eps = cfg.rms_norm_eps
        self._dtype, self._device = dtype, device

    def mat(self, *shape):
        return nn.Parameter(torch.empty(*shape, dtype=self._dtype, device=self._device))

    def vec(self, *shape):
        return nn.Parameter(torch.empty(*shape, dtype=torch.float32, device=self._device))

    carried = {}             # what the layer around the block keeps in a request's slot
    lists_pages = False      # its portions want the pages that they see in one list

    def cache_shapes(self) -> dict:
        return {}

    def memory(self) -> dict:
        """Shapes of what the cache holds for the block, per token and per request."""
        return {**self.cache_shapes(), **self.carried}

    def const(self, values):
        """Constants of the configuration as an fp32 buffer (no part of a checkpoint)."""
        return torch.tensor(values, dtype=torch.float32, device=self._device)

    @staticmethod
    def check(m, where):
        """Raises ``ValueError`` for sizes that no kernel could run."""

    rotary = None            # (frequencies, factor of cos and sin) when the block rotates; its column in the step's table is ``rot_at``

    def rot(self, b):
        return b.rot[:, self.rot_at:self.rot_at + len(self.rotary[0])]


def _need(ok, where, what):
    if not ok:
        raise ValueError(where + what)


def _check_heads(m, where):
    _need(min(m[k] for k in ("heads", "kv_heads", "dim", "vdim")) >= 1 and m["heads"] % m["kv_heads"] == 0, where,
          f"{m['heads']} query heads over {m['kv_heads']} key/value heads")


# ----------------------------------------------------------------------------- rotation frequencies
def rotary_frequencies(rot: dict):
    """(frequencies, 1.0) of ``rot.dims / 2`` pairs, all divided by ``rot.scaling.factor`` when there is one."""
    f = float((rot.get("scaling") or {}).get("factor") or 1.0)
    return tuple(rot["base"] ** (-2.0 * i / rot["dims"]) / f for i in range(rot["dims"] // 2)), 1.0


def yarn_frequencies(rot: dict):
    """(frequencies, factor of cos and sin) under YaRN: pairs that turn more than ``fast`` times within ``original`` positions
    keep their frequency, those that turn less than ``slow`` times are stretched by ``factor``, with a ramp between."""
    s = rot.get("scaling")
    if not s:
        return rotary_frequencies(rot)
    dims, base = rot["dims"], float(rot["base"])
    at = [dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base)) for turns in (s["fast"], s["slow"])]
    lo, hi = max(math.floor(at[0]), 0), min(math.ceil(at[1]), dims - 1)
    out = []
    for i in range(dims // 2):
        f, r = base ** (-2.0 * i / dims), min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1.0 - r))
    return tuple(out), 0.1 * math.log(s["factor"]) + 1.0


def llama3_frequencies(rot: dict):
    """(frequencies, 1.0) scaled by wavelength: pairs that turn more than ``high`` times within ``original`` positions keep their
    frequency, those that turn less than ``low`` times are slowed by ``factor``, in between the two are blended."""
    base, s = rotary_frequencies(dict(rot, scaling=None))[0], rot.get("scaling")
    if not s:
        return base, 1.0
    out = []
    for f in base:
        turns = s["original"] * f / (2.0 * math.pi)
        keep = 1.0 if turns > s["high"] else (0.0 if turns < s["low"] else (turns - s["low"]) / max(s["high"] - s["low"], 1e-30))
        out.append((1.0 - keep) * f / s["factor"] + keep * f)
    return tuple(out), 1.0


class ChunkAttention(_Block):
    @staticmethod
    def check(m, where):
        _need(m["heads"] % m["kv_heads"] == 0, where, f"{m['heads']} query heads over {m['kv_heads']} key/value heads")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        H, w = cfg.hidden_size, m
        self.nq, self.nkv, self.D, self.Dv = w["heads"], w["kv_heads"], w["dim"], w["vdim"]
        self.scale, self.softcap = float(w["scale"]), float(w.get("softcap") or 0.0)
        self.chunk = int((w.get("mask") or {}).get("size") or 0)
        self.qkv_proj = self.mat((self.nq + self.nkv) * self.D + self.nkv * self.Dv, H)
        self.q_norm, self.k_norm = self.vec(self.nq * self.D), self.vec(self.nkv * self.D)
        self.dist_r1, self.dist_r2 = self.vec(self.nq), self.vec(self.nq)
        self.o_proj = self.mat(H, self.nq * self.Dv)

    def cache_shapes(self):
        return {"kv": ((self.nkv, self.D), (self.nkv, self.Dv))}

    def first_visible(self, pos: int) -> int:
        return pos // self.chunk * self.chunk if self.chunk else 0

    @property
    def span(self) -> int:
        return self.chunk

    def forward(self, x, b, lc):
        q = M.qk_norm_append(M.linear(x, self.qkv_proj), self.q_norm, self.k_norm, self.eps, b, lc.k, lc.v, self.nq)
        o = M.chunk_attention(q, lc.k, lc.v, b, self.scale, self.softcap, self.dist_r1, self.dist_r2, self.chunk)
        return M.linear(o.view(x.shape[0], -1), self.o_proj)

    @staticmethod
    def checkpoint_names(p, m, h):
        rq, rk, rv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        return {p + "qkv_proj": [(h + "q", (0, rq), None), (h + "k", (rq, rq + rk), None), (h + "v", (rq + rk, rq + rk + rv), None)],
                p + "q_norm": [(h + "q.norm", None, None)], p + "k_norm": [(h + "k.norm", None, None)],
                p + "dist_r1": [(h + "r1", None, None)], p + "dist_r2": [(h + "r2", None, None)], p + "o_proj": [(h + "o", None, None)]}


class RGLRU(_Block):
    @staticmethod
    def check(m, where):
        _need(m["width"] % m["blocks"] == 0, where, f"{m['blocks']} blocks do not divide {m['width']}")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        H, W, n = cfg.hidden_size, m["width"], m["blocks"]
        self.W, self.taps = W, m["conv"]
        self.yx_proj, self.yx_bias = self.mat(2 * W, H), self.vec(2 * W)
        self.conv_w, self.conv_b = self.vec(W, self.taps), self.vec(W)
        self.gate_w, self.gate_b = self.mat(2, n, W // n, W // n), self.vec(2, n, W // n)      # r, then i
        self.lam = self.vec(W)
        self.o_proj = self.mat(H, W)

    def cache_shapes(self):
        return {"tail": (self.W, self.taps - 1), "state": (self.W,)}

    def forward(self, x, b, lc):
        yx, W = M.linear(x, self.yx_proj), self.W
        u = M.causal_conv(yx[:, W:], self.yx_bias[W:], self.conv_w, self.conv_b, False, b, lc.tail)
        h = M.rglru(u, yx[:, :W], self.yx_bias[:W], self.gate_w, self.gate_b, self.lam, b, lc.state)
        return M.linear(h, self.o_proj)

    @staticmethod
    def checkpoint_names(p, m, h):
        W = m["width"]
        return {p + "yx_proj": [(h + "y", (0, W), None), (h + "x", (W, 2 * W), None)],
                p + "yx_bias": [(h + "y.b", (0, W), None), (h + "x.b", (W, 2 * W), None)],
                p + "conv_w": [(h + "conv", None, None)], p + "conv_b": [(h + "conv.b", None, None)],
                p + "gate_w": [(h + "ra", None, 0), (h + "ri", None, 1)], p + "gate_b": [(h + "ra.b", None, 0), (h + "ri.b", None, 1)],
                p + "lam": [(h + "lam", None, None)], p + "o_proj": [(h + "o", None, None)]}


class Mamba2(_Block):
    @staticmethod
    def check(m, where):
        _need(m["heads"] % m["groups"] == 0 and (m["heads"] * m["vdim"]) % m["norm_groups"] == 0, where,
              "groups do not divide the heads or the norm groups the channels")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        H = cfg.hidden_size
        self.heads, self.vdim, self.N, self.G = m["heads"], m["vdim"], m["state"], m["groups"]
        self.norm_groups, self.taps = m["norm_groups"], m["conv"]
        self.inner = self.heads * self.vdim
        self.conv_dim = self.inner + 2 * self.G * self.N
        self.in_proj = self.mat(self.inner + self.conv_dim + self.heads, H)
        self.conv_w, self.conv_b = self.vec(self.conv_dim, self.taps), self.vec(self.conv_dim)
        self.dt_bias, self.A_log, self.D = self.vec(self.heads), self.vec(self.heads), self.vec(self.heads)
        self.norm = self.vec(self.inner)
        self.o_proj = self.mat(H, self.inner)

    def cache_shapes(self):
        return {"tail": (self.conv_dim, self.taps - 1), "state": (self.heads, self.vdim, self.N)}

    def forward(self, x, b, lc):
        zxd, I, C = M.linear(x, self.in_proj), self.inner, self.conv_dim
        xbc = M.causal_conv(zxd[:, I:I + C], None, self.conv_w, self.conv_b, True, b, lc.tail)
        y = M.mamba2_scan(xbc, zxd[:, I + C:], self.dt_bias, self.A_log, self.D, self.heads, self.vdim, self.N, self.G, b, lc.state)
        return M.linear(M.gated_group_norm(y, zxd[:, :I], self.norm, self.norm_groups, self.eps), self.o_proj)

    @staticmethod
    def checkpoint_names(p, m, h):
        return {p + native: [(h + name, None, None)] for native, name in
                (("in_proj", "in"), ("conv_w", "conv"), ("conv_b", "conv.b"), ("dt_bias", "dt_bias"), ("A_log", "A_log"), ("D", "D"),
                 ("norm", "norm"), ("o_proj", "o"))}


class LatentAttention(_Block):
    """Attention whose cache row is one normed latent per token. Heads read it through ``ukv_proj``: for single tokens the
    key part is applied to the queries and the value part to the outputs (all heads then share the latent as key and value),
    for portions the keys and values of the visible tokens are worked out once."""

    lists_pages = True

    @staticmethod
    def check(m, where):
        _need(min(m[k] for k in ("heads", "dim", "vdim", "q_rank", "kv_rank")) >= 1, where, "a latent attention needs positive sizes")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        H = cfg.hidden_size
        self.nq, self.D, self.Dv, self.q_rank, self.kv_rank = m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"]
        self.scale, self.window = float(m["scale"]), int((m.get("mask") or {}).get("size") or 0)
        self.down_proj = self.mat(self.q_rank + self.kv_rank, H)                 # query latent, then the cached one
        self.q_norm, self.kv_norm = self.vec(self.q_rank), self.vec(self.kv_rank)
        self.uq_proj = self.mat(self.nq * self.D, self.q_rank)
        self.ukv_proj = self.mat(self.nq * (self.D + self.Dv), self.kv_rank)     # keys of all heads, then values
        self.o_proj = self.mat(H, self.nq * self.Dv)

    def cache_shapes(self):
        return {"kv": ((1, self.kv_rank), None)}

    def first_visible(self, pos: int) -> int:
        return max(0, pos - self.window + 1) if self.window else 0

    @property
    def span(self) -> int:
        return self.window

    def forward(self, x, b, lc):
        cq = M.latent_norm_append(M.linear(x, self.down_proj), self.q_norm, self.kv_norm, self.eps, b, lc.k)
        q = M.linear(cq, self.uq_proj).view(x.shape[0], self.nq, self.D)
        o = M.latent_attention(q, lc.k, self.ukv_proj, self.Dv, b, self.scale, self.window)
        return M.linear(o.view(x.shape[0], -1), self.o_proj)

    @staticmethod
    def checkpoint_names(p, m, h):
        rq, rc, nk, nv = m["q_rank"], m["kv_rank"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
        return {p + "down_proj": [(h + "dq", (0, rq), None), (h + "dkv", (rq, rq + rc), None)],
                p + "q_norm": [(h + "dq.norm", None, None)], p + "kv_norm": [(h + "dkv.norm", None, None)], p + "uq_proj": [(h + "uq", None, None)],
                p + "ukv_proj": [(h + "uk", (0, nk), None), (h + "uv", (nk, nk + nv), None)], p + "o_proj": [(h + "o", None, None)]}


class RotaryLatentAttention(_Block):
    """Latent attention with positions: queries come straight from the layer's input as [unrotated, rotated] heads, and the
    cache row is the normed latent followed by one rotated key part that all heads share. Rotation of neighbouring pairs,
    YaRN frequencies; a learned sink and a sigmoid gate per head. Sees everything before it."""

    @staticmethod
    def check(m, where):
        _need(min(m[k] for k in ("heads", "dim", "vdim", "kv_rank")) >= 1 and m["rot_dim"] >= 2, where, "a latent attention needs positive sizes")
        _need(m["rot"]["dims"] == m["rot_dim"] and m["rot_dim"] % 2 == 0, where, "the rotated part turns as a whole, in pairs")

    span = 0
    lists_pages = True

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        H = cfg.hidden_size
        self.nq, self.D, self.Dv, self.kv_rank, self.rot_dim = m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["rot_dim"]
        self.scale, self.rotary = float(m["scale"]), yarn_frequencies(m["rot"])
        self.q_rows = self.nq * (self.D + self.rot_dim)
        self.gate_at = self.q_rows + self.kv_rank + self.rot_dim
        self.in_proj = self.mat(self.gate_at + self.nq, H)                       # queries, latent, shared key part, gate
        self.kv_norm, self.sink = self.vec(self.kv_rank), self.vec(self.nq)
        self.ukv_proj = self.mat(self.nq * (self.D + self.Dv), self.kv_rank)
        self.o_proj = self.mat(H, self.nq * self.Dv)

    def cache_shapes(self):
        return {"kv": ((1, self.kv_rank + self.rot_dim), None)}

    def first_visible(self, pos: int) -> int:
        return 0

    def forward(self, x, b, lc):
        R, z = x.shape[0], M.linear(x, self.in_proj)
        M.latent_rope_append(z, self.kv_norm, self.eps, self.rot(b), True, b, lc.k, self.nq, self.D)
        q = z[:, :self.q_rows].unflatten(1, (self.nq, self.D + self.rot_dim))
        o = M.latent_attention(q, lc.k, self.ukv_proj, self.Dv, b, self.scale, 0, self.rot_dim, self.sink, z[:, self.gate_at:])
        return M.linear(o.view(R, -1), self.o_proj)

    @staticmethod
    def checkpoint_names(p, m, h):
        rq, rd, nk, nv = m["heads"] * (m["dim"] + m["rot_dim"]), m["kv_rank"] + m["rot_dim"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
        return {p + "in_proj": [(h + "q", (0, rq), None), (h + "dkv", (rq, rq + rd), None), (h + "g", (rq + rd, rq + rd + m["heads"]), None)],
                p + "kv_norm": [(h + "dkv.norm", None, None)], p + "sink": [(h + "sink", None, None)],
                p + "ukv_proj": [(h + "uk", (0, nk), None), (h + "uv", (nk, nk + nv), None)], p + "o_proj": [(h + "o", None, None)]}


ONE_IN_DENOMINATOR = 0.0       # sink whose exponential is the 1 that a softmax's denominator gets


class RotaryAttention(_Block):
    """Grouped-query attention that sees everything before it. q and k are rotated (neighbouring numbers paired, frequencies
    scaled by wavelength) and brought to a root mean square of one, scores are multiplied by a learned number per head, the
    softmax has one more in its denominator."""

    span = 0

    @staticmethod
    def check(m, where):
        _check_heads(m, where)
        _need(2 <= m["rot"]["dims"] <= m["dim"] and m["rot"]["dims"] % 2 == 0, where, "rotated numbers come in pairs within a head")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        H = cfg.hidden_size
        self.nq, self.nkv, self.D, self.Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.scale, self.rotary = float(m["scale"]), llama3_frequencies(m["rot"])
        self.qkv_proj = self.mat((self.nq + self.nkv) * self.D + self.nkv * self.Dv, H)
        self.temp = self.vec(self.nq)
        self.o_proj = self.mat(H, self.nq * self.Dv)

    def cache_shapes(self):
        return {"kv": ((self.nkv, self.D), (self.nkv, self.Dv))}

    def first_visible(self, pos: int) -> int:
        return 0

    def forward(self, x, b, lc):
        q = M.qk_head_norm_append(M.linear(x, self.qkv_proj), None, None, self.eps, self.rot(b), True, b, lc.k, lc.v, self.nq, unit=True, q_factor=self.temp)
        o = M.chunk_attention(q, lc.k, lc.v, b, self.scale, sink=ONE_IN_DENOMINATOR)
        return M.linear(o.view(x.shape[0], -1), self.o_proj)

    @staticmethod
    def checkpoint_names(p, m, h):
        rq, rk, rv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        return {p + "qkv_proj": [(h + "q", (0, rq), None), (h + "k", (rq, rq + rk), None), (h + "v", (rq + rk, rq + rk + rv), None)],
                p + "temp": [(h + "temp", None, None)], p + "o_proj": [(h + "o", None, None)]}


# ----------------------------------------------------------------------------- branches side by side
class WindowBranch(_Block):
    """Grouped-query attention in a sliding window: per-head norms and rotation (halves paired) on q and k, capped scores, one
    added to the softmax's denominator, a gate per output channel. Works on its rows q | k | v | g of a fused projection."""

    parts = ("q", "k", "v", "g")

    @staticmethod
    def check(m, where):
        _check_heads(m, where)
        _need(m["rot"]["dims"] % 2 == 0 and m["rot"]["dims"] <= m["dim"], where, "rotated numbers come in pairs within a head")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        self.nq, self.nkv, self.D, self.Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        self.scale, self.softcap, self.window = float(m["scale"]), float(m.get("softcap") or 0.0), int((m.get("mask") or {}).get("size") or 0)
        self.rotary = rotary_frequencies(m["rot"])
        self.q_norm, self.k_norm = self.vec(self.D), self.vec(self.D)

    @staticmethod
    def rows(m):
        return m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]

    @staticmethod
    def columns(m):
        return m["heads"] * m["vdim"]

    def cache_shapes(self):
        return {"kv": ((self.nkv, self.D), (self.nkv, self.Dv))}

    def forward(self, z, b, lc, factor, out):
        q = M.qk_head_norm_append(z, self.q_norm, self.k_norm, self.eps, self.rot(b), False, b, lc.k, lc.v, self.nq)
        gate = z[:, self.nq * self.D + self.nkv * (self.D + self.Dv):][:, :self.nq * self.Dv]
        M.chunk_attention(q, lc.k, lc.v, b, self.scale, self.softcap, window=self.window, sink=ONE_IN_DENOMINATOR, gate=gate, out_scale=factor, out=out)

    @staticmethod
    def own_names(p, m, h):
        return {p + "q_norm": [(h + "q.norm", None, None)], p + "k_norm": [(h + "k.norm", None, None)]}


class RetentionBranch(_Block):
    """Linear attention with a fixed decay per head and no denominator: rotated q and k (halves paired), every head's output
    over its root mean square, gated. Works on its rows q | k | v | g of a fused projection."""

    parts = ("q", "k", "v", "g")

    @staticmethod
    def check(m, where):
        _need(min(m[k] for k in ("heads", "dim", "vdim")) >= 1 and len(m["decay"]) == m["heads"], where, f"{len(m['decay'])} decays for {m['heads']} heads")
        _need(m["rot"]["dims"] % 2 == 0 and m["rot"]["dims"] <= m["dim"] <= 512, where, "rotated numbers come in pairs within a head of up to 512")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        self.heads, self.D, self.Dv = m["heads"], m["dim"], m["vdim"]
        self.rotary = rotary_frequencies(m["rot"])
        self.register_buffer("decay", self.const(m["decay"]), persistent=False)
        self.register_buffer("log2_decay", self.const([max(math.log2(a), -1e4) if a > 0 else -1e4 for a in m["decay"]]), persistent=False)

    @staticmethod
    def rows(m):
        return m["heads"] * m["dim"], m["heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"] * m["vdim"]

    @staticmethod
    def columns(m):
        return m["heads"] * m["vdim"]

    def cache_shapes(self):
        return {"state": (self.heads, self.Dv, self.D)}

    def forward(self, z, b, lc, factor, out):
        M.retention(z, self.decay, self.log2_decay, self.rot(b), self.eps, factor, out, self.heads, self.D, self.Dv, b, lc.state)

    @staticmethod
    def own_names(p, m, h):
        return {}


class KeyValueBranch(_Block):
    """Grouped-query attention without positions that sees everything before it; its keys, as projected, are its values, while q and
    k meet with a root mean square of one. The cache holds the projected keys once, and the number that norms each of them. Works
    on its rows q | k of a fused projection."""

    parts = ("q", "k")

    @staticmethod
    def check(m, where):
        _check_heads(m, where)
        _need(m["dim"] == m["vdim"], where, f"keys of {m['dim']} numbers cannot be values of {m['vdim']}")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        self.nq, self.nkv, self.D, self.scale = m["heads"], m["kv_heads"], m["dim"], float(m["scale"])

    @staticmethod
    def rows(m):
        return m["heads"] * m["dim"], m["kv_heads"] * m["dim"]

    @staticmethod
    def columns(m):
        return m["heads"] * m["dim"]

    def cache_shapes(self):
        return {"kv": ((self.nkv, self.D), None), "key_factor": (self.nkv,)}

    def forward(self, z, b, lc):
        q = M.qk_head_norm_append(z, None, None, self.eps, None, False, b, lc.k, None, self.nq, unit=True, key_factor=lc.key_factor)
        return M.chunk_attention(q, lc.k, None, b, self.scale, key_factor=lc.key_factor).view(z.shape[0], -1)

    @staticmethod
    def own_names(p, m, h):
        return {}


class MinGRUBranch(_Block):
    """Element-wise recurrence with gates made from the token alone, not from the state. Works on its rows z | x | g of a fused projection."""

    parts = ("z", "x", "g")

    @staticmethod
    def check(m, where):
        _need(m["width"] >= 1, where, "a recurrence needs a width")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        self.W = m["width"]
        self.zx_bias = self.vec(2 * self.W)

    @staticmethod
    def rows(m):
        return (m["width"],) * 3

    @staticmethod
    def columns(m):
        return m["width"]

    def cache_shapes(self):
        return {"state": (self.W,)}

    def forward(self, z, b, lc):
        return M.min_gru(z, self.zx_bias, b, lc.state)

    @staticmethod
    def own_names(p, m, h):
        W = m["width"]
        return {p + "zx_bias": [(h + "z.b", (0, W), None), (h + "x.b", (W, 2 * W), None)]}


class Parallel(_Block):
    """Windowed attention and retention on the same input, their outputs weighted and added: one product makes the rows of
    both, one takes their outputs, which lie side by side, to the layer's width."""

    BRANCHES = (("left", WindowBranch), ("right", RetentionBranch))

    @classmethod
    def check(cls, m, where):
        for n, branch in cls.BRANCHES:
            branch.check(m[n], f"{where}{n}: ")

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        H = cfg.hidden_size
        self.factors = [float(m[n + "_scale"]) for n, _ in self.BRANCHES]
        self.in_rows, self.out_cols = self._layout(m)
        self.in_proj, self.o_proj = self.mat(self.in_rows[-1], H), self.mat(H, self.out_cols[-1])
        self.branches = nn.ModuleList([branch(cfg, m[n], dtype, device) for n, branch in self.BRANCHES])
        self.window = self.branches[0].window

    @classmethod
    def _layout(cls, m):
        """First row of every branch in the input projection and first column in the output projection, and their ends."""
        rows, cols = [0], [0]
        for n, branch in cls.BRANCHES:
            rows.append(rows[-1] + sum(branch.rows(m[n])))
            cols.append(cols[-1] + branch.columns(m[n]))
        return rows, cols

    def cache_shapes(self):
        out = {}
        for br in self.branches:
            out.update(br.cache_shapes())
        return out

    def first_visible(self, pos: int) -> int:
        return max(0, pos - self.window + 1) if self.window else 0

    @property
    def span(self) -> int:
        return self.window

    def forward(self, x, b, lc):
        z = M.linear(x, self.in_proj)
        o = torch.empty(x.shape[0], self.out_cols[-1], device=x.device, dtype=x.dtype)
        for i, br in enumerate(self.branches):
            br(z[:, self.in_rows[i]:self.in_rows[i + 1]], b, lc, self.factors[i], o[:, self.out_cols[i]:self.out_cols[i + 1]])
        return M.linear(o, self.o_proj)

    @classmethod
    def checkpoint_names(cls, p, m, h):
        rows, cols = cls._layout(m)
        out = {p + "in_proj": [], p + "o_proj": []}
        for i, (n, branch) in enumerate(cls.BRANCHES):
            at, hb = rows[i], f"{h}{n}."
            for part, r in zip(branch.parts, branch.rows(m[n])):
                out[p + "in_proj"].append((hb + part, (at, at + r), None))
                at += r
            out[p + "o_proj"].append((hb + "o", None, (slice(None), slice(cols[i], cols[i + 1]))))
            out.update(branch.own_names(f"{p}branches.{i}.", m[n], hb))
        return out


class NormedParallel(Parallel):
    """Attention whose keys are its values beside minGRU: one product makes the rows of both, each has an output projection of its
    own, and half the sum of the two outputs, each normed over the layer's width, is left to the residual sum behind the mixer."""

    BRANCHES = (("left", KeyValueBranch), ("right", MinGRUBranch))
    FACTOR = 0.5

    def __init__(self, cfg, m, dtype, device):
        _Block.__init__(self, cfg, dtype, device)
        H = cfg.hidden_size
        self.in_rows, self.out_cols = self._layout(m)
        self.in_proj = self.mat(self.in_rows[-1], H)
        self.o_proj = nn.ParameterList([self.mat(H, branch.columns(m[n])) for n, branch in self.BRANCHES])
        self.left_norm, self.right_norm = self.vec(H), self.vec(H)
        self.branches = nn.ModuleList([branch(cfg, m[n], dtype, device) for n, branch in self.BRANCHES])
        self.window = 0

    def forward(self, x, b, lc):
        z = M.linear(x, self.in_proj)
        left, right = (M.linear(br(z[:, self.in_rows[i]:self.in_rows[i + 1]], b, lc), self.o_proj[i]) for i, br in enumerate(self.branches))
        return M.BranchSum(left, right, self.left_norm, self.right_norm, self.FACTOR, self.eps)

    @classmethod
    def checkpoint_names(cls, p, m, h):
        out = super().checkpoint_names(p, m, h)
        del out[p + "o_proj"]
        for i, (n, _) in enumerate(cls.BRANCHES):
            out[f"{p}o_proj.{i}"] = [(f"{h}{n}.o", None, None)]
            out[f"{p}{n}_norm"] = [(f"{h}{n}.out", None, None)]
        return out


class XieluMLP(_Block):
    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        self.up_proj, self.down_proj = self.mat(m["ff"], cfg.hidden_size), self.mat(cfg.hidden_size, m["ff"])
        self.act = self.vec(2)

    def forward(self, x):
        return M.linear(M.xielu(M.linear(x, self.up_proj), self.act), self.down_proj)

    @staticmethod
    def checkpoint_names(p, m, h):
        return {p + "up_proj": [(h + "up", None, None)], p + "down_proj": [(h + "down", None, None)], p + "act": [(h + "act", None, None)]}


class RoutedMLP(_Block):
    """Top-k experts: 32-bit softmax scores choose with a correction added, and weigh without it."""

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        E, I, H = m["router"]["experts"], m["expert"]["ff"], cfg.hidden_size
        self.top = m["router"]["top"]
        self.router, self.correction = self.mat(E, H), self.vec(E)
        self.w_gate_up, self.w_down = self.mat(E, 2 * I, H), self.mat(E, H, I)

    def forward(self, x):
        rt = OF.moe_route(M.router_logits(x, self.router), self.top, bias=self.correction, norm=False, want_probs=False, want_host=False)
        h = M.expert_linear(x.index_select(0, rt.token_of), self.w_gate_up, rt)
        return M.expert_combine(M.expert_linear(M.glu_silu(h), self.w_down, rt), rt, rt.topw)

    @staticmethod
    def checkpoint_names(p, m, h):
        E, I = m["router"]["experts"], m["expert"]["ff"]
        return {p + "router": [(h + "router", None, None)], p + "correction": [(h + "correction", None, None)],
                p + "w_gate_up": [(h + f"e{e}.{n}", r, e) for e in range(E) for n, r in (("gate", (0, I)), ("up", (I, 2 * I)))],
                p + "w_down": [(h + f"e{e}.down", None, e) for e in range(E)]}


class GeluMLP(_Block):
    """Dense feed-forward with the exact (erf) GELU."""

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        self.up_proj, self.down_proj = self.mat(m["ff"], cfg.hidden_size), self.mat(cfg.hidden_size, m["ff"])

    def forward(self, x):
        return M.linear(M.gelu_erf(M.linear(x, self.up_proj)), self.down_proj)

    @staticmethod
    def checkpoint_names(p, m, h):
        return {p + "up_proj": [(h + "up", None, None)], p + "down_proj": [(h + "down", None, None)]}


GLU_ALPHA = 1.702        # slope of the clamped units' gate


class ClampedMLP(_Block):
    """Dense feed-forward of clamped gated units."""

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        self.limit = float(m["limit"])
        self.gate_up_proj, self.down_proj = self.mat(2 * m["ff"], cfg.hidden_size), self.mat(cfg.hidden_size, m["ff"])

    def forward(self, x):
        return M.linear(M.glu_clamped(M.linear(x, self.gate_up_proj), self.limit, GLU_ALPHA), self.down_proj)

    @staticmethod
    def checkpoint_names(p, m, h):
        I = m["ff"]
        return {p + "gate_up_proj": [(h + "gate", (0, I), None), (h + "up", (I, 2 * I), None)], p + "down_proj": [(h + "down", None, None)]}


class InputWeightedMLP(_Block):
    """Top-k experts of clamped gated units. Sigmoid scores choose, and multiply each chosen expert's input as they are;
    an expert that every token visits, with sizes and a limit of its own, may stand beside them."""

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        E, I, H = m["router"]["experts"], m["expert"]["ff"], cfg.hidden_size
        self.top, self.limit = m["router"]["top"], float(m["expert"]["limit"])
        self.router = self.mat(E, H)
        self.w_gate_up, self.w_down = self.mat(E, 2 * I, H), self.mat(E, H, I)
        sh = m.get("shared")
        self.shared_limit = float(sh["limit"]) if sh else None
        if sh:
            self.shared_gate_up, self.shared_down = self.mat(2 * sh["ff"], H), self.mat(H, sh["ff"])

    def forward(self, x):
        rt = OF.moe_route(M.router_logits(x, self.router), self.top, sigmoid=True, norm=False, want_probs=False, want_host=False)
        # gate and up are linear: the weight of the input is applied to their outputs, where it costs no rounding
        h = M.glu_clamped(M.expert_linear(x.index_select(0, rt.token_of), self.w_gate_up, rt), self.limit, GLU_ALPHA, rt)
        y = M.expert_linear(h, self.w_down, rt)
        shared = None
        if self.shared_limit is not None:
            shared = M.linear(M.glu_clamped(M.linear(x, self.shared_gate_up), self.shared_limit, GLU_ALPHA), self.shared_down)
        return M.ExpertSum(y, rt, shared)

    @staticmethod
    def checkpoint_names(p, m, h):
        E, I = m["router"]["experts"], m["expert"]["ff"]
        out = {p + "router": [(h + "router", None, None)],
               p + "w_gate_up": [(h + f"e{e}.{n}", r, e) for e in range(E) for n, r in (("gate", (0, I)), ("up", (I, 2 * I)))],
               p + "w_down": [(h + f"e{e}.down", None, e) for e in range(E)]}
        if m.get("shared"):
            I = m["shared"]["ff"]
            out[p + "shared_gate_up"] = [(h + "shared.gate", (0, I), None), (h + "shared.up", (I, 2 * I), None)]
            out[p + "shared_down"] = [(h + "shared.down", None, None)]
        return out


class SharedExpertMLP(_Block):
    """Top-k experts of gated units: softmax scores choose, and the chosen ones, renormalised, weigh the experts' outputs. An
    expert that every token visits may stand beside them, behind a sigmoid gate of one number per token whose logit is made
    with the router's."""

    def __init__(self, cfg, m, dtype, device):
        super().__init__(cfg, dtype, device)
        E, I, H = m["router"]["experts"], m["expert"]["ff"], cfg.hidden_size
        self.experts, self.top = E, m["router"]["top"]
        sh = m.get("shared")
        self.router = self.mat(-(-(E + 1) // 8) * 8 if sh else E, H)             # experts, the shared one's gate, rows without a use
        self.w_gate_up, self.w_down = self.mat(E, 2 * I, H), self.mat(E, H, I)
        self.shared = bool(sh)
        if sh:
            self.shared_gate_up, self.shared_down = self.mat(2 * sh["ff"], H), self.mat(H, sh["ff"])

    def forward(self, x):
        z = M.router_logits(x, self.router)
        rt = OF.moe_route(z[:, :self.experts], self.top, norm=True, want_probs=False, want_host=False)
        y = M.expert_linear(M.glu_silu(M.expert_linear(x.index_select(0, rt.token_of), self.w_gate_up, rt)), self.w_down, rt)
        if not self.shared:
            return M.ExpertSum(y, rt, None, rt.topw)
        return M.ExpertSum(y, rt, M.linear(M.glu_silu(M.linear(x, self.shared_gate_up)), self.shared_down), rt.topw, z[:, self.experts])

    @staticmethod
    def checkpoint_names(p, m, h):
        E, I = m["router"]["experts"], m["expert"]["ff"]
        out = {p + "router": [(h + "router", (0, E), None)] + ([(h + "shared.sg", (E, E + 1), None)] if m.get("shared") else []),
               p + "w_gate_up": [(h + f"e{e}.{n}", r, e) for e in range(E) for n, r in (("gate", (0, I)), ("up", (I, 2 * I)))],
               p + "w_down": [(h + f"e{e}.down", None, e) for e in range(E)]}
        if m.get("shared"):
            I = m["shared"]["ff"]
            out[p + "shared_gate_up"] = [(h + "shared.gate", (0, I), None), (h + "shared.up", (I, 2 * I), None)]
            out[p + "shared_down"] = [(h + "shared.down", None, None)]
        return out


@dataclass(frozen=True)
class Design:
    """What tells one kind of mixer stack from another, apart from the constants of its configuration."""

    name: str                    # ``architecture`` in config.json
    mixers: dict                 # mixer kinds
    mlps: dict                   # feed-forward kinds
    layer_norms: tuple           # norms of a layer with a feed-forward ...
    layer_norms_bare: tuple      # ... and of one without
    kernels: tuple               # sources of its own kernels (beside those of every stack)


EXPERTS = ("gemm_grouped", "router")         # kernel sources of routed feed-forwards (and of products per head)

DESIGNS = {
    "kagolix": Design("Kagolix", {"attention": ChunkAttention, "rglru": RGLRU, "mamba2": Mamba2}, {"dense": XieluMLP, "moe": RoutedMLP}, ("norm1", "norm1b", "norm2", "norm2b"),
                      ("norm1", "norm1b"), ("mixer_attention", "mixer_scan", "mixer_ssd", *EXPERTS)),
    "vogilix": Design("Vogilix", {"latent_attention": LatentAttention}, {"dense": GeluMLP, "moe": InputWeightedMLP}, ("norm1", "norm2"), ("norm1",),
                      ("mixer_attention", "mixer_latent", *EXPERTS)),
    "bumotar": Design("Bumotar", {"latent_attention": RotaryLatentAttention, "parallel": Parallel}, {"moe": SharedExpertMLP}, ("norm1", "norm2"), ("norm1",),
                      ("mixer_attention", "mixer_latent", "mixer_retention", "mixer_rotary", "mixer_stream", *EXPERTS)),
    "goganex": Design("Goganex", {"attention": RotaryAttention, "parallel": NormedParallel}, {"dense": ClampedMLP}, ("norm1", "norm2"), ("norm1",),
                      ("mixer_attention", "mixer_rotary", "mixer_stream", "mixer_gru")),
}


class MixerLayer(_Block):
    def __init__(self, cfg: ModelConfig, idx: int, dtype, device):
        super().__init__(cfg, dtype, device)
        spec, H, design = cfg.mixer_layers[idx], cfg.hidden_size, DESIGNS[cfg.arch]
        for n in design.layer_norms if spec["mlp"] else design.layer_norms_bare:
            setattr(self, n, self.vec(H))
        self.mix = design.mixers[spec["type"]](cfg, spec["mixer"], dtype, device)
        self.mlp = design.mlps[spec["mlp"]["kind"]](cfg, spec["mlp"], dtype, device) if spec["mlp"] else None
        self.shift = None
        if cfg.token_shift:
            self.shift = self.vec(H)
            self.mix.carried = {"shift": (H,)}
        self.side_dim = cfg.token_side_dim
        if self.side_dim:
            self.side_col = idx * self.side_dim
            self.side_gate, self.side_proj, self.side_norm = self.mat(self.side_dim, H), self.mat(H, self.side_dim), self.vec(H)

    def side(self, x, tokens, table):
        """The layer's gated input from its part of the tokens' rows in ``table``."""
        return M.linear(M.side_gate(M.linear(x, self.side_gate), tokens, table, self.side_col), self.side_proj)


def checkpoint_plan(cfg: ModelConfig) -> dict:
    """Native parameter name -> [(checkpoint name, row range, index)], as in :mod:`.hf_io`."""
    design = DESIGNS[cfg.arch]
    plan = {"embed_tokens": [("embed", None, None)], "norm": [("final.norm", None, None)], "lm_head": [("head", None, None)]}
    if cfg.learned_positions:
        plan["embed_positions"] = [("pos", None, None)]
    if cfg.token_side_dim:
        plan["embed_side"] = [("side.embed", None, None)]
    if cfg.layer_loop and cfg.loop_mixes_embedding:
        plan["loop_in"], plan["loop_step"] = [("loop.in", None, None)], [("loop.step", None, None)]
    for i, e in enumerate(cfg.mixer_layers):
        p, h = f"layers.{i}.", f"l{i}."
        for n in design.layer_norms if e["mlp"] else design.layer_norms_bare:
            plan[p + n] = [(h + n, None, None)]
        if cfg.token_shift:
            plan[p + "shift"] = [(h + "shift", None, None)]
        plan.update(design.mixers[e["type"]].checkpoint_names(p + "mix.", e["mixer"], h + "mix."))
        if e["mlp"]:
            plan.update(design.mlps[e["mlp"]["kind"]].checkpoint_names(p + "mlp.", e["mlp"], h + "mlp."))
        if cfg.token_side_dim:
            for n in ("gate", "proj", "norm"):
                plan[p + "side_" + n] = [(h + "side." + n, None, None)]
    return plan


class MixerStackLM(CausalLM):
    """A :class:`CausalLM` of :class:`MixerLayer`: same embedding / head / loading / weight-update surface, forward by steps."""

    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu", init_std: float = 0.02, seed=None):
        if cfg.is_critic:
            raise NotImplementedError("mixer stacks have no value head")
        super().__init__(cfg, dtype, device, init_std, seed)

    @torch.no_grad()
    def reset_parameters(self, std: float = 0.02, seed=None):
        cfg = self.cfg
        self.norm = nn.Parameter(self.norm.data.float())          # used in 32 bits, like every norm weight
        like = dict(dtype=self.dtype, device=self.embed_tokens.device)
        if cfg.learned_positions:
            self.embed_positions = nn.Parameter(torch.empty(cfg.max_position_embeddings, cfg.hidden_size, **like))
        if cfg.token_side_dim:
            self.embed_side = nn.Parameter(torch.empty(cfg.vocab_size, cfg.num_layers * cfg.token_side_dim, **like))
        if cfg.layer_loop and cfg.loop_mixes_embedding:
            self.loop_in = nn.Parameter(torch.empty(cfg.hidden_size, 2 * cfg.hidden_size, **like))
            self.loop_step = nn.Parameter(torch.empty(cfg.layer_loop["times"], cfg.hidden_size, **dict(like, dtype=torch.float32)))
        self._place_rotations()
        if self.embed_tokens.device.type == "meta":
            return
        super().reset_parameters(std, seed)
        gen = torch.Generator(device=self.embed_tokens.device)
        gen.manual_seed(0 if seed is None else seed + 1)

        def uniform(p, lo, hi):
            p.copy_(torch.rand(p.shape, device=p.device, dtype=torch.float32, generator=gen) * (hi - lo) + lo)

        for name, p in self.named_parameters():
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("norm", "norm1", "norm1b", "norm2", "norm2b") and "mix." not in name:
                p.fill_(0.0 if cfg.rms_norm_offset else 1.0)
            elif leaf in ("D", "temp"):
                p.fill_(1.0)
            elif leaf == "shift":
                uniform(p, 0.0, 1.0)
            elif leaf in ("correction", "conv_b", "yx_bias", "gate_b"):
                p.zero_()
            elif leaf == "conv_w":
                uniform(p, -p.shape[1] ** -0.5, p.shape[1] ** -0.5)
            elif leaf == "A_log":
                uniform(p, 0.0, 2.7)
            elif leaf == "dt_bias":
                uniform(p, -6.0, -2.0)
            elif leaf == "lam":
                uniform(p, -5.0, -1.0)
            elif leaf in ("dist_r1", "dist_r2"):
                uniform(p, 0.1, 1.0)
            elif leaf == "act":
                p.fill_(0.5)

    def _place_rotations(self):
        """Every block that rotates gets its columns in the step's table of angles; equal rotations share theirs."""
        at, freqs, mults = {}, [], []
        for mod in self.modules():
            if isinstance(mod, _Block) and mod.rotary is not None:
                if mod.rotary not in at:
                    at[mod.rotary] = len(freqs)
                    freqs += mod.rotary[0]
                    mults += [mod.rotary[1]] * len(mod.rotary[0])
                mod.rot_at = at[mod.rotary]
        if freqs:
            dev = self.embed_tokens.device
            self.register_buffer("rot_freq", torch.tensor([f / (2.0 * math.pi) for f in freqs], dtype=torch.float64, device=dev), persistent=False)
            self.register_buffer("rot_mult", torch.tensor(mults, dtype=torch.float32, device=dev), persistent=False)

    @property
    def layer_runs(self) -> list[int]:
        """The layers in the order in which they run; looped ones once per pass."""
        n, loop = self.cfg.num_layers, self.cfg.layer_loop
        if not loop:
            return list(range(n))
        a, z = loop["start"], loop["stop"]
        return list(range(a)) + list(range(a, z)) * loop["times"] + list(range(z, n))

    def cache_mixers(self) -> list:
        """The mixer of every layer run: each has its own pages and states."""
        return [self.layers[i].mix for i in self.layer_runs]

    def forward_step(self, b: M.RaggedBatch, cache, on_layer=None) -> torch.Tensor:
        """Final normed hidden rows [R, H] of one step; reads and advances ``cache``. ``on_layer(i, resid)`` sees the
        32-bit residual stream after everything the i-th layer run adds to it."""
        return {"post": self._step_post, "pre": self._step_pre, "sandwich": self._step_sandwich}[self.cfg.norm_placement](b, cache, on_layer)

    def _step_sandwich(self, b, cache, on_layer):
        cfg, layers = self.cfg, self.layers
        g, eps = cfg.norm_groups, cfg.rms_norm_eps
        resid, x = M.embed_norm(b.tokens, self.embed_tokens, layers[0].norm1, g, eps)
        for i, layer in enumerate(layers):
            nxt = layers[i + 1].norm1 if i + 1 < len(layers) else self.norm
            h = layer.mix(x, b, cache.layers[i])
            if layer.mlp is not None:
                x = M.sandwich_norm(h, layer.norm1b, resid, layer.norm2, g, eps)
                x = M.sandwich_norm(layer.mlp(x), layer.norm2b, resid, nxt, g, eps)
            else:
                x = M.sandwich_norm(h, layer.norm1b, resid, nxt, g, eps)
            if on_layer is not None:
                on_layer(i, resid)
        return x

    def _step_post(self, b, cache, on_layer):
        cfg, last = self.cfg, len(self.layers) - 1
        eps, mult, off = cfg.rms_norm_eps, cfg.residual_mult, 1.0 if cfg.rms_norm_offset else 0.0
        resid, x = M.embed_rows(b.tokens, self.embed_tokens, b.pos, self.embed_positions if cfg.learned_positions else None)
        for i, layer in enumerate(self.layers):
            # (output of a sublayer, its norm weight, what is added to that weight), the final norm after the very last one
            parts = [(lambda: layer.mix(x, b, cache.layers[i]), layer.norm1, off)]
            if layer.mlp is not None:
                parts.append((lambda: layer.mlp(x), layer.norm2, off))
            if layer.side_dim:
                parts.append((lambda: layer.side(x, b.tokens, self.embed_side), layer.side_norm, 0.0))
            for n, (sub, w, o) in enumerate(parts):
                end = i == last and n + 1 == len(parts)
                x = M.post_norm(sub(), w, resid, eps, mult, o, self.norm if end else None, off)
            if on_layer is not None:
                on_layer(i, resid)
        return x

    def _step_pre(self, b, cache, on_layer):
        cfg, layers, runs, dt = self.cfg, self.layers, self.layer_runs, self.dtype
        eps, H = cfg.rms_norm_eps, cfg.hidden_size
        b.rot = M.rotary_table(b.pos, self.rot_freq, self.rot_mult) if hasattr(self, "rot_freq") else None
        loop = cfg.layer_loop if cfg.loop_mixes_embedding else None
        a, size, times = (loop["start"], loop["stop"] - loop["start"], loop["times"]) if loop else (0, 0, 0)
        enters = {a + t * size: t for t in range(times)}            # layer run -> pass that begins with it

        def reads(r, src, resid, vec=None):
            """The stream after ``src`` and ``vec`` were added, and what the mixer of layer run ``r`` reads of it."""
            layer = layers[runs[r]]
            return M.stream_norm(src, resid, layer.norm1, eps, dt, vec, layer.shift, b, cache.layers[r].shift)
        if loop:
            # what enters a pass: the stream beside the embedding
            both = torch.empty(b.n_rows, 2 * H, device=self.embed_tokens.device, dtype=dt)
            resid, x = M.embed_rows(b.tokens, self.embed_tokens, b.pos, None, both[:, H:], both[:, :H])
            if 0 not in enters:
                resid, x = reads(0, None, resid)
        else:
            resid, x = reads(0, M.EmbeddingRows(b.tokens, self.embed_tokens, cfg.embedding_scale), None)
        for r, i in enumerate(runs):
            layer = layers[i]
            if r in enters:
                resid, x = reads(r, None, M.linear(both, self.loop_in, fp32_out=True).contiguous(), self.loop_step[enters[r]])
            h = layer.mix(x, b, cache.layers[r])
            if layer.mlp is not None:
                h = layer.mlp(M.residual_norm(h, resid, layer.norm2, eps, dt))
            # the stream and what comes next: a pass's entrance, the next layer's norm, or the final norm (with the logits' factor)
            if r + 1 in enters:
                M.residual_norm(h, resid, None, eps, dt, out=both[:, :H])
            elif r + 1 < len(runs):
                resid, x = reads(r + 1, h, resid)
            else:
                x = M.residual_norm(h, resid, self.norm, eps, dt, mult=cfg.logit_scale)
            if on_layer is not None:
                on_layer(r, resid)
        return x

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return M.softcap_(M.linear(hidden, self.output_weight, fp32_out=True), self.cfg.logit_softcap)

    def forward_hidden(self, *a, **kw):
        raise NotImplementedError("mixer stacks run step by step on a StateCache (forward_step); they are served, not trained")
