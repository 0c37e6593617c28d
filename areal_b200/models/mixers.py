"""Mixer stacks: decoder models whose layers are listed one by one, each with its own token mixer and feed-forward.

Two designs are built from the parts below (:data:`DESIGNS`):

* Kagolix normalises twice around every sublayer, in groups: ``x += norm_b(f(norm_a(x)))``; its output is capped;
* Vogilix normalises the sublayer's output only, ``x += m * norm(f(x))``, adds a learned vector per position to the
  embedding, and ends every layer with a gated input from the layer's own part of a per-token row.

The sum x stays in 32 bits in both. The mixers

* ``attention``: grouped-query attention inside chunks of positions, whole-projection RMS norms on q and k, no rotation,
  capped scores and a logarithmic distance bias (two numbers per head);
* ``rglru``: a gated branch times a real-gated linear recurrence behind a short causal convolution;
* ``mamba2``: the scalar-decay state-space recurrence, gated and normalised in groups;
* ``latent_attention``: keys and values of all heads from one normed latent per token (the only thing cached), queries from
  a latent of their own, no positions, a sliding window;

and the feed-forwards (dense with xIELU or the exact GELU; experts behind a softmax or a sigmoid router, weighted at their
output or at their input) are built from the ops of :mod:`..ops.mixer_ops`. A forward pass runs the rows of one step
(:class:`~..ops.mixer_ops.RaggedBatch`) from the pages and state slots of :class:`~..engine.state_cache.StateCache`; whole
prompts, portions and single tokens are the same call.

Matrices are stored in the model's dtype, everything that is used in 32 bits (norm weights, biases, taps, decay and bias
parameters) as fp32. Serving only: there is no backward pass.
"""
from __future__ import annotations

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
        if t not in MIXERS:
            raise ValueError(f"layer {i}: unknown mixer '{t}' (have {sorted(MIXERS)})")
        if t == "attention" and m["heads"] % m["kv_heads"]:
            raise ValueError(f"layer {i}: {m['heads']} query heads over {m['kv_heads']} key/value heads")
        if t == "rglru" and m["width"] % m["blocks"]:
            raise ValueError(f"layer {i}: {m['blocks']} blocks do not divide {m['width']}")
        if t == "mamba2" and (m["heads"] % m["groups"] or (m["heads"] * m["vdim"]) % m["norm_groups"]):
            raise ValueError(f"layer {i}: groups do not divide the heads or the norm groups the channels")
        if t == "latent_attention" and min(m[k] for k in ("heads", "dim", "vdim", "q_rank", "kv_rank")) < 1:
            raise ValueError(f"layer {i}: a latent attention needs positive sizes")
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


class ChunkAttention(_Block):
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


MIXERS = {"attention": ChunkAttention, "rglru": RGLRU, "mamba2": Mamba2, "latent_attention": LatentAttention}


@dataclass(frozen=True)
class Design:
    """What tells one kind of mixer stack from another, apart from the constants of its configuration."""

    name: str                    # ``architecture`` in config.json
    mlps: dict                   # feed-forward kinds
    layer_norms: tuple           # norms of a layer with a feed-forward ...
    layer_norms_bare: tuple      # ... and of one without


DESIGNS = {
    "kagolix": Design("Kagolix", {"dense": XieluMLP, "moe": RoutedMLP}, ("norm1", "norm1b", "norm2", "norm2b"), ("norm1", "norm1b")),
    "vogilix": Design("Vogilix", {"dense": GeluMLP, "moe": InputWeightedMLP}, ("norm1", "norm2"), ("norm1",)),
}


class MixerLayer(_Block):
    def __init__(self, cfg: ModelConfig, idx: int, dtype, device):
        super().__init__(cfg, dtype, device)
        spec, H, design = cfg.mixer_layers[idx], cfg.hidden_size, DESIGNS[cfg.arch]
        for n in design.layer_norms if spec["mlp"] else design.layer_norms_bare:
            setattr(self, n, self.vec(H))
        self.mix = MIXERS[spec["type"]](cfg, spec["mixer"], dtype, device)
        self.mlp = design.mlps[spec["mlp"]["kind"]](cfg, spec["mlp"], dtype, device) if spec["mlp"] else None
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
    for i, e in enumerate(cfg.mixer_layers):
        p, h = f"layers.{i}.", f"l{i}."
        for n in design.layer_norms if e["mlp"] else design.layer_norms_bare:
            plan[p + n] = [(h + n, None, None)]
        plan.update(MIXERS[e["type"]].checkpoint_names(p + "mix.", e["mixer"], h + "mix."))
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
            elif leaf == "D":
                p.fill_(1.0)
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

    def forward_step(self, b: M.RaggedBatch, cache, on_layer=None) -> torch.Tensor:
        """Final normed hidden rows [R, H] of one step; reads and advances ``cache``. ``on_layer(i, resid)`` sees the
        32-bit residual stream after everything a layer adds to it."""
        return (self._step_post if self.cfg.norm_placement == "post" else self._step_sandwich)(b, cache, on_layer)

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

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return M.softcap_(M.linear(hidden, self.output_weight, fp32_out=True), self.cfg.logit_softcap)

    def forward_hidden(self, *a, **kw):
        raise NotImplementedError("mixer stacks run step by step on a StateCache (forward_step); they are served, not trained")
