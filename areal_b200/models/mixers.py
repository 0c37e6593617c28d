"""Mixer stacks: decoder models whose layers are listed one by one, each with its own token mixer and feed-forward
(the Kagolix design).

Around every sublayer the stack normalises twice, in groups: ``x += norm_b(f(norm_a(x)))``; the sum x stays in 32 bits.
The mixers

* ``attention``: grouped-query attention inside chunks of positions, whole-projection RMS norms on q and k, no rotation,
  capped scores and a logarithmic distance bias (two numbers per head);
* ``rglru``: a gated branch times a real-gated linear recurrence behind a short causal convolution;
* ``mamba2``: the scalar-decay state-space recurrence, gated and normalised in groups;

and the feed-forwards (dense with xIELU, or softmax-routed experts whose choice adds a correction) are built from the ops
of :mod:`..ops.mixer_ops`. A forward pass runs the rows of one step (:class:`~..ops.mixer_ops.RaggedBatch`) from the pages
and state slots of :class:`~..engine.state_cache.StateCache`; whole prompts, portions and single tokens are the same call.

Matrices are stored in the model's dtype, everything that is used in 32 bits (norm weights, biases, taps, decay and bias
parameters) as fp32. Serving only: there is no backward pass.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ..ops import functional as OF
from ..ops import mixer_ops as M
from .config import ModelConfig
from .decoder import CausalLM


def check_layer_specs(layers: list, width: int, norm_groups: int) -> None:
    """Raises ``ValueError`` for a layer list that no kernel could run."""
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
        if mlp and mlp["kind"] not in ("dense", "moe"):
            raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")


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


MIXERS = {"attention": ChunkAttention, "rglru": RGLRU, "mamba2": Mamba2}
MLPS = {"dense": XieluMLP, "moe": RoutedMLP}


class MixerLayer(_Block):
    def __init__(self, cfg: ModelConfig, idx: int, dtype, device):
        super().__init__(cfg, dtype, device)
        spec, H = cfg.mixer_layers[idx], cfg.hidden_size
        self.norm1, self.norm1b = self.vec(H), self.vec(H)
        self.mix = MIXERS[spec["type"]](cfg, spec["mixer"], dtype, device)
        self.mlp = MLPS[spec["mlp"]["kind"]](cfg, spec["mlp"], dtype, device) if spec["mlp"] else None
        if self.mlp is not None:
            self.norm2, self.norm2b = self.vec(H), self.vec(H)


def checkpoint_plan(cfg: ModelConfig) -> dict:
    """Native parameter name -> [(checkpoint name, row range, index)], as in :mod:`.hf_io`."""
    plan = {"embed_tokens": [("embed", None, None)], "norm": [("final.norm", None, None)], "lm_head": [("head", None, None)]}
    for i, e in enumerate(cfg.mixer_layers):
        p, h = f"layers.{i}.", f"l{i}."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if e["mlp"] else ()):
            plan[p + n] = [(h + n, None, None)]
        plan.update(MIXERS[e["type"]].checkpoint_names(p + "mix.", e["mixer"], h + "mix."))
        if e["mlp"]:
            plan.update(MLPS[e["mlp"]["kind"]].checkpoint_names(p + "mlp.", e["mlp"], h + "mlp."))
    return plan


class MixerStackLM(CausalLM):
    """A :class:`CausalLM` of :class:`MixerLayer`: same embedding / head / loading / weight-update surface, forward by steps."""

    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu", init_std: float = 0.02, seed=None):
        if cfg.is_critic:
            raise NotImplementedError("mixer stacks have no value head")
        super().__init__(cfg, dtype, device, init_std, seed)

    @torch.no_grad()
    def reset_parameters(self, std: float = 0.02, seed=None):
        self.norm = nn.Parameter(self.norm.data.float())          # used in 32 bits, like every norm weight
        if self.embed_tokens.device.type == "meta":
            return
        super().reset_parameters(std, seed)
        gen = torch.Generator(device=self.embed_tokens.device)
        gen.manual_seed(0 if seed is None else seed + 1)

        def uniform(p, lo, hi):
            p.copy_(torch.rand(p.shape, device=p.device, dtype=torch.float32, generator=gen) * (hi - lo) + lo)

        for name, p in self.named_parameters():
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("norm1", "norm1b", "norm2", "norm2b", "D"):
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
        32-bit residual stream after every layer's mixer and feed-forward."""
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

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return M.softcap_(M.linear(hidden, self.output_weight, fp32_out=True), self.cfg.logit_softcap)

    def forward_hidden(self, *a, **kw):
        raise NotImplementedError("mixer stacks run step by step on a StateCache (forward_step); they are served, not trained")
