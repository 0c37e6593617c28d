"""Plain, slow statement of the Bumotar model, one function per mechanism.

Used by the tests as the oracle. Written straight from the equations, one sequence at a time and (in the attentions, the
retention and the experts) one token at a time; shares no code with the package (it reads the same config.json keys and
tensor names). Everything is computed in the dtype of the weights it is given (the tests pass float64)."""
import math

import torch


def rms(x, eps):
    return torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return x / rms(x, eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ----------------------------------------------------------------------------- rotation
def base_frequencies(rot):
    return [rot["base"] ** (-2 * i / rot["dims"]) for i in range(rot["dims"] // 2)]


def linear_frequencies(rot):
    """Every frequency divided by the stretch factor."""
    f = (rot.get("scaling") or {}).get("factor", 1.0)
    return [x / f for x in base_frequencies(rot)]


def yarn_frequencies(rot):
    """(frequencies, factor of cos and sin): low frequencies stretched, high ones kept, a ramp between."""
    s, d, freqs = rot.get("scaling"), rot["dims"], base_frequencies(rot)
    if not s:
        return freqs, 1.0

    def place(turns):
        return d * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(rot["base"]))
    lo, hi = max(math.floor(place(s["fast"])), 0), min(math.ceil(place(s["slow"])), d - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0), 1)
        out.append(f / s["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, positions, freqs, pairs, mult=1.0):
    """x [L, ..., d]: the given (u, v) pairs of the last axis turned by position times frequency."""
    x = x.clone()
    shape = [len(positions)] + [1] * (x.dim() - 2)
    for (a, b), f in zip(pairs, freqs):
        ang = torch.as_tensor(positions, dtype=x.dtype).view(shape) * f
        u, v, c, s = x[..., a].clone(), x[..., b].clone(), torch.cos(ang) * mult, torch.sin(ang) * mult
        x[..., a], x[..., b] = u * c - v * s, v * c + u * s
    return x


def halves(dims):
    return [(i, i + dims // 2) for i in range(dims // 2)]


def neighbours(dims):
    return [(2 * i, 2 * i + 1) for i in range(dims // 2)]


# ----------------------------------------------------------------------------- attention
def first_visible(i, window):
    """First position that position i sees: itself and the window - 1 before it."""
    return max(0, i - window + 1) if window else 0


def cap(s, c):
    return c * torch.tanh(s / c) if c else s


def weights(s, sink):
    """s [H, n]: softmax with exp(sink) in the denominator (None: nothing)."""
    top = s.max(-1, keepdim=True).values
    e, more = torch.exp(s - top), 0.0
    if sink is not None:
        more = torch.exp(torch.as_tensor(sink, dtype=s.dtype).view(-1, 1) - top)
    return e / (e.sum(-1, keepdim=True) + more)


def attend(q, k, v, scale, softcap, window, sink):
    """q [L, H, d], k [L, G, d], v [L, G, e]: query head h reads key / value head h // (H / G)."""
    L, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for i in range(L):
        j = first_visible(i, window)
        kk, vv = k[j:i + 1].repeat_interleave(rep, 1), v[j:i + 1].repeat_interleave(rep, 1)
        w = weights(cap(torch.einsum("hd,jhd->hj", q[i], kk) * scale, softcap), sink)
        out[i] = torch.einsum("hj,jhe->he", w, vv)
    return out


def windowed(W, p, h, m, eps):
    """Capped attention in a sliding window with normed, rotated queries and keys, one added to the softmax's denominator
    and a gate on every channel."""
    L, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = norm((h @ W[p + "q"].T).view(L, H, d), W[p + "q.norm"], eps)
    k = norm((h @ W[p + "k"].T).view(L, G, d), W[p + "k.norm"], eps)
    v = (h @ W[p + "v"].T).view(L, G, e)
    f, pairs, t = linear_frequencies(m["rot"]), halves(m["rot"]["dims"]), range(L)
    o = attend(rotate(q, t, f, pairs), rotate(k, t, f, pairs), v, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"),
               ONE_SINK if ONE_SINK is None else torch.full((H,), ONE_SINK))
    return (o.reshape(L, -1) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


ONE_SINK = 0.0           # score of the entry that adds one to the denominator


def latents(W, p, h, m, eps):
    """(normed latent, the key part that all heads share, not yet rotated)."""
    z = h @ W[p + "dkv"].T
    return norm(z[:, :m["kv_rank"]], W[p + "dkv.norm"], eps), z[:, m["kv_rank"]:]


def latent_attention(W, p, h, m, eps, steady=None):
    L, H, d, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    q = (h @ W[p + "q"].T).view(L, H, d + r)
    c, shared = latents(W, p, h, m, eps)
    f, mult = yarn_frequencies(m["rot"])
    q = torch.cat([q[..., :d], rotate(q[..., d:], range(L), f, neighbours(r), mult)], -1)
    shared = rotate(shared, range(L), f, neighbours(r), mult)
    k = torch.cat([(c @ W[p + "uk"].T).view(L, H, d), shared[:, None, :].expand(L, H, r)], -1)
    v = (c @ W[p + "uv"].T).view(L, H, m["vdim"])
    o = attend(q, k, v, m["scale"], None, None, W[p + "sink"])
    return (o * sigmoid(h @ W[p + "g"].T)[..., None]).reshape(L, -1) @ W[p + "o"].T


# ----------------------------------------------------------------------------- retention
def retain(q, k, v, decay):
    """q, k [L, H, d], v [L, H, e], a factor per head: the state forgets by it, takes k v^T in, and is read with q."""
    L, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    a, out = torch.as_tensor(decay, dtype=q.dtype).view(H, 1, 1), []
    for t in range(L):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def steadiness(o, q, k, v, decay):
    """[L]: size of a head's output beside the terms it is a sum of (per token, of the worst head). What it is divided by is its
    own size, so an output whose terms cancel carries their rounding, enlarged."""
    term = torch.zeros(o.shape[1], dtype=o.dtype)
    a, out = torch.as_tensor(decay, dtype=o.dtype), []
    for t in range(o.shape[0]):
        term = a ** 2 * term + (k[t] * k[t]).sum(-1) * (v[t] * v[t]).mean(-1)
        out.append(((o[t] * o[t]).mean(-1) / (term * (q[t] * q[t]).sum(-1))).sqrt().min())
    return torch.stack(out)


def retention(W, p, h, m, eps, steady=None):
    L, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ W[p + n].T).view(L, H, x) for n, x in (("q", d), ("k", d), ("v", e)))
    f, pairs = base_frequencies(m["rot"]), halves(m["rot"]["dims"])
    q, k = rotate(q, range(L), f, pairs), rotate(k, range(L), f, pairs) * d ** -0.5
    o = retain(q, k, v, m["decay"])
    if steady is not None:
        steady.append(steadiness(o, q, k, v, m["decay"]))
    return ((o / rms(o, eps)).reshape(L, -1) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel(W, p, h, m, eps, steady=None):
    return m["left_scale"] * windowed(W, p + "left.", h, m["left"], eps) + m["right_scale"] * retention(W, p + "right.", h, m["right"], eps, steady)


# ----------------------------------------------------------------------------- feed-forward
def expert(W, p, h):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, router, top):
    """Chosen experts and what they count, per token."""
    z = h @ router.T
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    chosen = torch.argsort(s, dim=-1, descending=True)[:, :top]
    s = s.gather(1, chosen)
    return chosen, s / (s.sum(-1, keepdim=True) + 1e-20)


def shared_expert(W, p, h):
    return sigmoid(h @ W[p + "sg"].T) * expert(W, p, h)


def feed_forward(W, p, h, mlp, margins=None):
    E, top = mlp["router"]["experts"], mlp["router"]["top"]
    chosen, weight = route(h, W[p + "router"], top)
    if margins is not None and top < E:
        z = (h @ W[p + "router"].T).sort(-1, descending=True).values
        margins.append(z[:, top - 1] - z[:, top])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weight[t]):
            out[t] += w * expert(W, f"{p}e{e}.", h[t])
    return out + shared_expert(W, p + "shared.", h) if mlp.get("shared") else out


# ----------------------------------------------------------------------------- the stack
def runs(config):
    """[(layer, number of its pass or None)] in the order in which they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    body = [(i, t) for t in range(loop["times"]) for i in range(loop["start"], loop["stop"])]
    return [(i, None) for i in range(loop["start"])] + body + [(i, None) for i in range(loop["stop"], n)]


def enter_pass(W, x, x0, t):
    return torch.cat([x, x0], -1) @ W["loop.in"].T + W["loop.step"][t]


MIXERS = {"latent_attention": latent_attention, "parallel": parallel}


def forward(W, config, tokens, margins=None, steady=None):
    """Logits [L, vocab] of one sequence, and the residual stream after every layer run. ``margins`` (a list) collects, per
    routed layer, how far each token's last chosen expert's logit is ahead of the first one left out, ``steady`` the
    :func:`steadiness` of every retention."""
    eps = config["norm"]["eps"]
    x0 = x = W["embed"][torch.as_tensor(tokens)]
    states = []
    for i, t in runs(config):
        layer, p = config["layers"][i], f"l{i}."
        if t is not None and i == config["loop"]["start"]:
            x = enter_pass(W, x, x0, t)
        x = x + MIXERS[layer["type"]](W, p + "mix.", norm(x, W[p + "norm1"], eps), layer["mixer"], eps, steady)
        if layer["mlp"] is not None:
            x = x + feed_forward(W, p + "mlp.", norm(x, W[p + "norm2"], eps), layer["mlp"], margins)
        states.append(x)
    return norm(x, W["final.norm"], eps) @ W["head"].T * config["logit_scale"], torch.stack(states)
