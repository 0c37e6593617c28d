"""Plain, slow statement of the Goganex model, one function per mechanism.

Used by the tests as the oracle. Written straight from the equations, one sequence at a time and (in the attentions and the
recurrence) one token at a time; shares no code with the package (it reads the same config.json keys and tensor names).
Everything is computed in the dtype of the weights it is given (the tests pass float64)."""
import math

import torch


def rms(x, eps):
    return torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return x / rms(x, eps) * w


def unit(x, eps):
    """Per head, without a weight."""
    return x / rms(x, eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ----------------------------------------------------------------------------- token shift
def previous(h):
    """Every token's predecessor, zeros before the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def shifted(h, share):
    return h + (previous(h) - h) * share


# ----------------------------------------------------------------------------- rotation
def base_frequencies(rot):
    return [rot["base"] ** (-2 * i / rot["dims"]) for i in range(rot["dims"] // 2)]


def scaled_frequencies(rot):
    """Short wavelengths kept, long ones stretched by the factor, a blend between the two."""
    s = rot.get("scaling")
    if not s:
        return base_frequencies(rot)
    out = []
    for f in base_frequencies(rot):
        wave = 2 * math.pi / f
        if wave < s["original"] / s["high"]:
            out.append(f)
        elif wave > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1 - t) * f / s["factor"] + t * f)
    return out


def pairs(dims):
    return [(2 * i, 2 * i + 1) for i in range(dims // 2)]


def rotate(x, positions, freqs, which):
    """x [L, heads, d]: the given (u, v) pairs of the last axis turned by position times frequency."""
    x = x.clone()
    for (a, b), f in zip(which, freqs):
        ang = torch.as_tensor(positions, dtype=x.dtype)[:, None] * f
        u, v, c, s = x[..., a].clone(), x[..., b].clone(), torch.cos(ang), torch.sin(ang)
        x[..., a], x[..., b] = u * c - v * s, v * c + u * s
    return x


# ----------------------------------------------------------------------------- attention
def first_visible(i):
    return 0


def weights(s, extra):
    """s [H, n]: exp(s) over its sum plus ``extra``."""
    top = s.max(-1, keepdim=True).values.clamp(min=0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + extra * torch.exp(-top))


def attend(q, k, v, scale, temp, extra):
    """q [L, H, d], k [L, G, d], v [L, G, e]: query head h reads key / value head h // (H / G)."""
    L, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for i in range(L):
        j = first_visible(i)
        kk, vv = k[j:i + 1].repeat_interleave(rep, 1), v[j:i + 1].repeat_interleave(rep, 1)
        s = torch.einsum("hd,jhd->hj", q[i], kk) * scale * temp[:, None]
        out[i] = torch.einsum("hj,jhe->he", weights(s, extra), vv)
    return out


SINK = 1.0               # what the rotated attention's softmax has in its denominator beside the keys


def rotary_attention(W, p, h, m, eps):
    """Rotation, then norms on q and k; a factor per head on the scores; one added to the softmax's denominator."""
    L, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ W[p + "q"].T).view(L, H, d), (h @ W[p + "k"].T).view(L, G, d), (h @ W[p + "v"].T).view(L, G, e)
    f, which = scaled_frequencies(m["rot"]), pairs(m["rot"]["dims"])
    q, k = (unit(rotate(x, range(L), f, which), eps) for x in (q, k))
    return attend(q, k, v, m["scale"], W[p + "temp"], SINK).reshape(L, -1) @ W[p + "o"].T


def values_of(k, eps):
    """The keys themselves, before their norm."""
    return k


def key_value_attention(W, p, h, m, eps):
    """No positions; the projected keys are the values."""
    L, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = (h @ W[p + "q"].T).view(L, H, d), (h @ W[p + "k"].T).view(L, G, d)
    ones = torch.ones(H, dtype=h.dtype)
    return attend(unit(q, eps), unit(k, eps), values_of(k, eps), m["scale"], ones, 0.0).reshape(L, -1) @ W[p + "o"].T


# ----------------------------------------------------------------------------- recurrence
def candidate(u):
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def recur(z, c):
    """S = (1 - z) S + z c, element by element, from zero; every state."""
    S, out = torch.zeros_like(z[0]), []
    for t in range(z.shape[0]):
        S = (1 - z[t]) * S + z[t] * c[t]
        out.append(S)
    return torch.stack(out)


def min_gru(W, p, h, m, eps):
    z = sigmoid(h @ W[p + "z"].T + W[p + "z.b"])
    S = recur(z, candidate(h @ W[p + "x"].T + W[p + "x.b"]))
    return (S * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def join(left, right):
    return 0.5 * (left + right)


def side_by_side(W, p, h, m, eps):
    left = key_value_attention(W, p + "left.", h, m["left"], eps)
    right = min_gru(W, p + "right.", h, m["right"], eps)
    return join(norm(left, W[p + "left.out"], eps), norm(right, W[p + "right.out"], eps))


# ----------------------------------------------------------------------------- feed-forward
def clipped(gate, up, limit):
    return gate.clamp(max=limit), up.clamp(-limit, limit)


def feed_forward(W, p, h, mlp):
    g, u = clipped(h @ W[p + "gate"].T, h @ W[p + "up"].T, mlp["limit"])
    return (g * sigmoid(1.702 * g) * (u + 1)) @ W[p + "down"].T


# ----------------------------------------------------------------------------- the stack
def runs(config):
    """Layers in the order in which they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


MIXERS = {"attention": rotary_attention, "parallel": side_by_side}


def embed(W, config, tokens):
    return W["embed"][torch.as_tensor(tokens)] * config["embedding"]["scale"]


def forward(W, config, tokens):
    """Logits [L, vocab] of one sequence, and the residual stream after every layer run."""
    eps = config["norm"]["eps"]
    x, states = embed(W, config, tokens), []
    for i in runs(config):
        layer, p = config["layers"][i], f"l{i}."
        h = shifted(norm(x, W[p + "norm1"], eps), W[p + "shift"])
        x = x + MIXERS[layer["type"]](W, p + "mix.", h, layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + feed_forward(W, p + "mlp.", norm(x, W[p + "norm2"], eps), layer["mlp"])
        states.append(x)
    return norm(x, W["final.norm"], eps) @ W["head"].T, torch.stack(states)
