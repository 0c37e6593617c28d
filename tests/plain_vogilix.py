"""Plain, slow statement of the Vogilix model, one function per mechanism.

Used by the tests as the oracle. Written straight from the equations, one sequence at a time and (in the
attention and the experts) one token at a time; shares no code with the package (it reads the same
config.json keys and tensor names). Everything is computed in the dtype of the weights it is given
(the tests pass float64)."""
import math

import torch


def rms(x, eps):
    return torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def plain_norm(x, w, eps):
    return x / rms(x, eps) * w


def offset_norm(x, w, eps):
    """The stored weight is the distance of the factor from one."""
    return x / rms(x, eps) * (1 + w)


def gelu_erf(z):
    return z * 0.5 * (1 + torch.erf(z / math.sqrt(2)))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def embed(W, tokens):
    """Token vector plus the vector of its position, counted from zero."""
    return W["embed"][tokens] + W["pos"][:len(tokens)]


def visible(i, window):
    """First position that position i sees: itself and the window - 1 before it."""
    return max(0, i - window + 1) if window else 0


def attend(q, k, v, scale, window):
    """q, k [L, H, d], v [L, H, e]: softmax over the window, every head with its own keys and values."""
    L, H, _ = q.shape
    out = torch.zeros(L, H, v.shape[2], dtype=q.dtype)
    for i in range(L):
        j = visible(i, window)
        s = torch.einsum("hd,jhd->hj", q[i], k[j:i + 1]) * scale
        w = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhe->he", w / w.sum(-1, keepdim=True), v[j:i + 1])
    return out


def latents(W, pre, h, eps):
    """(query latent, key / value latent), each normed over its whole width."""
    return plain_norm(h @ W[pre + "dq"].T, W[pre + "dq.norm"], eps), plain_norm(h @ W[pre + "dkv"].T, W[pre + "dkv.norm"], eps)


def latent_attention(W, pre, h, m, eps):
    H, L = m["heads"], h.shape[0]
    cq, c = latents(W, pre, h, eps)
    q, k, v = cq @ W[pre + "uq"].T, c @ W[pre + "uk"].T, c @ W[pre + "uv"].T
    o = attend(q.view(L, H, m["dim"]), k.view(L, H, m["dim"]), v.view(L, H, m["vdim"]), m["scale"], (m.get("mask") or {}).get("size") or 0)
    return o.reshape(L, -1) @ W[pre + "o"].T


def expert(W, pre, h, limit):
    g = (h @ W[pre + "gate"].T).clamp(max=limit)
    u = (h @ W[pre + "up"].T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ W[pre + "down"].T


def route(h, router, top):
    """Chosen experts and their scores, per token."""
    s = sigmoid(h @ router.T)
    chosen = torch.argsort(s, dim=-1, descending=True)[:, :top]
    return chosen, s.gather(1, chosen)


def feed_forward(W, pre, h, mlp, margins=None):
    if mlp["kind"] == "dense":
        return gelu_erf(h @ W[pre + "up"].T) @ W[pre + "down"].T
    E, top = mlp["router"]["experts"], mlp["router"]["top"]
    chosen, weight = route(h, W[pre + "router"], top)
    if margins is not None and top < E:
        s = (h @ W[pre + "router"].T).sort(-1, descending=True).values
        margins.append(s[:, top - 1] - s[:, top])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weight[t]):
            out[t] += expert(W, f"{pre}e{e}.", w * h[t], mlp["expert"]["limit"])
    if mlp.get("shared"):
        out = out + expert(W, pre + "shared.", h, mlp["shared"]["limit"])
    return out


def side_input(W, i, x, tokens, dim):
    """What a layer gets from the token itself, before its norm: a gate of x on the layer's part of the token's row."""
    e = W["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    return (gelu_tanh(x @ W[f"l{i}.side.gate"].T) * e) @ W[f"l{i}.side.proj"].T


def forward(W, config, tokens, margins=None):
    """Logits [L, vocab] of one sequence, and the residual stream after every layer. ``margins`` (a list) collects, per
    routed layer, how far each token's last chosen expert's logit is ahead of the first one left out."""
    eps, m = config["norm"]["eps"], config["residual_mult"]
    tokens = torch.as_tensor(tokens)
    x = embed(W, tokens)
    states = []
    for i, layer in enumerate(config["layers"]):
        pre = f"l{i}."
        x = x + m * offset_norm(latent_attention(W, pre + "mix.", x, layer["mixer"], eps), W[pre + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + m * offset_norm(feed_forward(W, pre + "mlp.", x, layer["mlp"], margins), W[pre + "norm2"], eps)
        if config.get("token_side"):
            x = x + m * plain_norm(side_input(W, i, x, tokens, config["token_side"]["dim"]), W[pre + "side.norm"], eps)
        states.append(x)
    return offset_norm(x, W["final.norm"], eps) @ W["head"].T, torch.stack(states)
