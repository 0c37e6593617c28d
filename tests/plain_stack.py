"""Plain, slow statement of the mixer-stack model (Kagolix), one function per mechanism.

Used by the tests as the oracle. Written straight from the equations, one sequence at a time and one
token at a time wherever there is a recurrence; shares no code with the package (it reads the same
config.json keys and tensor names). Everything is computed in the dtype of the weights it is given
(the tests pass float64)."""
import math

import torch


def root_mean_square_norm(x, w, eps, groups=1):
    """Each of ``groups`` consecutive parts divided by sqrt(mean(part^2) + eps); the whole times w."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    rms = torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)
    return (parts / rms).reshape(x.shape) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def xielu(z, p, q):
    neg = (0.5 + softplus(q)) * (torch.expm1(z.clamp(max=0)) - z.clamp(max=0)) + z / 2
    return torch.where(z > 0, softplus(p) * z * z + z / 2, neg)


def attend(q, k, v, scale, softcap, r1, r2, chunk):
    """q [L, H, d], k [L, G, d], v [L, G, e]: capped scores less a logarithmic distance bias, softmax over
    the earlier positions of the query's own chunk."""
    L, H, _ = q.shape
    per = H // k.shape[1]
    at = torch.arange(L)
    dist = (at[:, None] - at[None, :]).to(q.dtype)
    seen = dist >= 0
    if chunk:
        seen &= (at // chunk)[:, None] == (at // chunk)[None, :]
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // per].T * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        s = s - r1[h] * torch.log(1 + r2[h] * dist.clamp(min=0))
        s = torch.where(seen, s, torch.full_like(s, -math.inf))
        w = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append(w / w.sum(-1, keepdim=True) @ v[:, h // per])
    return torch.stack(out, 1)


def attention(W, pre, h, cfg, eps):
    m = cfg["mixer"]
    H, G, L = m["heads"], m["kv_heads"], h.shape[0]
    q, k, v = h @ W[pre + "q"].T, h @ W[pre + "k"].T, h @ W[pre + "v"].T
    q = root_mean_square_norm(q, W[pre + "q.norm"], eps)
    k = root_mean_square_norm(k, W[pre + "k.norm"], eps)
    o = attend(q.view(L, H, m["dim"]), k.view(L, G, m["dim"]), v.view(L, G, m["vdim"]), m["scale"], m["softcap"],
               W[pre + "r1"], W[pre + "r2"], m["mask"]["size"])
    return o.reshape(L, -1) @ W[pre + "o"].T


def causal_conv(x, w, b):
    """out[t, c] = b[c] + sum_j w[c, K - 1 - j] x[t - j, c], zeros before the start."""
    out = b.expand_as(x).clone()
    for j in range(w.shape[1]):
        out[j:] += w[:, w.shape[1] - 1 - j] * x[:x.shape[0] - j]
    return out


def rglru(W, pre, h, cfg, eps):
    n = cfg["mixer"]["blocks"]
    y = gelu_tanh(h @ W[pre + "y"].T + W[pre + "y.b"])
    u = causal_conv(h @ W[pre + "x"].T + W[pre + "x.b"], W[pre + "conv"], W[pre + "conv.b"])
    L, width = u.shape
    ub = u.view(L, n, width // n)
    r = torch.stack([sigmoid(ub[:, b] @ W[pre + "ra"][b].T + W[pre + "ra.b"][b]) for b in range(n)], 1).reshape(L, width)
    i = torch.stack([sigmoid(ub[:, b] @ W[pre + "ri"][b].T + W[pre + "ri.b"][b]) for b in range(n)], 1).reshape(L, width)
    log_a = -8 * r * softplus(W[pre + "lam"])
    S = torch.zeros(width, dtype=h.dtype)
    outs = []
    for t in range(L):
        S = torch.exp(log_a[t]) * S + torch.sqrt(-torch.expm1(2 * log_a[t])) * i[t] * u[t]
        outs.append(S)
    return (torch.stack(outs) * y) @ W[pre + "o"].T


def mamba2(W, pre, h, cfg, eps):
    m = cfg["mixer"]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, L = H * P, h.shape[0]
    z, xbc, dt = torch.split(h @ W[pre + "in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(causal_conv(xbc, W[pre + "conv"], W[pre + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    x, B, C = x.view(L, H, P), B.view(L, G, N), C.view(L, G, N)
    dt = softplus(dt + W[pre + "dt_bias"])
    B, C = (t[:, [hd // (H // G) for hd in range(H)]] for t in (B, C))          # each head's group
    decay = torch.exp(-torch.exp(W[pre + "A_log"]) * dt)
    S, y = torch.zeros(H, N, P, dtype=h.dtype), []
    for t in range(L):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        y.append(torch.einsum("hnp,hn->hp", S, C[t]) + W[pre + "D"][:, None] * x[t])
    y = torch.stack(y)
    y = y.reshape(L, inner) * silu(z)
    return root_mean_square_norm(y, W[pre + "norm"], eps, m["norm_groups"]) @ W[pre + "o"].T


MIXERS = {"attention": attention, "rglru": rglru, "mamba2": mamba2}


def route(h, router, correction, top):
    z = h @ router.T
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    chosen = torch.argsort(s + correction, dim=-1, descending=True)[:, :top]
    return chosen, s.gather(1, chosen)


def feed_forward(W, pre, h, mlp, margins=None):
    if mlp["kind"] == "dense":
        p, q = W[pre + "act"]
        return xielu(h @ W[pre + "up"].T, p, q) @ W[pre + "down"].T
    chosen, weight = route(h, W[pre + "router"], W[pre + "correction"], mlp["router"]["top"])
    if margins is not None and mlp["router"]["top"] < mlp["router"]["experts"]:
        c = torch.softmax(h @ W[pre + "router"].T, -1) + W[pre + "correction"]
        c = c.sort(-1, descending=True).values
        margins.append(c[:, mlp["router"]["top"] - 1] - c[:, mlp["router"]["top"]])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, slot = torch.where(chosen == e)
        p = f"{pre}e{e}."
        y = (silu(h[t] @ W[p + "gate"].T) * (h[t] @ W[p + "up"].T)) @ W[p + "down"].T
        out[t] += weight[t, slot, None] * y
    return out


def forward(W, config, tokens, margins=None):
    """Logits [L, vocab] of one sequence, and the residual stream after every layer. ``margins`` (a list) collects, per
    routed layer, how far each token's last chosen expert is ahead of the first one left out."""
    eps, groups = config["norm"]["eps"], config["norm"]["groups"]

    def norm(x, name):
        return root_mean_square_norm(x, W[name], eps, groups)

    x = W["embed"][torch.as_tensor(tokens)]
    states = []
    for i, layer in enumerate(config["layers"]):
        pre = f"l{i}."
        x = x + norm(MIXERS[layer["type"]](W, pre + "mix.", norm(x, pre + "norm1"), layer, eps), pre + "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(feed_forward(W, pre + "mlp.", norm(x, pre + "norm2"), layer["mlp"], margins), pre + "norm2b")
        states.append(x)
    logits = norm(x, "final.norm") @ W["head"].T
    cap = config["logit_softcap"]
    return cap * torch.tanh(logits / cap), torch.stack(states)
