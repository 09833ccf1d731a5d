"""Plain implementation of the Tobadra decoder for tests: one sequence, whole matrices, the recurrences token by token, one
function per mechanism, no cache, no paging, no code of the package.  ``cfg`` is the plain dict of a ``config.json``; ``w``
maps checkpoint tensor names to tensors (already in the wanted dtype)."""
import math

import torch


# ---- norms and element-wise pieces -----------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit_length(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.where(z > 0, z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(x, taps):
    """``x [n, channels]``, ``taps [channels, k]``: the last tap multiplies the current row; zeros before the start."""
    n, k = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(k - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[j:j + n] * taps[:, j] for j in range(k))


def turn_halves(x, base, dims, sign=1.0, first=0):
    """``x [n, heads, width]`` at positions ``first ..``: dimension i turns with ``i + dims / 2`` by ``sign`` times the position times
    ``base ** (-2 i / dims)``."""
    n, half, out = x.shape[0], dims // 2, x.clone()
    for i in range(half):
        a = sign * torch.arange(first, first + n, dtype=torch.float64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        out[..., i] = x[..., i] * c - x[..., i + half] * s
        out[..., i + half] = x[..., i + half] * c + x[..., i] * s
    return out


# ---- mixers -----------------------------------------------------------------------------------------
def attend(q, k, v, scale, window):
    """``q [n, H, dim]``, ``k [n, G, dim]``, ``v [n, G, vdim]``: softmax over a query's own key and the ``window - 1`` before it."""
    n, per = q.shape[0], q.shape[1] // k.shape[1]
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    seen = (back >= 0) & (back < window)
    outs = []
    for h in range(q.shape[1]):
        score = ((q[:, h] @ k[:, h // per].T) * scale).masked_fill(~seen, -math.inf)
        e = torch.exp(score - score.max(dim=1, keepdim=True).values)
        outs.append((e / e.sum(dim=1, keepdim=True)) @ v[:, h // per])
    return torch.stack(outs, dim=1)


def attention(h, w, p, m, eps):
    """Values carry their positions: turned like keys (over the whole head), the weighted sum is turned back by the query's position."""
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q, k, v = ((h @ w[p + x].T + w[p + x + ".b"]).reshape(n, g, -1) for x, g in (("q", H), ("k", G), ("v", G)))
    q, k = turn_halves(q, base, dims), turn_halves(k, base, dims)
    o = attend(q, k, turn_halves(v, base, m["vdim"]), m["scale"], m["mask"]["size"])
    return turn_halves(o, base, m["vdim"], -1.0).reshape(n, -1) @ w[p + "o"].T + w[p + "o.b"]


def scan_fixed(q, k, v, decay):
    """``q, k [n, H, D]``, ``v [n, H, V]``, ``decay [H]``."""
    s, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype), []
    for t in range(q.shape[0]):
        s = decay[:, None, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", s, q[t]))
    return torch.stack(out)


def lightning(h, w, p, m, eps):
    n, H = h.shape[0], m["heads"]
    q, k, v = (silu(h @ w[p + x].T).reshape(n, H, -1) for x in "qkv")
    o = scan_fixed(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)).reshape(n, -1)
    return (unit_rms(o, eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def scan_delta(q, k, v, g, beta):
    """``q, k, g [n, H, D]`` (``g``: what is kept of every key channel), ``v [n, H, V]``, ``beta [n, H]``."""
    s, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype), []
    for t in range(q.shape[0]):
        s = g[t][:, :, None] * s
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", s, k[t]))
        s = s + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", s, q[t]))
    return torch.stack(out)


def channel_decay(h, w, p, heads):
    """What every key channel keeps, ``[n, heads, dim]``."""
    n = h.shape[0]
    step = softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(n, heads, -1)
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * step)


def channel_delta(h, w, p, m, eps):
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (silu(causal_conv(h @ w[p + x].T, w[f"{p}{x}.conv"])) for x in "qkv")
    q, k = (unit_length(x.reshape(n, G, -1)).repeat_interleave(H // G, dim=1) for x in (q, k))
    o = scan_delta(q * m["dim"] ** -0.5, k, v.reshape(n, H, -1), channel_decay(h, w, p, H), sigmoid(h @ w[p + "b"].T))
    z = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return ((unit_rms(o, eps) * w[p + "norm"]).reshape(n, -1) * z) @ w[p + "o"].T


MIXERS = {"attention": attention, "lightning": lightning, "channel_delta": channel_delta}


# ---- feed-forwards ----------------------------------------------------------------------------------------
def plain_ff(h, w, p, act):
    return act(h @ w[p + "up"].T) @ w[p + "down"].T


def route(z, correction, r):
    """Router logits ``z [n, outputs]`` -> (outputs chosen ``[n, top]``, their weights)."""
    e = torch.exp(z - z.max(dim=1, keepdim=True).values)
    s = e / e.sum(dim=1, keepdim=True)
    choice = s + correction
    n, outputs = choice.shape
    count, keep = r["groups"]["count"], r["groups"]["keep"]
    best = choice.reshape(n, count, -1).max(dim=2).values
    for t in range(n):
        kept = sorted(range(count), key=lambda g: (-float(best[t, g]), g))[:keep]
        for g in range(count):
            if g not in kept:
                choice[t, g * outputs // count:(g + 1) * outputs // count] = -math.inf
    idx = torch.sort(choice, dim=1, descending=True, stable=True).indices[:, :r["top"]]
    return idx, s.gather(1, idx) * r["scale"]


def experts(h, w, p, f):
    r = f["router"]
    idx, weight = route(h @ w[p + "router"].T, w[p + "correction"], r)
    out = torch.zeros_like(h)
    if f.get("shared") is not None:
        out = sigmoid(h @ w[p + "shared.sg"].T) * plain_ff(h, w, p + "shared.", gelu_erf)
    for e in range(r["experts"] + r["identity"]):
        rows, place = torch.nonzero(idx == e, as_tuple=True)
        if len(rows):
            y = plain_ff(h[rows], w, f"{p}e{e}.", gelu_erf) if e < r["experts"] else h[rows]
            out[rows] += weight[rows, place][:, None] * y
    return out


def feed_forward(h, w, p, f):
    return plain_ff(h, w, p, gelu_tanh) if f["kind"] == "dense" else experts(h, w, p, f)


# ---- the model --------------------------------------------------------------------------------------------
def gated(y, h, w, p):
    return y * sigmoid(h @ w[p].T + w[p + ".b"])


def forward(cfg, w, tokens, dtype=torch.float64):
    """(logits ``[n, vocab]``, stream after every layer ``[layers, n, width]``)."""
    w = {k: t.detach().cpu().to(dtype) for k, t in w.items()}
    eps, states = cfg["norm"]["eps"], []
    norm = lambda x, name: unit_rms(x, eps) * w[name]
    x = norm(w["embed"][torch.tensor(tokens)], "embed.norm")
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        h = norm(x, p + "norm1")
        y = MIXERS[layer["type"]](h + causal_conv(h, w[p + "canon1"]), w, p + "mix.", layer["mixer"], eps)
        x = x + norm(gated(y, h, w, p + "rg1"), p + "norm1b")
        if layer["mlp"] is not None:
            h = norm(x, p + "norm2")
            x = x + norm(gated(feed_forward(h, w, p + "mlp.", layer["mlp"]), h, w, p + "rg2"), p + "norm2b")
        states.append(x)
    return norm(x, "final.norm") @ w["embed"].T * cfg["logit_scale"], torch.stack(states)
