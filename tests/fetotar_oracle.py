"""Plain implementation of the Fetotar decoder for tests: one sequence, one token after the other where the design
recurs, whole matrices elsewhere, one function per mechanism, no cache, no paging, no code of the package.  ``cfg`` is
the plain dict of a ``config.json``; ``w`` maps checkpoint tensor names to tensors (already in the wanted dtype)."""
import math

import torch


# ---- norms and element-wise pieces -----------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * weight + bias


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 0, z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def clamped_glu(gate, up, limit):
    g = torch.minimum(gate, torch.full_like(gate, limit))
    u = torch.maximum(torch.minimum(up, torch.full_like(up, limit)), torch.full_like(up, -limit))
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


# ---- rotary positions ---------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """(frequencies, amplitude) of the ``dims / 2`` pairs."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if s is None:
        return freq, 1.0

    def where(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """``x [n, ..., width]``: neighbouring dimensions (2i, 2i + 1) turn together; dimensions past ``dims`` stay."""
    freq, amp = rotary_frequencies(rot)
    out = x.clone()
    for i, f in enumerate(freq):
        a = torch.tensor(positions, dtype=torch.float64) * f
        c, s = (amp * torch.cos(a)).to(x.dtype), (amp * torch.sin(a)).to(x.dtype)
        shape = [-1] + [1] * (x.dim() - 2)
        c, s = c.reshape(shape), s.reshape(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ---- mixers --------------------------------------------------------------------------------------------
def causal_conv(x, taps, bias):
    """``x [n, channels]``, ``taps [channels, k]``: the last tap multiplies the current row; zeros before the start."""
    n, k = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(k - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[j:j + n] * taps[:, j] for j in range(k)) + bias


def scan_mamba2(x, b, c, dt, a_log, skip):
    """``x [n, heads, vdim]``, ``b, c [n, groups, state]``, ``dt [n, heads]`` (after softplus)."""
    n, heads, vdim = x.shape
    per = heads // b.shape[1]
    y = torch.zeros_like(x)
    for h in range(heads):
        s = torch.zeros(b.shape[2], vdim, dtype=x.dtype)
        for t in range(n):
            s = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * s + dt[t, h] * torch.outer(b[t, h // per], x[t, h])
            y[t, h] = s.T @ c[t, h // per] + skip[h] * x[t, h]
    return y


def mamba2(h, w, p, m, eps):
    n, heads, vdim = h.shape[0], m["heads"], m["vdim"]
    inner, gn = heads * vdim, m["groups"] * m["state"]
    z, xbc, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * gn, heads], dim=1)
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, b, c = xbc.split([inner, gn, gn], dim=1)
    y = scan_mamba2(x.reshape(n, heads, vdim), b.reshape(n, m["groups"], m["state"]), c.reshape(n, m["groups"], m["state"]),
                    softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"]).reshape(n, inner)
    y = unit_rms((y * silu(z)).reshape(n, m["norm_groups"], -1), eps).reshape(n, inner)
    return (y * w[p + "norm"]) @ w[p + "o"].T


def scan_mlstm(q, k, v, i, f):
    """``q, k [n, heads, dim]``, ``v [n, heads, vdim]``, log gates ``i, f [n, heads]``."""
    n, heads, vdim = v.shape
    out = torch.zeros_like(v)
    for h in range(heads):
        s = torch.zeros(q.shape[2], vdim, dtype=v.dtype)
        norm = torch.zeros(q.shape[2], dtype=v.dtype)
        top = torch.zeros((), dtype=v.dtype)
        for t in range(n):
            new = torch.maximum(f[t, h] + top, i[t, h])
            keep, add = torch.exp(f[t, h] + top - new), torch.exp(i[t, h] - new)
            s = keep * s + add * torch.outer(k[t, h], v[t, h])
            norm = keep * norm + add * k[t, h]
            top = new
            out[t, h] = (s.T @ q[t, h]) / (torch.maximum((norm @ q[t, h]).abs(), torch.exp(-top)) + 1e-6)
    return out


def mlstm(h, w, p, m, eps):
    n, heads, dim, vdim, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).reshape(n, heads, dim) * dim ** -0.5
    k = (h @ w[p + "k"].T).reshape(n, heads, dim)
    v = (h @ w[p + "v"].T).reshape(n, heads, vdim)
    soft = lambda z: cap * torch.tanh(z / cap)
    i = soft(h @ w[p + "i"].T + w[p + "i.b"])
    f = -softplus(-soft(h @ w[p + "f"].T + w[p + "f.b"]))
    o = unit_rms(scan_mlstm(q, k, v, i, f), eps).reshape(n, heads * vdim)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def window_softmax(score, size):
    """``score [n, n]`` of one head; a query sees itself and the ``size - 1`` keys before it."""
    n = score.shape[0]
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    seen = (back >= 0) & (back < size)
    e = torch.where(seen, torch.exp(score - score.masked_fill(~seen, -math.inf).max(dim=1, keepdim=True).values),
                    torch.zeros_like(score))
    return e / e.sum(dim=1, keepdim=True)


def latent_attention(h, w, p, m, eps):
    n, heads, dim, rd, vdim, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = list(range(n))
    cq = unit_rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(n, heads, dim + rd)
    dkv = h @ w[p + "dkv"].T
    c = unit_rms(dkv[:, :rank], eps) * w[p + "dkv.norm"]
    kr = rotate(dkv[:, rank:], pos, m["rot"])
    qr = rotate(q[:, :, dim:], pos, m["rot"])
    k = (c @ w[p + "uk"].T).reshape(n, heads, dim)
    v = (c @ w[p + "uv"].T).reshape(n, heads, vdim)
    outs = []
    for hd in range(heads):
        score = (q[:, hd, :dim] @ k[:, hd].T + qr[:, hd] @ kr.T) * m["scale"]
        outs.append(window_softmax(score, m["mask"]["size"]) @ v[:, hd])
    return (torch.cat(outs, dim=1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"mamba2": mamba2, "mlstm": mlstm, "latent_attention": latent_attention}


# ---- the rest of a layer, the model -----------------------------------------------------------------------
def feed_forward(h, w, p, limit):
    return clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def token_side(x, w, p, e, eps):
    y = (gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return unit_rms(y, eps) * w[p + "side.norm"]


def embedding(cfg, w, tokens):
    return w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]


def forward(cfg, w, tokens, dtype=torch.float64):
    """(logits ``[n, vocab]``, stream after every layer ``[layers, n, width]``)."""
    w = {k: t.detach().cpu().to(dtype) for k, t in w.items()}
    eps, sd = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    ids = torch.tensor(tokens)
    norm = lambda x, name: layer_norm(x, w[name], w[name + ".b"], eps)
    x, states = embedding(cfg, w, tokens), []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](norm(x, p + "norm1"), w, p + "mix.", layer["mixer"], eps)
        x = x + norm(y, p + "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(feed_forward(norm(x, p + "norm2"), w, p + "mlp.", layer["mlp"]["limit"]), p + "norm2b")
        x = x + token_side(x, w, p, w["side.embed"][ids, i * sd:(i + 1) * sd], eps)
        states.append(x)
    return norm(x, "final.norm") @ w["head"].T, torch.stack(states)
