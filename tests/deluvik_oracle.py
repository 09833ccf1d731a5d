"""Plain implementation of the Deluvik decoder for tests: one sequence, whole matrices, the recurrence token by token, one
function per mechanism, no cache, no paging, no code of the package.  ``cfg`` is the plain dict of a ``config.json``; ``w``
maps checkpoint tensor names to tensors (already in the wanted dtype)."""
import math

import torch


# ---- norms and element-wise pieces -----------------------------------------------------------------
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.where(z > 0, z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def causal_conv(x, taps):
    """``x [n, channels]``, ``taps [channels, k]``: the last tap multiplies the current row; zeros before the start."""
    n, k = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(k - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[j:j + n] * taps[:, j] for j in range(k))


# ---- rotary positions ---------------------------------------------------------------------------------
def rotary_frequencies(rot):
    freq = [rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
    s = rot.get("scaling")
    if s is None:
        return freq
    out = []
    for f in freq:
        wave = 2.0 * math.pi / f
        if wave < s["original"] / s["high"]:
            out.append(f)
        elif wave > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            mix = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - mix) * f / s["factor"] + mix * f)
    return out


def rotate(x, rot, half, first=0):
    """``x [n, heads, width]`` at positions ``first ..``.  ``half``: dimension i turns with i + dims / 2, else 2i with 2i + 1."""
    n, d = x.shape[0], rot["dims"]
    out = x.clone()
    for i, f in enumerate(rotary_frequencies(rot)):
        a = torch.arange(first, first + n, dtype=torch.float64) * f
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        j, k = (i, i + d // 2) if half else (2 * i, 2 * i + 1)
        out[..., j] = x[..., j] * c - x[..., k] * s
        out[..., k] = x[..., k] * c + x[..., j] * s
    return out


# ---- attention -----------------------------------------------------------------------------------------
def attend(q, k, v, scale, *, window=None, cap=None, sink=None):
    """``q [n, H, dim]``, ``k [n, G, dim]``, ``v [n, G, vdim]``; ``sink [H]`` joins the denominator."""
    n, heads = q.shape[0], q.shape[1]
    per = heads // k.shape[1]
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    seen = back >= 0
    if window is not None:
        seen &= back < window
    outs = []
    for h in range(heads):
        score = (q[:, h] @ k[:, h // per].T) * scale
        if cap is not None:
            score = soft_cap(score, cap)
        score = score.masked_fill(~seen, -math.inf)
        top = score.max(dim=1, keepdim=True).values
        if sink is not None:
            top = torch.maximum(top, sink[h])
        e = torch.exp(score - top)
        den = e.sum(dim=1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - top)
        outs.append((e / den) @ v[:, h // per])
    return torch.stack(outs, dim=1)


def attention(h, w, p, m, eps, shared):
    """The values are the keys as projected; norm over the whole projection, then rotation, cap and sink."""
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
    v = k.reshape(n, G, m["vdim"])
    q = rotate((unit_rms(q, eps) * w[p + "q.norm"]).reshape(n, H, d), m["rot"], True)
    k = rotate((unit_rms(k, eps) * w[p + "k.norm"]).reshape(n, G, d), m["rot"], True)
    o = attend(q, k, v, m["scale"], cap=m["softcap"], sink=w[p + "sink"])
    return o.reshape(n, -1) @ w[p + "o"].T


def conv_attention(h, w, p, m, eps, shared):
    """Projections pass a short convolution first; a layer with ``kv_from`` reads another layer's keys and values."""
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = causal_conv(h @ w[p + "q"].T, w[p + "q.conv"])
    q = rotate((unit_rms(q, eps) * w[p + "q.norm"]).reshape(n, H, d), m["rot"], True)
    if m.get("kv_from") is None:
        k = causal_conv(h @ w[p + "k"].T, w[p + "k.conv"])
        v = causal_conv(h @ w[p + "v"].T, w[p + "v.conv"]).reshape(n, G, m["vdim"])
        k = rotate((unit_rms(k, eps) * w[p + "k.norm"]).reshape(n, G, d), m["rot"], True)
        shared[p.split(".")[0]] = (k, v)
    else:
        k, v = shared[f"l{m['kv_from']}"]
    o = attend(q, k, v, m["scale"], sink=w[p + "sink"])
    return o.reshape(n, -1) @ w[p + "o"].T


def window_attention(h, w, p, m, eps):
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = (h @ w[p + "q"].T).reshape(n, H, d), (h @ w[p + "k"].T).reshape(n, G, d)
    v = (h @ w[p + "v"].T).reshape(n, G, m["vdim"])
    q = rotate(unit_rms(q, eps) * w[p + "q.norm"], m["rot"], False)
    k = rotate(unit_rms(k, eps) * w[p + "k.norm"], m["rot"], False)
    return attend(q, k, v, m["scale"], window=m["mask"]["size"]).reshape(n, -1) @ w[p + "o"].T


# ---- gated linear recurrence -----------------------------------------------------------------------------
def block_gate(u, mats, bias):
    """``u [n, width]``, ``mats [blocks, part, part]``: a sigmoid gate from every part's own matrix."""
    n, (b, part, _) = u.shape[0], mats.shape
    z = torch.stack([u.reshape(n, b, part)[:, i] @ mats[i].T + bias[i] for i in range(b)], dim=1)
    return sigmoid(z.reshape(n, b * part))


def scan_lru(u, r, i, lam):
    log_a = -8.0 * r * softplus(lam)
    s, out = torch.zeros(u.shape[1], dtype=u.dtype), []
    for t in range(u.shape[0]):
        s = torch.exp(log_a[t]) * s + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * i[t] * u[t]
        out.append(s)
    return torch.stack(out)


def recurrent_block(h, w, p):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"]) + w[p + "conv.b"]
    s = scan_lru(u, block_gate(u, w[p + "ra"], w[p + "ra.b"]), block_gate(u, w[p + "ri"], w[p + "ri.b"]), w[p + "lam"])
    return (s * y) @ w[p + "o"].T


def parallel(h, w, p, m, eps, shared):
    return m["left_scale"] * window_attention(h, w, p + "left.", m["left"], eps) + m["right_scale"] * recurrent_block(h, w, p + "right.")


MIXERS = {"attention": attention, "parallel": parallel, "attention_2": conv_attention}


# ---- feed-forwards ----------------------------------------------------------------------------------------
def glu(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, top):
    """(chosen experts ``[n, top]``, their weights)."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    best, idx = torch.sort(z, dim=1, descending=True, stable=True)
    e = torch.exp(best[:, :top] - best[:, :1])
    return idx[:, :top], e / e.sum(dim=1, keepdim=True)


def experts(h, w, p, m):
    idx, weight = route(h, w, p, m["router"]["top"])
    out = glu(h, w, p + "shared.", silu) if m.get("shared") is not None else torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows, place = torch.nonzero(idx == e, as_tuple=True)
        if len(rows):
            out[rows] += weight[rows, place][:, None] * glu(h[rows], w, f"{p}e{e}.", silu)
    return out


def feed_forward(h, w, p, f):
    return glu(h, w, p, gelu_tanh) if f["kind"] == "dense" else experts(h, w, p, f)


# ---- the model --------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, dtype=torch.float64):
    """(logits ``[n, vocab]``, stream after every layer ``[layers, n, width]``)."""
    w = {k: t.detach().cpu().to(dtype) for k, t in w.items()}
    eps, shared, states = cfg["norm"]["eps"], {}, []
    x = w["embed"][torch.tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + unit_rms(MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps, shared), eps) * w[p + "norm1"]
        if layer["mlp"] is not None:
            x = x + unit_rms(feed_forward(x, w, p + "mlp.", layer["mlp"]), eps) * w[p + "norm2"]
        states.append(x)
    return soft_cap((unit_rms(x, eps) * w["final.norm"]) @ w["head"].T, cfg["logit_softcap"]), torch.stack(states)
