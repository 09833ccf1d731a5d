"""Plain implementation of the Zinutar decoder for tests: one sequence, whole matrices, one function per mechanism,
no cache, no paging, no code of the package.  ``cfg`` is the plain dict of a ``config.json``; ``w`` maps checkpoint
tensor names to tensors."""
import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def embedding_output(w, tokens, eps):
    return rms(w["embed"][torch.tensor(tokens)], eps) * w["embed.norm"]


def execution_order(n_layers, loop):
    """[(layer, add the embedding output first?)]"""
    if not loop:
        return [(i, False) for i in range(n_layers)]
    order = [(i, False) for i in range(0, loop["start"])]
    for turn in range(loop["times"]):
        for i in range(loop["start"], loop["stop"]):
            order.append((i, turn >= 1 and i == loop["start"]))
    order += [(i, False) for i in range(loop["stop"], n_layers)]
    return order


def key_weights(q, k, scale, bias):
    """``q [n, dim]``, ``k [n, dim]`` of one head -> weights ``[n, n]``: a sigmoid per visible key."""
    s = (q @ k.T) * scale + bias
    n = q.shape[0]
    seen = torch.arange(n)[None, :] <= torch.arange(n)[:, None]
    return torch.where(seen, 1.0 / (1.0 + torch.exp(-s)), torch.zeros_like(s))


def attention(h, w, p, m, eps):
    n, outs = h.shape[0], []
    q = (h @ w[p + "mix.q"].T).reshape(n, m["heads"], m["dim"])
    k = (h @ w[p + "mix.k"].T).reshape(n, m["kv_heads"], m["dim"])
    v = (h @ w[p + "mix.v"].T).reshape(n, m["kv_heads"], m["vdim"])
    for head in range(m["heads"]):
        kv = head // (m["heads"] // m["kv_heads"])
        a = key_weights(rms(q[:, head], eps), rms(k[:, kv], eps), m["scale"], w[p + "mix.pb"][head])
        outs.append(a @ v[:, kv])
    return torch.cat(outs, dim=1) @ w[p + "mix.o"].T


def poly_act(z, coef, eps):
    return coef[0] * rms(z, eps) + coef[1] * rms(z ** 2, eps) + coef[2] * rms(z ** 3, eps) + coef[3]


def feed_forward(h, w, p, eps):
    return poly_act(h @ w[p + "mlp.up"].T, w[p + "mlp.act"], eps) @ w[p + "mlp.down"].T


def forward(cfg, w, tokens, dtype=torch.float64):
    """(logits ``[n, vocab]``, stream after every layer execution ``[runs, n, width]``)."""
    w = {k: t.detach().cpu().to(dtype) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = x0 = embedding_output(w, tokens, eps)
    states = []
    for i, again in execution_order(len(cfg["layers"]), cfg.get("loop")):
        if again:
            x = x + x0
        layer, p = cfg["layers"][i], f"l{i}."
        h = rms(x, eps) * w[p + "norm1"]
        y = attention(h, w, p, layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + feed_forward(h, w, p, eps)
        x = x + y
        states.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T, torch.stack(states)
