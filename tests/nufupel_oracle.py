"""Plain restatement of the Nufupel decoder for tests: one function per mechanism, loops where loops are
clearest, float64 by default.  Nothing here is shared with the product path.

``forward`` runs a whole sequence at once; there is no cache and no batching: every query looks at every key
and the window is a condition on the pair.
"""
import math

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def embed(tokens, table, scale):
    return table[torch.as_tensor(tokens)] * scale


def frequencies(base, dims, scaling):
    """Frequency of every pair; a wave longer than original / low is slowed by factor, one shorter than
    original / high keeps its frequency, between the two both are blended."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            wave = 2 * math.pi / f
            short, long_ = scaling["original"] / scaling["high"], scaling["original"] / scaling["low"]
            if wave > long_:
                f = f / scaling["factor"]
            elif wave >= short:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate(x, positions, rot):
    """x [T, ..., d]: element i of the first rot.dims turns with element i + dims / 2, the rest stays."""
    n, half = rot["dims"], rot["dims"] // 2
    f = torch.tensor(frequencies(rot["base"], n, rot.get("scaling")), dtype=x.dtype)
    ang = torch.as_tensor(positions, dtype=x.dtype)[:, None] * f
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    c, s = ang.cos().reshape(shape), ang.sin().reshape(shape)
    u, v = x[..., :half], x[..., half:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


def window_attention(q, k, v, scale, sink, window, offset=0):
    """One head: q [T, d], k [S, d], v [S, e]; query i stands at position offset + i and sees key j when
    0 <= offset + i - j < window.  The sink adds exp(sink) to the denominator and nothing to the numerator."""
    out = []
    for i in range(q.shape[0]):
        p = offset + i
        lo = max(0, p - window + 1)
        s = (k[lo:p + 1] @ q[i]) * scale
        top = max(float(s.max()), float(sink))
        e = torch.exp(s - top)
        out.append((e @ v[lo:p + 1]) / (e.sum() + torch.exp(sink - top)))
    return torch.stack(out)


def projections(h, w, p, mx, kind, positions, eps):
    """Queries [T, H, dim], keys [T, G, dim], values [T, G, vdim] as attention uses them."""
    H, G = mx["heads"], mx["kv_heads"]
    q = (h @ w[p + "q"].T).reshape(-1, H, mx["dim"])
    k = (h @ w[p + "k"].T).reshape(-1, G, mx["dim"])
    v = (h @ w[p + "v"].T).reshape(-1, G, mx["vdim"])
    if kind == "attention_2":
        q = rotate(rms_norm(q, w[p + "q.norm"], eps), positions, mx["rot"])
        k = rotate(rms_norm(k, w[p + "k.norm"], eps), positions, mx["rot"])
    return q, k, v


def attention_heads(q, k, v, sink, mx, offset=0):
    """[T, H, vdim]; head h reads key / value head h // (H / G)."""
    H, per = mx["heads"], mx["heads"] // mx["kv_heads"]
    return torch.stack([window_attention(q[:, h], k[:, h // per], v[:, h // per], mx["scale"], sink[h], mx["mask"]["size"], offset)
                        for h in range(H)], 1)


def output_gate(o, h, w, p, kind):
    """o [T, H, vdim] times a sigmoid: one gate per number ("attention"), or one per head ("attention_2")."""
    g = torch.sigmoid(h @ w[p + "g"].T)
    return o * (g[..., None] if kind == "attention_2" else g.reshape(o.shape))


def mixer(h, w, p, mx, kind, positions, eps):
    q, k, v = projections(h, w, p, mx, kind, positions, eps)
    o = output_gate(attention_heads(q, k, v, w[p + "sink"], mx), h, w, p, kind)
    return o.flatten(1) @ w[p + "o"].T


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def gated_unit(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, top):
    """Per token the chosen experts and their weights (softmax over the chosen logits)."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    out = []
    for row in z:
        order = sorted(range(len(row)), key=lambda e: -float(row[e]))[:top]
        m = max(float(row[e]) for e in order)
        ex = [math.exp(float(row[e]) - m) for e in order]
        out.append([(e, x / sum(ex)) for e, x in zip(order, ex)])
    return out


def call_margins(h, w, p, top):
    """Per token, how far the last chosen expert's logit is above the best one left out."""
    z = (h @ w[p + "router"].T + w[p + "router.b"]).sort(-1, descending=True).values
    return z[:, top - 1] - z[:, top] if top < z.shape[1] else torch.full_like(z[:, 0], math.inf)


def mixture(h, w, p, mlp):
    y = gated_unit(h, w, p + "shared.", silu)
    for t, chosen in enumerate(route(h, w, p, mlp["router"]["top"])):
        for e, weight in chosen:
            y[t] = y[t] + weight * gated_unit(h[t:t + 1], w, f"{p}e{e}.", silu)[0]
    return y


def feed_forward(h, w, p, mlp):
    return gated_unit(h, w, p, gelu_tanh) if mlp["kind"] == "dense" else mixture(h, w, p, mlp)


def softcap(logits, cap):
    return cap * torch.tanh(logits / cap)


def forward(cfg, weights, tokens, dtype=torch.float64, residuals=None, margins=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives x after every layer, ``margins`` the
    ``call_margins`` of every mixture."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    pos = list(range(len(tokens)))
    x = embed(tokens, w["embed"], cfg["embedding"]["scale"])
    for i, layer in enumerate(cfg["layers"]):
        owner = layer.get("weights_of")
        n = f"l{i if owner is None else owner}."
        h = rms_norm(x, 1 + w[n + "norm1"], eps)
        y = mixer(h, w, n + "mix.", layer["mixer"], layer["type"], pos, eps)
        if layer.get("mlp") is not None:
            if margins is not None and layer["mlp"]["kind"] == "moe":
                margins.append(call_margins(h, w, n + "mlp.", layer["mlp"]["router"]["top"]))
            y = y + feed_forward(h, w, n + "mlp.", layer["mlp"])
        x = x + y
        if residuals is not None:
            residuals.append(x)
    x = rms_norm(x, 1 + w["final.norm"], eps)
    return softcap(x @ w["head"].T, cfg["logit_softcap"])


def greedy(cfg, weights, prompt, n, dtype=torch.float64):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(cfg, weights, seq, dtype)[-1].argmax()))
    return seq[len(prompt):]
