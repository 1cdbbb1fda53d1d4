"""Plain restatement of the Potodra decoder for tests: one function per mechanism, loops where loops are clearest,
float64 by default.  Nothing here is shared with the product path.

``forward`` runs a whole sequence at once; there is no cache, no state that outlives the call and no batching: every
query looks at every key and what it may see is a condition on the pair; recurrences go token by token.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def embed(tokens, table, scale):
    return table[torch.as_tensor(tokens)] * scale


# ---------------------------------------------------------------- hyper-connections
def streams_read(xs, w_in):
    """xs [T, s, d] -> the sublayer's input [T, d]."""
    return sum(w_in[s] * xs[:, s] for s in range(xs.shape[1]))


def streams_write(xs, mix, w_out, y):
    """mix is [from, to]; every stream gains the sublayer's result."""
    n = xs.shape[1]
    return torch.stack([sum(mix[s, t] * xs[:, s] for s in range(n)) + w_out[t] * y for t in range(n)], 1)


# ---------------------------------------------------------------- attention
def rotate(x, positions, rot, neighbours):
    """x [T, heads, d]; pair i is (i, i + dims / 2), or (2 i, 2 i + 1) with ``neighbours``."""
    out = x.clone()
    n = rot["dims"]
    for i in range(n // 2):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + n // 2)
        ang = torch.as_tensor(positions, dtype=x.dtype) * rot["base"] ** (-2.0 * i / n)
        c, s = ang.cos()[:, None], ang.sin()[:, None]
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


def visible(i, j, mask):
    """mask None: all keys up to one's own; else a window and the first tokens."""
    return j <= i and (mask is None or i - j < mask["size"] or j < mask.get("keep_first", 0))


def attend(q, k, v, scale, cap=None, sink=None, mask=None, offset=0):
    """One head: q [T, d] at positions offset ..., k [S, d], v [S, e]."""
    out = []
    for i in range(q.shape[0]):
        p = offset + i
        see = torch.tensor([visible(p, j, mask) for j in range(k.shape[0])])
        s = (k[see] @ q[i]) * scale
        if cap is not None:
            s = cap * torch.tanh(s / cap)
        top = float(s.max()) if sink is None else max(float(s.max()), float(sink))
        e = torch.exp(s - top)
        den = e.sum() if sink is None else e.sum() + torch.exp(sink - top)
        out.append((e @ v[see]) / den)
    return torch.stack(out)


def attention(h, w, p, mx, positions, neighbours, sink):
    H, G = mx["heads"], mx["kv_heads"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(-1, H, mx["dim"])
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(-1, G, mx["dim"])
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(-1, G, mx["vdim"])
    q, k = (rotate(x, positions, mx["rot"], neighbours) for x in (q, k))
    o = [attend(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], mx["scale"], mx.get("softcap"), sink[i] if sink is not None else None,
                mx.get("mask")) for i in range(H)]
    return torch.cat(o, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- matrix memory with exponential gates
def mlstm_memory(q, k, v, i, f):
    """One head: q, k [T, d], v [T, e], log gates i, f [T] -> (o [T, e], state (S, n, m))."""
    S, n, m = q.new_zeros(q.shape[1], v.shape[1]), q.new_zeros(q.shape[1]), q.new_zeros(())
    out = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep * S + put * torch.outer(k[t], v[t])
        n = keep * n + put * k[t]
        m = new
        out.append((q[t] @ S) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(out), (S, n, m)


def mlstm_gates(h, w, p, cap):
    """Log input and forget gates [T, heads]."""
    squash = lambda name: cap * torch.tanh((h @ w[p + name].T + w[p + name + ".b"]) / cap)
    return squash("i"), -softplus(-squash("f"))


def mlstm(h, w, p, mx, eps):
    H, d, e = mx["heads"], mx["dim"], mx["vdim"]
    q, k = (h @ w[p + "q"].T).reshape(-1, H, d) * d ** -0.5, (h @ w[p + "k"].T).reshape(-1, H, d)
    v = (h @ w[p + "v"].T).reshape(-1, H, e)
    i, f = mlstm_gates(h, w, p, mx["gate_cap"])
    o = torch.cat([rms(mlstm_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a])[0], eps) for a in range(H)], -1)
    return (o * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---------------------------------------------------------------- gated delta rule
def short_conv(x, taps):
    """x [T, c], taps [c, n]: causal, per channel, zeros before the start; then silu."""
    n = taps.shape[1]
    wide = torch.cat([x.new_zeros(n - 1, x.shape[1]), x])
    return silu(sum(wide[j:j + x.shape[0]] * taps[:, j] for j in range(n)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_memory(q, k, v, g, beta):
    """One head: q, k, g [T, d], v [T, e], beta [T] -> (o [T, e], S)."""
    S, out = q.new_zeros(q.shape[1], v.shape[1]), []
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        S = S + torch.outer(k[t], beta[t] * (v[t] - k[t] @ S))
        out.append(q[t] @ S)
    return torch.stack(out), S


def delta(h, w, p, mx, eps):
    H, G, d, e = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = unit(short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).reshape(-1, G, d)) * d ** -0.5
    k = unit(short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).reshape(-1, G, d))
    v = short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).reshape(-1, H, e)
    beta = sigmoid(h @ w[p + "b"].T)
    step = softplus(h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(-1, H, d)
    g = torch.exp(-torch.exp(w[p + "A_log"])[:, None] * step)
    gate = sigmoid(h @ w[p + "g1"].T @ w[p + "g2"].T).reshape(-1, H, e)
    per = H // G
    o = [rms(delta_memory(q[:, a // per], k[:, a // per], v[:, a], g[:, a], beta[:, a])[0], eps) * w[p + "norm"] * gate[:, a] for a in range(H)]
    return torch.cat(o, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward
def dense(h, w, p):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def clamped_unit(h, w, p, limit):
    g = (h @ w[p + "gate"].T).clamp(max=limit)
    u = (h @ w[p + "up"].T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def choose(s, correction, top, groups):
    """One token: experts by s + correction among the best groups; returns (experts, how close the choice was)."""
    c = s + correction
    n, size = groups["count"], c.shape[0] // groups["count"]
    score = torch.stack([c[g * size:(g + 1) * size].sort(descending=True).values[:2].sum() for g in range(n)])
    order = score.sort(descending=True)
    kept = order.indices[:groups["keep"]].tolist()
    margin = float(order.values[groups["keep"] - 1] - order.values[groups["keep"]]) if groups["keep"] < n else math.inf
    open_ = [e for e in range(c.shape[0]) if e // size in kept]
    ranked = sorted(open_, key=lambda e: -float(c[e]))
    if top < len(ranked):
        margin = min(margin, float(c[ranked[top - 1]] - c[ranked[top]]))
    return ranked[:top], margin


def mixture(h, w, p, m, margins=None):
    s = sigmoid(h @ w[p + "router"].T)
    y = sigmoid(h @ w[p + "shared.sg"].T) * clamped_unit(h, w, p + "shared.", m["shared"]["limit"])
    rows, close = [], []
    for t in range(h.shape[0]):
        chosen, margin = choose(s[t], w[p + "correction"], m["router"]["top"], m["router"]["groups"])
        close.append(margin)
        rows.append(y[t] + sum(s[t, e] * clamped_unit(h[t:t + 1], w, f"{p}e{e}.", m["expert"]["limit"])[0] for e in chosen))
    if margins is not None:
        margins.append(torch.tensor(close))
    return torch.stack(rows)


# ---------------------------------------------------------------- the model
def mixer(h, w, p, layer, eps):
    mx, positions = layer["mixer"], list(range(h.shape[0]))
    if layer["type"] == "attention":
        return attention(h, w, p, mx, positions, False, w[p + "sink"])
    if layer["type"] == "mlstm":
        return mlstm(h, w, p, mx, eps)
    assert layer["type"] == "parallel"
    return mx["left_scale"] * attention(h, w, p + "left.", mx["left"], positions, True, None) + \
        mx["right_scale"] * delta(h, w, p + "right.", mx["right"], eps)


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None, margins=None):
    """Logits [T, vocab]; ``layers_out`` collects the sum of the streams after every layer, ``margins`` how close the
    choices of experts were, [T] per mixture."""
    w = {k: t.to(dtype) for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, w["embed"], cfg["embedding"]["scale"])
    xs = torch.stack([x] * cfg["streams"], 1)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."

        def sublayer(xs, q, f):
            hc = f"{p}hc{q}."
            y = f(rms(streams_read(xs, w[hc + "in"]), eps) * w[f"{p}norm{q}"])
            return streams_write(xs, w[hc + "mix"], w[hc + "out"], y)

        xs = sublayer(xs, 1, lambda h: mixer(h, w, p + "mix.", layer, eps))
        m = layer.get("mlp")
        if m is not None:
            xs = sublayer(xs, 2, lambda h: dense(h, w, p + "mlp.") if m["kind"] == "dense" else mixture(h, w, p + "mlp.", m, margins))
        if layers_out is not None:
            layers_out.append(xs.sum(1))
    return (rms(xs.sum(1), eps) * w["final.norm"]) @ w["embed"].T
