"""Plain restatement of the Lerosun decoder for tests: one function per mechanism, loops where loops are clearest,
float64 by default.  Nothing here is shared with the product path.

``forward`` runs a whole sequence at once; there is no cache, no state that outlives the call and no batching: every
query looks at every key and what it may see is a condition on the pair; the recurrence goes token by token.
"""
import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def embed(tokens, table, g, eps):
    return rms(table[torch.as_tensor(tokens)], eps) * g


# ---------------------------------------------------------------- attention
def rotate(x, positions, rot):
    """x [T, heads, d]; dimension i turns with i + dims / 2."""
    out = x.clone()
    n = rot["dims"]
    for i in range(n // 2):
        ang = torch.as_tensor(positions, dtype=x.dtype) * rot["base"] ** (-2.0 * i / n)
        c, s = ang.cos()[:, None], ang.sin()[:, None]
        out[..., i] = x[..., i] * c - x[..., i + n // 2] * s
        out[..., i + n // 2] = x[..., i + n // 2] * c + x[..., i] * s
    return out


def scores(q, k, scale, temp):
    """q [T, H, d], k [S, G, d] -> [H, T, S], before the heads talk."""
    H, G = q.shape[1], k.shape[1]
    return torch.stack([(q[:, h] @ k[:, h // (H // G)].T) * scale * temp[h] for h in range(H)])


def talk(s, mix):
    """Every head's scores become a mixture of all heads' scores."""
    H = s.shape[0]
    return torch.stack([sum(mix[h, g] * s[g] for g in range(H)) for h in range(H)])


def visible(i, j, size):
    return 0 <= i - j < size


def attend(s, v, sink, size, offset=0):
    """One head: mixed scores s [T, S] of queries at positions offset ..., values v [S, e]."""
    out = []
    for i in range(s.shape[0]):
        see = torch.tensor([visible(offset + i, j, size) for j in range(v.shape[0])])
        x = s[i][see]
        top = torch.maximum(x.max(), sink)
        e = torch.exp(x - top)
        out.append((e @ v[see]) / (e.sum() + torch.exp(sink - top)))
    return torch.stack(out)


def attention_heads(q, k, mx, w, p, offset=0):
    """Rotation to softmax: q [T, H, d] at positions offset ..., k [S, G, d] from position 0 on -> [T, H, e]."""
    H, G = q.shape[1], k.shape[1]
    qr = rotate(q, [offset + i for i in range(q.shape[0])], mx["rot"])
    kr = rotate(k, list(range(k.shape[0])), mx["rot"])
    s = talk(scores(qr, kr, mx["scale"], w[p + "temp"]), w[p + "talk"])
    return torch.stack([attend(s[h], k[:, h // (H // G)], w[p + "sink"][h], mx["mask"]["size"], offset) for h in range(H)], 1)


def attention(h, w, p, mx):
    H, G = mx["heads"], mx["kv_heads"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(-1, H, mx["dim"])
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(-1, G, mx["dim"])
    o = attention_heads(q, k, mx, w, p) * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.flatten(1) @ w[p + "o"].T


# ---------------------------------------------------------------- gated delta rule
def short_conv(x, taps):
    """x [T, c], taps [c, n]: causal, per channel, zeros before the start; then silu."""
    n = taps.shape[1]
    wide = torch.cat([x.new_zeros(n - 1, x.shape[1]), x])
    return silu(sum(wide[j:j + x.shape[0]] * taps[:, j] for j in range(n)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_memory(q, k, v, g, beta):
    """One head: q, k [T, d], v [T, e], g, beta [T] -> (o [T, e], S)."""
    S, out = q.new_zeros(q.shape[1], v.shape[1]), []
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + torch.outer(k[t], beta[t] * (v[t] - k[t] @ S))
        out.append(q[t] @ S)
    return torch.stack(out), S


def delta(h, w, p, mx, eps):
    H, G, d, e = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = unit(short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).reshape(-1, G, d)) * d ** -0.5
    k = unit(short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).reshape(-1, G, d))
    v = short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).reshape(-1, H, e)
    beta = sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    gate = silu(h @ w[p + "g"].T).reshape(-1, H, e)
    per = H // G
    o = [rms(delta_memory(q[:, a // per], k[:, a // per], v[:, a], g[:, a], beta[:, a])[0], eps) * w[p + "norm"] * gate[:, a] for a in range(H)]
    return torch.cat(o, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward
def dense(h, w, p):
    return (torch.relu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ---------------------------------------------------------------- the model
def order(cfg):
    """Layer numbers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab]; ``layers_out`` collects the residual after every layer run."""
    w = {k: t.to(dtype) for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, w["embed"], w["embed.norm"], eps)
    for i in order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        h = rms(x, eps) * w[p + "norm1"]
        y = attention(h, w, p + "mix.", layer["mixer"]) if layer["type"] == "attention" else delta(h, w, p + "mix.", layer["mixer"], eps)
        x = x + w[p + "ls1"] * y
        if layer.get("mlp") is not None:
            x = x + w[p + "ls2"] * dense(rms(x, eps) * w[p + "norm2"], w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T
