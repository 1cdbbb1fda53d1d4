"""Plain restatement of the Zidalix decoder for tests: one function per mechanism, loops where loops are
clearest, float64 by default.  Nothing here is shared with the product path.

``forward`` runs a whole sequence at once; there is no cache, no batching and no absorbed form: keys and
values of every head are written out and every query looks at every key.
"""
import math

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def embed(tokens, table, scale):
    return table[torch.as_tensor(tokens)] * scale


def yarn(base, dims, scaling):
    """Per-pair frequencies and the factor on cos / sin.  ``scaling`` None: plain rotary."""
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freqs, 1.0

    def turns_to_dim(t):
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo = max(math.floor(turns_to_dim(scaling["fast"])), 0)
    hi = min(math.ceil(turns_to_dim(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, ..., dims]; neighbouring elements (2i, 2i+1) form pair i."""
    freqs, m = yarn(rot["base"], rot["dims"], rot.get("scaling"))
    ang = torch.as_tensor(positions, dtype=x.dtype)[:, None] * torch.tensor(freqs, dtype=x.dtype)
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [len(freqs)]
    c, s = (ang.cos() * m).reshape(shape), (ang.sin() * m).reshape(shape)
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)


def latents(h, w, p, mx, positions, eps):
    """The normed latent [T, kv_rank] and the rotated shared key part [T, rot_dim] of the tokens of h."""
    z = h @ w[p + "dkv"].T
    c = rms_norm(z[:, :mx["kv_rank"]], w[p + "dkv.norm"], eps)
    return c, rotate(z[:, mx["kv_rank"]:], positions, mx["rot"])


def sink_attention(q, k, v, scale, sink, offset=0):
    """One head: q [T, d], k [S, d], v [S, e]; query i (position offset + i) sees keys 0 .. offset + i.  The
    sink adds exp(sink) to the denominator and nothing to the numerator."""
    out = []
    for i in range(q.shape[0]):
        s = (k[:offset + i + 1] @ q[i]) * scale
        top = max(float(s.max()), float(sink))
        e = torch.exp(s - top)
        out.append((e @ v[:offset + i + 1]) / (e.sum() + torch.exp(sink - top)))
    return torch.stack(out)


def attention_core(q, c, kr, w, p, mx, offset=0):
    """Heads before gate and output projection: q [T, H, dim + rot_dim] (rotated), c / kr of all keys."""
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    k_n = (c @ w[p + "uk"].T).reshape(-1, H, D)
    vals = (c @ w[p + "uv"].T).reshape(-1, H, V)
    heads = [sink_attention(q[:, h], torch.cat([k_n[:, h], kr], -1), vals[:, h], mx["scale"], w[p + "sink"][h], offset)
             for h in range(H)]
    return torch.cat(heads, -1)


def queries(h, w, p, mx, positions):
    q = (h @ w[p + "q"].T).reshape(-1, mx["heads"], mx["dim"] + mx["rot_dim"])
    return torch.cat([q[..., :mx["dim"]], rotate(q[..., mx["dim"]:], positions, mx["rot"])], -1)


def output_gate(o, h, w, p):
    return o * torch.sigmoid(h @ w[p + "g"].T)


def clamped_glu(h, w, p, limit):
    g, u = h @ w[p + "gate"].T, h @ w[p + "up"].T
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def forward(cfg, weights, tokens, dtype=torch.float64, residuals=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives x after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    pos = list(range(len(tokens)))
    x = embed(tokens, w["embed"], cfg["embedding"]["scale"])
    store = {}
    for i, layer in enumerate(cfg["layers"]):
        n, mx = f"l{i}.", layer["mixer"]
        p = n + "mix."
        h = rms_norm(x, w[n + "norm1"], eps)
        q = queries(h, w, p, mx, pos)
        if mx.get("kv_from") is None:
            store[i] = latents(h, w, p, mx, pos, eps)
        c, kr = store[i if mx.get("kv_from") is None else mx["kv_from"]]
        o = attention_core(q, c, kr, w, p, mx)
        y = output_gate(o, h, w, p) @ w[p + "o"].T
        if layer.get("mlp") is not None:
            y = y + clamped_glu(rms_norm(x, w[n + "norm2"], eps), w, n + "mlp.", layer["mlp"]["limit"])
        x = x + y
        if residuals is not None:
            residuals.append(x)
    x = rms_norm(x, w["final.norm"], eps)
    return (x @ w["head"].T) * cfg["logit_scale"]


def greedy(cfg, weights, prompt, n, dtype=torch.float64):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(cfg, weights, seq, dtype)[-1].argmax()))
    return seq[len(prompt):]
