"""Plain, slow statement of the Tasadra design, one function per mechanism, for the tests.

Everything is a direct loop-or-matrix form of the equations on CPU tensors (float64 unless the caller passes another
dtype).  It shares no code with the package: configurations are plain dictionaries, weights a dictionary of tensors,
and there is no cache and no carried state -- a sequence is always evaluated from its first token.

Notation: x is the residual stream [T, width]; h what a sublayer reads; p the position of a token; W @ h for linear
maps stored [out, in].
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps)


def dyt(x, w, name):
    """Dynamic Tanh: a squashing with one learned slope instead of a norm."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def token_shift(h, mix):
    """h_t + (h_(t-1) - h_t) * mix, nothing (zeros) in front of the first token."""
    back = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (back - h) * mix


def yarn_frequencies(rot):
    """(frequencies of the pairs, gain on sine and cosine)."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if sc is None:
        return f, 1.0
    dim = lambda turns: n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def turn(v, positions, freqs, gain=1.0):
    """v [T, heads, n]: with m = len(freqs), entries i and i + m of the first 2 m turn by p * f_i, the rest stay."""
    y, m = v.clone(), len(freqs)
    for i, f in enumerate(freqs):
        a = (positions.to(v.dtype) * f)[:, None]
        c, s = torch.cos(a) * gain, torch.sin(a) * gain
        p, q = v[..., i], v[..., i + m]
        y[..., i] = p * c - q * s
        y[..., i + m] = q * c + p * s
    return y


def value_frequencies(base, vdim):
    return [base ** (-2.0 * m / vdim) for m in range(vdim // 2)]


def softcap(scores, cap):
    return cap * torch.tanh(scores / cap) if cap else scores


def visible(T, chunk=None):
    """[T, T] bool: a query sees itself and what is before it, with chunks only inside its own."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // chunk == j // chunk) if chunk else j <= i


def attend(q, k, v, scale, chunk=None, cap=None):
    """q [T, heads, dim], k / v [T, kv heads, ..] -> [T, heads, vdim]."""
    T, H, g = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    hidden = ~visible(T, chunk)
    for h in range(H):
        s = softcap((q[:, h] @ k[:, h // g].T) * scale, cap)
        out[:, h] = torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, h // g]
    return out


def chunk_of(mx):
    return mx["mask"]["size"] if mx.get("mask") else None


def attention_mixer(h, w, name, mx, eps, kv):
    """Normed and rotated queries and keys, rotated values, one gate per head."""
    T, H, G = h.shape[0], mx["heads"], mx["kv_heads"]
    pos = torch.arange(T)
    q = rms((h @ w[name + ".q"].T).reshape(T, H, mx["dim"]), eps) * w[name + ".q.norm"]
    k = rms((h @ w[name + ".k"].T).reshape(T, G, mx["dim"]), eps) * w[name + ".k.norm"]
    v = (h @ w[name + ".v"].T).reshape(T, G, mx["vdim"])
    freqs, gain = yarn_frequencies(mx["rot"])
    vf = value_frequencies(mx["rot"]["base"], mx["vdim"])
    o = attend(turn(q, pos, freqs, gain), turn(k, pos, freqs, gain), turn(v, pos, vf), mx["scale"], chunk_of(mx), mx.get("softcap"))
    o = turn(o, -pos, vf) * sigmoid(h @ w[name + ".g"].T)[..., None]
    return o.reshape(T, -1) @ w[name + ".o"].T


def difference(a1, a2, lam, diff, eps):
    """Two maps' outputs [.., vdim] into one."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def lambda_of(w, name, diff):
    dot = lambda n: (w[f"{name}.lq{n}"] * w[f"{name}.lk{n}"]).sum()
    return torch.exp(dot(1)) - torch.exp(dot(2)) + diff


def differential_mixer(h, w, name, mx, eps, kv):
    """Two attentions per head over the same values, subtracted; one gate per output channel.  ``kv``: the keys and values of
    the layers so far, for those that have none of their own."""
    T, H, G, D = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    if mx.get("kv_from") is None:
        kv[name] = ((h @ w[name + ".k"].T).reshape(T, G, 2, D), (h @ w[name + ".v"].T).reshape(T, G, mx["vdim"]))
    k, v = kv[name if mx.get("kv_from") is None else f"l{mx['kv_from']}.mix"]
    q = (h @ w[name + ".q"].T).reshape(T, H, 2, D)
    a1, a2 = (attend(q[:, :, m], k[:, :, m], v, mx["scale"], chunk_of(mx)) for m in (0, 1))
    o = difference(a1, a2, lambda_of(w, name, mx["diff"]), mx["diff"], eps)
    return (o.reshape(T, -1) * sigmoid(h @ w[name + ".g"].T)) @ w[name + ".o"].T


def short_conv(y, taps):
    """Causal, per channel: y [T, C], taps [C, n], the last column meets the token itself; zeros in front."""
    T, n = y.shape[0], taps.shape[1]
    out = torch.zeros_like(y)
    for j in range(n):
        back = n - 1 - j
        if back < T:
            out[back:] += taps[:, j] * y[:T - back]
    return out


def unit(x):
    return x / torch.sqrt((x ** 2).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, g, beta):
    """q, k, g [T, heads, dim], v [T, heads, vdim], beta [T, heads] -> [T, heads, vdim].  S [dim, vdim] per head: every row
    decays at its own rate, then the part of v that S does not yet answer k with is written, then q reads."""
    T, H, D = q.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(D, v.shape[-1], dtype=q.dtype)
        for t in range(T):
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + torch.outer(k[t, h], u)
            out[t, h] = S.T @ q[t, h]
    return out


def channel_decay(h, w, name, H, D):
    raw = (h @ w[name + ".a1"].T) @ w[name + ".a2"].T + w[name + ".dt_bias"]
    return torch.exp(-torch.exp(w[name + ".A_log"])[:, None] * softplus(raw).reshape(-1, H, D))


def delta_mixer(h, w, name, mx, eps, kv):
    T, H, G, D = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    q, k, v = (silu(short_conv(h @ w[f"{name}.{c}"].T, w[f"{name}.{c}.conv"])) for c in "qkv")
    rep = lambda x: unit(x.reshape(T, G, D)).repeat_interleave(H // G, dim=1)
    beta = sigmoid(h @ w[name + ".b"].T)
    o = delta_recurrence(rep(q) * D ** -0.5, rep(k), v.reshape(T, H, mx["vdim"]), channel_decay(h, w, name, H, D), beta)
    gate = sigmoid((h @ w[name + ".g1"].T) @ w[name + ".g2"].T)
    return ((rms(o, eps) * w[name + ".norm"]).reshape(T, -1) * gate) @ w[name + ".o"].T


MIXERS = {"attention": attention_mixer, "channel_delta": delta_mixer, "attention_2": differential_mixer}


def feed_forward(h, w, name):
    """Squared relu between two maps with biases."""
    up = torch.clamp(h @ w[name + ".up"].T + w[name + ".up.b"], min=0.0)
    return up ** 2 @ w[name + ".down"].T + w[name + ".down.b"]


def depth_average(streams, weights):
    """Weighted sum of the embedding output and all layers' results so far."""
    return sum(weights[j] * s for j, s in enumerate(streams))


def forward(cfg, weights, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [T, vocab] (and the residual stream after every layer) of one whole sequence."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.tensor(tokens)]
    streams, after, kv = [x], [], {}
    for i, lay in enumerate(cfg["layers"]):
        L = f"l{i}."
        h = token_shift(dyt(x, w, L + "norm1"), w[L + "shift"])
        x = x + m * MIXERS[lay["type"]](h, w, L + "mix", lay["mixer"], eps, kv)
        if lay.get("mlp") is not None:
            x = x + m * feed_forward(dyt(x, w, L + "norm2"), w, L + "mlp")
        streams.append(x)
        x = depth_average(streams, w[L + "dwa"])
        after.append(x)
    logits = dyt(x, w, "final.norm") @ w["head"].T
    return (logits, torch.stack(after)) if keep_layers else logits
