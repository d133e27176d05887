"""Plain, slow statement of the Bakasun design, one function per mechanism, for the tests.

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


def norm(x, w, eps):
    """Root-mean-square norm whose stored weight is the distance from one."""
    return rms(x, eps) * (1.0 + w)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(v, positions, rot):
    """v [T, heads, n]: entries i and i + dims / 2 of the first ``dims`` turn by p * f_i, the rest stay."""
    y, n = v.clone(), rot["dims"]
    slow = rot["scaling"]["factor"] if rot.get("scaling") else 1.0
    for i in range(n // 2):
        a = (positions.to(v.dtype) * (rot["base"] ** (-2.0 * i / n) / slow))[:, None]
        c, s = torch.cos(a), torch.sin(a)
        p, q = v[..., i], v[..., i + n // 2]
        y[..., i] = p * c - q * s
        y[..., i + n // 2] = q * c + p * s
    return y


def off_by_one_softmax(scores):
    """Softmax over the last axis whose denominator has one more term, exp(0), without a value."""
    m = torch.clamp(scores.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(scores - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-m))


def softcap(scores, cap):
    return cap * torch.tanh(scores / cap)


def visible(T, size):
    """[T, T] bool: a query sees itself and the size - 1 tokens before it (everything before it without a size)."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < size) if size else back >= 0


def attend(q, k, v, scale, size=None, cap=None):
    """q [T, heads, dim], k / v [T, kv heads, ..] -> [T, heads, vdim]."""
    T, H, g = q.shape[0], q.shape[1], q.shape[1] // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    hidden = ~visible(T, size)
    for h in range(H):
        s = (q[:, h] @ k[:, h // g].T) * scale
        if cap is not None:
            s = softcap(s, cap)
        out[:, h] = off_by_one_softmax(s.masked_fill(hidden, -math.inf)) @ v[:, h // g]
    return out


def linear(h, w, name):
    y = h @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


def attention(h, w, name, mx, eps, bias, qk_norm):
    T = h.shape[0]
    lin = linear if bias else (lambda h, w, n: h @ w[n].T)
    q, k, v = (lin(h, w, f"{name}.{c}") for c in "qkv")
    if qk_norm:                                   # over all rows of the projection at once
        q, k = rms(q, eps) * w[name + ".q.norm"], rms(k, eps) * w[name + ".k.norm"]
    q, k = q.reshape(T, mx["heads"], mx["dim"]), k.reshape(T, mx["kv_heads"], mx["dim"])
    pos = torch.arange(T)
    if mx.get("rot"):
        q, k = rotate(q, pos, mx["rot"]), rotate(k, pos, mx["rot"])
    o = attend(q, k, v.reshape(T, mx["kv_heads"], mx["vdim"]), mx["scale"], mx["mask"]["size"] if mx.get("mask") else None,
               mx.get("softcap"))
    return o.reshape(T, -1) @ w[name + ".o"].T


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
    """q, k [T, heads, dim], v [T, heads, vdim], g, beta [T, heads] -> [T, heads, vdim].  S [dim, vdim] per head: decay, then
    the part of v that S does not yet answer k with is written, then q reads."""
    T, H, D = q.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(D, v.shape[-1], dtype=q.dtype)
        for t in range(T):
            S = g[t, h] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + torch.outer(k[t, h], u)
            out[t, h] = S.T @ q[t, h]
    return out


def delta_mixer(h, w, name, mx, eps):
    T, H, G, D = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    q, k, v = (silu(short_conv(h @ w[f"{name}.{c}"].T, w[f"{name}.{c}.conv"])) for c in "qkv")
    rep = lambda x: unit(x.reshape(T, G, D)).repeat_interleave(H // G, dim=1)
    beta = sigmoid(h @ w[name + ".b"].T)
    g = torch.exp(-torch.exp(w[name + ".A_log"]) * softplus(h @ w[name + ".a"].T + w[name + ".dt_bias"]))
    o = delta_recurrence(rep(q) * D ** -0.5, rep(k), v.reshape(T, H, mx["vdim"]), g, beta)
    gate = silu(h @ w[name + ".g"].T)
    return ((rms(o, eps) * w[name + ".norm"]).reshape(T, -1) * gate) @ w[name + ".o"].T


def attention_mixer(h, w, name, mx, eps):
    return attention(h, w, name, mx, eps, bias=False, qk_norm=True)


def parallel_mixer(h, w, name, mx, eps):
    return mx["left_scale"] * attention(h, w, name + ".left", mx["left"], eps, bias=True, qk_norm=False) + \
        mx["right_scale"] * delta_mixer(h, w, name + ".right", mx["right"], eps)


MIXERS = {"attention": attention_mixer, "parallel": parallel_mixer}


def gated(h, w, name, act):
    return (act(h @ w[name + ".gate"].T) * (h @ w[name + ".up"].T)) @ w[name + ".down"].T


def choose(choice, top, groups):
    """Indices of the ``top`` largest entries of a vector, looked for in the best groups of neighbours only."""
    if groups:
        size = len(choice) // groups["count"]
        best = sorted(range(groups["count"]), key=lambda i: -float(choice[i * size:(i + 1) * size].max()))[:groups["keep"]]
        open_ = [e for e in range(len(choice)) if e // size in best]
    else:
        open_ = list(range(len(choice)))
    return sorted(open_, key=lambda e: -float(choice[e]))[:top]


def mixture(h, w, name, mlp):
    r = mlp["router"]
    s = torch.softmax(h @ w[name + ".router"].T, -1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose(s[t] + w[name + ".correction"], r["top"], r.get("groups"))
        total = sum(s[t, e] for e in ids) + 1e-20
        for e in ids:
            out[t] += s[t, e] / total * gated(h[t], w, f"{name}.e{e}", silu)
    if mlp.get("shared"):
        out = out + sigmoid(h @ w[name + ".shared.sg"].T) * gated(h, w, name + ".shared", silu)
    return out


def feed_forward(h, w, name, mlp):
    return gated(h, w, name, gelu_tanh) if mlp["kind"] == "dense" else mixture(h, w, name, mlp)


def forward(cfg, weights, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [T, vocab] (and the residual stream after every layer) of one whole sequence."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    after = []
    for i, lay in enumerate(cfg["layers"]):
        L = f"l{i}."
        x = x + norm(MIXERS[lay["type"]](norm(x, w[L + "norm1"], eps), w, L + "mix", lay["mixer"], eps), w[L + "norm1b"], eps)
        if lay.get("mlp") is not None:
            x = x + norm(feed_forward(norm(x, w[L + "norm2"], eps), w, L + "mlp", lay["mlp"]), w[L + "norm2b"], eps)
        after.append(x)
    logits = norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(after)) if keep_layers else logits
