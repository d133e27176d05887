"""Plain, slow statement of the Nipulorn design, one function per mechanism, for the tests.

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


def input_conv(h, taps):
    """h_t + sum_j taps[:, j] * h_(t - n + 1 + j), zeros in front of the sequence."""
    T, n = h.shape[0], taps.shape[1]
    y = h.clone()
    for j in range(n):
        back = n - 1 - j
        if back < T:
            y[back:] += taps[:, j] * h[:T - back]
    return y


def token_mix(h, mu):
    """h + (previous token's h - h) * mu."""
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (prev - h) * mu


def silu(z):
    return z / (1.0 + torch.exp(-z))


def decay(h, w, name):
    """Per key channel, between 0 and 1."""
    low = torch.tanh(token_mix(h, w[name + ".mu.w"]) @ w[name + ".w1"].T)
    return torch.exp(-torch.exp(low @ w[name + ".w2"].T + w[name + ".w0"]))


def wkv_recurrence(r, k, v, d, u):
    """r, k, v, d [T, heads, dim], u [heads, dim] -> [T, heads, dim].  The state holds one row per key channel."""
    T, H, D = r.shape
    out = torch.zeros_like(v)
    S = torch.zeros(H, D, D, dtype=r.dtype)
    for t in range(T):
        kv = k[t, :, :, None] * v[t, :, None, :]
        out[t] = ((S + u[:, :, None] * kv) * r[t, :, :, None]).sum(1)
        S = d[t, :, :, None] * S + kv
    return out


def wkv_mixer(h, w, name, mx, eps):
    T, shape = h.shape[0], (h.shape[0], mx["heads"], mx["dim"])
    r, k, v = ((token_mix(h, w[f"{name}.mu.{c}"]) @ w[f"{name}.{c}"].T).reshape(shape) for c in "rkv")
    gate = silu(token_mix(h, w[name + ".mu.g"]) @ w[name + ".g"].T)
    o = wkv_recurrence(r, k, v, decay(h, w, name).reshape(shape), w[name + ".u"])
    return (rms(o, eps).reshape(T, -1) * w[name + ".norm"] * gate) @ w[name + ".o"].T


def yarn_frequencies(rot):
    """(frequency per rotated pair, factor on cosine and sine)."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if sc is None:
        return f, 1.0
    dim = lambda turns: n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(v, positions, rot):
    """v [T, ..., n]: adjacent pairs (2i, 2i + 1) of the first ``dims`` entries turn by p * f_i."""
    y = v.clone()
    freq, gain = yarn_frequencies(rot)
    for i, f in enumerate(freq):
        a = (positions.to(v.dtype) * f).reshape(-1, *([1] * (v.dim() - 2)))
        c, s = torch.cos(a) * gain, torch.sin(a) * gain
        p, q = v[..., 2 * i], v[..., 2 * i + 1]
        y[..., 2 * i] = p * c - q * s
        y[..., 2 * i + 1] = q * c + p * s
    return y


def sink_softmax(scores, sink):
    """Softmax over the last axis with one more term exp(sink) in the denominator that has no value."""
    m = torch.maximum(scores.max(-1, keepdim=True).values, sink)
    e = torch.exp(scores - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def latent_attention(qn, qr, c, kr, wuk, wuv, sink, scale):
    """qn [T, H, dim], qr [T, H, rot], latents c [S, rank], shared rotated keys kr [S, rot], wuk [H, dim, rank],
    wuv [H, vdim, rank]; the queries are the last T of the S positions and see everything up to their own.
    -> [T, H, vdim]."""
    T, H, S = qn.shape[0], qn.shape[1], c.shape[0]
    out = torch.zeros(T, H, wuv.shape[1], dtype=qn.dtype)
    later = torch.arange(S)[None, :] > torch.arange(S - T, S)[:, None]
    for h in range(H):
        k, v = c @ wuk[h].T, c @ wuv[h].T
        scores = (qn[:, h] @ k.T + qr[:, h] @ kr.T) * scale
        out[:, h] = sink_softmax(scores.masked_fill(later, -math.inf), sink[h]) @ v
    return out


def latent_mixer(h, w, name, mx, eps):
    T, H, dim, R = h.shape[0], mx["heads"], mx["dim"], mx["kv_rank"]
    pos = torch.arange(T)
    cq = rms(h @ w[name + ".dq"].T, eps) * w[name + ".dq.norm"]
    q = (cq @ w[name + ".uq"].T).reshape(T, H, dim + mx["rot_dim"])
    low = h @ w[name + ".dkv"].T
    c = rms(low[:, :R], eps) * w[name + ".dkv.norm"]
    o = latent_attention(q[..., :dim], rotate(q[..., dim:], pos, mx["rot"]), c, rotate(low[:, R:], pos, mx["rot"]),
                         w[name + ".uk"].reshape(H, dim, R), w[name + ".uv"].reshape(H, mx["vdim"], R), w[name + ".sink"],
                         mx["scale"])
    return o.reshape(T, -1) @ w[name + ".o"].T


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def xielu(z, p, q):
    """Quadratic above zero, exponential below, slope one half at zero on both sides."""
    up = softplus(p) * z ** 2 + z / 2
    down = (0.5 + softplus(q)) * (torch.expm1(z) - z) + z / 2
    return torch.where(z > 0, up, down)


def feed_forward(h, w, name):
    p, q = w[name + ".act"]
    return xielu(h @ w[name + ".up"].T, p, q) @ w[name + ".down"].T


MIXERS = {"wkv": wkv_mixer, "latent_attention": latent_mixer}


def forward(cfg, weights, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [T, vocab] (and the residual stream after every layer) of one whole sequence."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    after = []
    for i, lay in enumerate(cfg["layers"]):
        L = f"l{i}."
        h = input_conv(norm(x, w[L + "norm1"], eps), w[L + "canon1"])
        x = x + norm(MIXERS[lay["type"]](h, w, L + "mix", lay["mixer"], eps), w[L + "norm1b"], eps)
        if lay.get("mlp") is not None:
            h = input_conv(norm(x, w[L + "norm2"], eps), w[L + "canon2"])
            x = x + norm(feed_forward(h, w, L + "mlp"), w[L + "norm2b"], eps)
        after.append(x)
    logits = norm(x, w["final.norm"], eps) @ w["embed"].T * cfg["logit_scale"]
    return (logits, torch.stack(after)) if keep_layers else logits
