"""Plain, slow statement of the Gekapel design, one function per mechanism, for the tests.

Everything is a direct loop-or-matrix form of the equations on CPU tensors (float64 unless the caller passes another
dtype).  It shares no code with the package: configurations are plain dictionaries, weights a dictionary of tensors,
and there is no cache -- a sequence is always evaluated from its first token.

Notation: x is the residual stream [T, width]; p the position of a token; W @ h for linear maps stored [out, in].
"""
import math

import torch


def layer_norm(x, w, b, eps):
    """(x - mean) / sqrt(var + eps) * w + b with the population variance."""
    mu = x.mean(-1, keepdim=True)
    var = ((x - mu) ** 2).mean(-1, keepdim=True)
    return (x - mu) / torch.sqrt(var + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps) * w


def rotary_frequencies(rot):
    """One frequency per rotated pair; long wavelengths are slowed down by ``factor`` with a linear blend between
    the two wavelength bounds."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc is not None:
            wave = 2.0 * math.pi / f
            if wave < sc["original"] / sc["high"]:
                pass
            elif wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            else:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(v, positions, rot):
    """v [T, heads, dim]: adjacent pairs (2i, 2i + 1) of the first ``dims`` entries turn by p * f_i."""
    y = v.clone()
    for i, f in enumerate(rotary_frequencies(rot)):
        a = positions.to(v.dtype) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, w = v[..., 2 * i], v[..., 2 * i + 1]
        y[..., 2 * i] = u * c - w * s
        y[..., 2 * i + 1] = w * c + u * s
    return y


def keys_values(h, w, name, mx, eps, positions):
    """Normalised, rotated keys [T, G, dim] and values [T, G, vdim] of a layer that has its own."""
    T = h.shape[0]
    k = (h @ w[name + ".k"].T).reshape(T, mx["kv_heads"], mx["dim"])
    v = (h @ w[name + ".v"].T).reshape(T, mx["kv_heads"], mx["vdim"])
    k = rotate(rms_norm(k, w[name + ".k.norm"], eps), positions, mx["rot"])
    return k, v


def queries(h, w, name, mx, eps, positions):
    q = (h @ w[name + ".q"].T).reshape(h.shape[0], mx["heads"], mx["dim"])
    return rotate(rms_norm(q, w[name + ".q.norm"], eps), positions, mx["rot"])


def sink_softmax(scores, sink):
    """Softmax over the last axis with one more term exp(sink) in the denominator that has no value."""
    m = torch.maximum(scores.max(), sink)
    e = torch.exp(scores - m)
    return e / (e.sum() + torch.exp(sink - m))


def window_attention(q, k, v, sink, scale, size):
    """Query i sees keys i - size + 1 .. i; query head h reads key/value head h // (H / G).  [T, H, vdim]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // per
        for i in range(T):
            lo = 0 if size is None else max(0, i - size + 1)
            sc = (k[lo:i + 1, g] @ q[i, h]) * scale
            out[i, h] = sink_softmax(sc, sink[h]) @ v[lo:i + 1, g]
    return out


def relu2(z):
    return torch.clamp(z, min=0.0) ** 2


def expert(h, up, down):
    return relu2(h @ up.T) @ down.T


def route(h, w_router, b_router, top):
    """(chosen experts [T, top], their weights): softmax over the chosen logits only."""
    z = h @ w_router.T + b_router
    val, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(val, dim=-1)


def mixture(h, w, name, mlp):
    idx, wt = route(h, w[name + ".router"], w[name + ".router.b"], mlp["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for c in range(idx.shape[1]):
            e = f"{name}.e{int(idx[t, c])}"
            y[t] += wt[t, c] * expert(h[t], w[e + ".up"], w[e + ".down"])
    if mlp.get("shared") is not None:
        y = y + expert(h, w[name + ".shared.up"], w[name + ".shared.down"])
    return y


def forward(cfg, weights, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [T, vocab] (and the residual stream after every layer) of one whole sequence."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = w["embed"][torch.tensor(tokens)]
    kv, after = {}, []
    for i, lay in enumerate(cfg["layers"]):
        mx, n = lay["mixer"], f"l{i}.mix"
        if mx.get("kv_from") is None:
            kv[i] = keys_values(x, w, n, mx, eps, pos)
            k, v = kv[i]
        else:
            k, v = kv[mx["kv_from"]]
        a = window_attention(queries(x, w, n, mx, eps, pos), k, v, w[n + ".sink"], mx["scale"],
                             mx["mask"]["size"] if mx.get("mask") else None)
        y = a.reshape(len(tokens), -1) @ w[n + ".o"].T
        x = x + layer_norm(y, w[f"l{i}.norm1"], w[f"l{i}.norm1.b"], eps)
        if lay.get("mlp") is not None:
            y = mixture(x, w, f"l{i}.mlp", lay["mlp"])
            x = x + layer_norm(y, w[f"l{i}.norm2"], w[f"l{i}.norm2.b"], eps)
        after.append(x)
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
    return (logits, torch.stack(after)) if keep_layers else logits
