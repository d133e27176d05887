"""Small Tasadra configurations and random weights for the tests, and helpers that run them through the engine.

The sizes differ from layer to layer and are picked so that nothing coincides by accident: widths, head and value sizes that
are not multiples of 8, rotations of part of a head, chunks of one token, chunks that end inside pages and chunks that no
sequence fills, convolutions of one tap and of many, decay and gate ranks of their own, mixers with and without a
feed-forward, layers that share another layer's keys under a chunk of their own.  Queries are large, so a softmax rests on few
keys and a key that is wrongly seen or missed shows in the logits; decays reach from almost none to almost everything within
one token, channel by channel; the two maps of a differential attention weigh about the same.
"""
import functools

import torch

import tasadra_plain as P
from nipulorn_cases import BATCH, BATCH_SIZES, portions, row_error, score, score_batch, tokens, write_model  # noqa: F401


def _attn(heads, kv, dim, vdim, dims, scale, base=10000.0, yarn=None, cap=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if yarn is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if cap is not None:
        m["softcap"] = cap
    return "attention", m


def _delta(heads, kv, dim, vdim, conv):
    return "channel_delta", {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def _diff(heads, kv, dim, vdim, chunk, scale, diff, src=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if chunk:
        m["mask"] = {"size": chunk}
    if src is not None:
        m["kv_from"] = src
    return "attention_2", m


def _layer(mixer, ff):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _cfg(vocab, width, layers, mult, eps=1e-5):
    return {"architecture": "Tasadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


CASES = {
    # every kind of layer, sharing across a layer of another kind
    "mixed": _cfg(151, 96, [_layer(_diff(4, 2, 16, 40, 13, 0.3, 0.35), 72),
                            _layer(_attn(6, 3, 24, 32, 16, 0.25, yarn=(12.0, 40, 4.0, 0.5), cap=9.0), 56),
                            _layer(_delta(4, 2, 32, 24, 4), None),
                            _layer(_diff(4, 2, 16, 40, 24, 0.25, 0.6, src=0), 40),
                            _layer(_attn(4, 1, 16, 16, 16, 0.3, base=500.0), None)], 0.7),
    # nothing is a multiple of 8; chunks of one token and of any length; no convolution history; sharing twice
    "odd": _cfg(37, 50, [_layer(_delta(3, 3, 13, 21, 1), 30), _layer(_attn(3, 1, 10, 14, 6, 0.4, base=700.0, yarn=(2.5, 16, 2.0, 1.0), cap=6.0), 18),
                         _layer(_diff(3, 1, 5, 9, 0, 0.5, 0.2), None), _layer(_diff(3, 1, 5, 9, 1, 0.4, 0.8, src=2), 22),
                         _layer(_diff(3, 1, 5, 9, 7, 0.6, 0.5, src=2), 26)], 1.3, eps=3e-4),
    # big heads, more query heads than one MMA tile has rows, many taps, states too large for a thread's registers
    "wide": _cfg(64, 136, [_layer(_attn(18, 1, 72, 136, 72, 0.15, base=1e6, yarn=(8.0, 2048, 32.0, 1.0), cap=30.0), 104),
                           _layer(_delta(2, 1, 136, 200, 7), 40), _layer(_diff(10, 1, 72, 128, 33, 0.12, 0.45), None),
                           _layer(_delta(6, 2, 64, 128, 5), 48), _layer(_diff(2, 2, 128, 64, 64, 0.1, 0.1), 24)], 0.4),
    # sizes that the tensor-core prompt kernel takes
    "even": _cfg(80, 64, [_layer(_attn(4, 2, 128, 128, 96, 0.1, base=3000.0, cap=7.0), 64), _layer(_diff(4, 1, 64, 128, 24, 0.15, 0.3), 32),
                          _layer(_diff(4, 1, 64, 128, 40, 0.15, 0.55, src=1), None), _layer(_attn(2, 2, 128, 128, 128, 0.09), 16)], 0.9),
}
RANKS = (6, 24, 16, 9)                            # of decays and gates, in turn


def make_weights(cfg, seed=0):
    """bf16 tensors under the design's names."""
    g = torch.Generator().manual_seed(seed)

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain / cols ** 0.5

    def vec(n, mean, dev):
        return mean + dev * torch.randn(n, generator=g)

    def norm(name):
        w[name], w[name + ".b"], w[name + ".alpha"] = vec(H, 1.2, 0.3), vec(H, 0.0, 0.2), 0.4 + 0.5 * torch.rand((), generator=g)

    H, used = cfg["width"], 0
    w = {"embed": torch.randn(cfg["vocab"], H, generator=g), "head": mat(cfg["vocab"], H)}
    norm("final.norm")
    for i, lay in enumerate(cfg["layers"]):
        L, p, m, mlp = f"l{i}.", f"l{i}.mix.", lay["mixer"], lay["mlp"]
        n, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        norm(L + "norm1")
        w[L + "shift"] = torch.rand(H, generator=g) * 1.2 - 0.1
        w[L + "dwa"] = torch.cat([0.4 * torch.randn(i + 1, generator=g), vec(1, 1.0, 0.2)])
        if lay["type"] == "attention":
            w[p + "q"], w[p + "k"], w[p + "v"] = mat(n * d, H, 1.6), mat(G * d, H, 1.6), mat(G * e, H)
            w[p + "q.norm"], w[p + "k.norm"], w[p + "g"] = vec(d, 1.6, 0.4), vec(d, 1.4, 0.4), mat(n, H, 2.0)
        elif lay["type"] == "attention_2":
            w[p + "q"], w[p + "g"] = mat(n * 2 * d, H, 2.5), mat(n * e, H, 2.0)
            if m.get("kv_from") is None:
                w[p + "k"], w[p + "v"] = mat(G * 2 * d, H, 2.0), mat(G * e, H)
            for c in ("lq1", "lk1", "lq2", "lk2"):
                w[p + c] = vec(d, 0.0, 0.7 / d ** 0.5)
        else:
            for c, rows in (("q", G * d), ("k", G * d), ("v", n * e)):
                w[p + c], w[p + c + ".conv"] = mat(rows, H, 1.5), 0.6 * torch.randn(rows, m["conv"], generator=g)
            ra, rg = RANKS[used % 4], RANKS[(used + 1) % 4]
            used += 1
            w[p + "b"], w[p + "a1"], w[p + "a2"] = mat(n, H, 2.0), mat(ra, H, 1.5), mat(n * d, ra, 1.5)
            w[p + "g1"], w[p + "g2"] = mat(rg, H, 1.5), mat(n * e, rg, 1.5)
            w[p + "A_log"], w[p + "dt_bias"] = torch.rand(n, generator=g) * 3 - 2, torch.rand(n * d, generator=g) * 5 - 5
            w[p + "norm"] = vec(e, 1.1, 0.3)
        w[p + "o"] = mat(H, n * e)
        if mlp is not None:
            norm(L + "norm2")
            w[L + "mlp.up"], w[L + "mlp.up.b"] = mat(mlp["ff"], H, 1.2), vec(mlp["ff"], 0.1, 0.3)
            w[L + "mlp.down"], w[L + "mlp.down.b"] = mat(H, mlp["ff"]), vec(H, 0.0, 0.3)
    return {k: t.to(torch.bfloat16) for k, t in w.items()}


def load_model(cfg, weights):
    from unillm_b200.models import ALL_MODELS
    from unillm_b200.model_core import ModelWeights

    cls = ALL_MODELS["tasadra"]
    return cls.from_weights(cls.config_class.from_hf_config(cfg), ModelWeights(dict(weights)))


PROMPTS = [(n, 30 + n) for n in (19, 3, 34, 1, 50)]


@functools.lru_cache(maxsize=None)
def expected_generation(name, count=6):
    """Greedy continuations of the case's prompts by the plain statement (the last prompt is the front of the one before)."""
    cfg = CASES[name]
    w = make_weights(cfg)
    prompts = [tokens(cfg, n, seed) for n, seed in PROMPTS]
    prompts.append(prompts[4][:40])
    return prompts, [greedy(cfg, w, p, count) for p in prompts]


def greedy(cfg, w, prompt, n):
    out = []
    for _ in range(n):
        out.append(int(P.forward(cfg, w, prompt + out)[-1].argmax()))
    return out
