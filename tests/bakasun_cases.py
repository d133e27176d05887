"""Small Bakasun configurations and random weights for the tests, and helpers that run them through the engine.

The sizes differ from layer to layer and are picked so that nothing coincides by accident: widths, head and value sizes that
are not multiples of 8, rotations of any even size, windows of one token and windows that no sequence fills, convolutions of
one tap and of many, one expert group and several, mixers with and without a feed-forward.  Queries are large, so a softmax
rests on few keys and a key that is wrongly seen or missed shows in the logits; decays reach from almost none to almost
everything within one token; corrections are as large as the differences between the experts' scores.
"""
import functools

import torch

import bakasun_plain as P
from nipulorn_cases import BATCH, BATCH_SIZES, portions, row_error, score, score_batch, tokens, write_model  # noqa: F401


def _attn(heads, kv, dim, vdim, window, dims, scale, base=10000.0, factor=None, cap=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if window:
        m["mask"] = {"size": window}
    if factor is not None:
        m["rot"]["scaling"] = {"factor": factor}
    if cap is not None:
        m["softcap"] = cap
    return m


def _delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared, groups=(1, 1)):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]}},
            "expert": {"ff": ff}, "shared": {"ff": shared}}


def _single(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def _pair(left, right, scales, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def _cfg(vocab, width, layers, eps=1e-5):
    return {"architecture": "Bakasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CASES = {
    # every kind of layer
    "mixed": _cfg(151, 96, [_single(_attn(4, 2, 24, 40, 20, 16, 0.2), _dense(72)),
                            _pair(_attn(6, 3, 16, 24, 33, 8, 0.3, factor=3.0, cap=9.0), _delta(4, 2, 32, 24, 4), (0.7, 1.2), _moe(12, 3, 40, 56, (4, 2))),
                            _pair(_attn(2, 1, 32, 16, 9, 32, 0.15, base=500.0, factor=1.5, cap=15.0), _delta(3, 1, 16, 40, 3), (1.1, 0.6), None),
                            _single(_attn(5, 5, 16, 16, 17, 12, 0.25), _moe(9, 4, 24, 32, (3, 2)))]),
    # nothing is a multiple of 8; two mixers come first; a window of one token; no convolution history
    "odd": _cfg(37, 50, [_pair(_attn(3, 1, 10, 14, 7, 6, 0.35, factor=2.5, cap=6.0), _delta(3, 3, 13, 21, 1), (0.4, 0.4), _dense(30)),
                         _single(_attn(3, 3, 20, 9, 1, 10, 0.3), _moe(5, 1, 18, 11)),
                         _pair(_attn(2, 2, 12, 12, 0, 2, 0.3, cap=4.0), _delta(2, 1, 6, 6, 2), (1.0, 1.0), _moe(6, 5, 10, 22, (2, 2)))], eps=3e-4),
    # big heads, more heads than one MMA tile has rows, many taps, many experts, states too large for a thread's registers
    "wide": _cfg(64, 136, [_single(_attn(18, 1, 72, 136, 70, 72, 0.12, base=1e6), _moe(40, 6, 16, 24, (8, 3))),
                           _pair(_attn(4, 1, 128, 64, 50, 40, 0.1, factor=8.0, cap=30.0), _delta(2, 1, 136, 200, 7), (0.9, 0.5), _dense(104)),
                           _pair(_attn(2, 2, 40, 72, 64, 40, 0.2, factor=1.0, cap=50.0), _delta(6, 2, 64, 128, 5), (0.3, 0.8), None)]),
    # attention only: nothing is carried but the cache
    "plain": _cfg(40, 72, [_single(_attn(4, 1, 24, 24, 25, 24, 0.25), _dense(48)), _single(_attn(2, 2, 32, 48, 0, 20, 0.2), None)]),
}


def make_weights(cfg, seed=0):
    """bf16 tensors under the design's names."""
    g = torch.Generator().manual_seed(seed)

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain / cols ** 0.5

    def vec(n, mean, dev):
        return mean + dev * torch.randn(n, generator=g)

    def attention(p, m, bias):
        n, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
        w[p + "q"], w[p + "k"], w[p + "v"] = mat(n, H, 1.6), mat(k, H, 1.6), mat(m["kv_heads"] * m["vdim"], H)
        if bias:
            w[p + "q.b"], w[p + "k.b"], w[p + "v.b"] = vec(n, 0.3, 0.5), vec(k, -0.2, 0.5), vec(m["kv_heads"] * m["vdim"], 0.0, 0.5)
        else:
            w[p + "q.norm"], w[p + "k.norm"] = vec(n, 1.6, 0.4), vec(k, 1.4, 0.4)
        w[p + "o"] = mat(H, m["heads"] * m["vdim"])

    def delta(p, m):
        n, d = m["heads"], m["kv_heads"] * m["dim"]
        for c, rows in (("q", d), ("k", d), ("v", n * m["vdim"])):
            w[p + c], w[p + c + ".conv"] = mat(rows, H, 1.5), 0.6 * torch.randn(rows, m["conv"], generator=g)
        w[p + "b"], w[p + "a"], w[p + "g"] = mat(n, H, 2.0), mat(n, H, 2.0), mat(n * m["vdim"], H)
        w[p + "A_log"], w[p + "dt_bias"] = torch.rand(n, generator=g) * 3 - 2, torch.rand(n, generator=g) * 5 - 5
        w[p + "norm"], w[p + "o"] = vec(m["vdim"], 1.1, 0.3), mat(H, n * m["vdim"])

    def gated(p, ff):
        w[p + "gate"], w[p + "up"], w[p + "down"] = mat(ff, H, 1.3), mat(ff, H, 1.3), mat(H, ff)

    H = cfg["width"]
    w = {"embed": torch.randn(cfg["vocab"], H, generator=g), "final.norm": vec(H, 0.1, 0.2), "head": mat(cfg["vocab"], H)}
    for i, lay in enumerate(cfg["layers"]):
        L, mlp = f"l{i}.", lay["mlp"]
        for k in ("1", "2") if mlp is not None else ("1",):
            w[L + "norm" + k], w[L + "norm" + k + "b"] = vec(H, 0.1, 0.2), vec(H, -0.1, 0.2)
        if lay["type"] == "attention":
            attention(L + "mix.", lay["mixer"], False)
        else:
            attention(L + "mix.left.", lay["mixer"]["left"], True)
            delta(L + "mix.right.", lay["mixer"]["right"])
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            gated(L + "mlp.", mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        for e in range(E):
            gated(f"{L}mlp.e{e}.", mlp["expert"]["ff"])
        w[L + "mlp.router"], w[L + "mlp.correction"] = mat(E, H, 1.5), vec(E, -0.05, 1.5 / E)
        gated(L + "mlp.shared.", mlp["shared"]["ff"])
        w[L + "mlp.shared.sg"] = mat(1, H, 2.0)
    return {k: t.to(torch.bfloat16) for k, t in w.items()}


def load_model(cfg, weights):
    from unillm_b200.models import ALL_MODELS
    from unillm_b200.model_core import ModelWeights

    cls = ALL_MODELS["bakasun"]
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
