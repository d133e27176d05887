"""Small Gekapel configurations and random weights for the tests, and helpers that run them through the engine.

The sizes differ from layer to layer and are picked so that nothing coincides by accident: value sizes other than the key
size, one or many query heads per key/value head, windows that are not page multiples, widths and head sizes that are
not multiples of 8, an odd vocabulary, layers without a feed-forward, without a shared expert, with every expert chosen.
Query norms are large, so a softmax rests on few keys and a key that is wrongly seen or missed shows in the logits.
"""
import json
import os

import torch


def _rot(dims, base=10000.0, factor=4.0, low=1.0, high=4.0, original=96):
    return {"base": base, "dims": dims, "scaling": {"factor": factor, "low": low, "high": high, "original": original}}


def _attn(heads, kv, dim, vdim, window, dims, scale, kv_from=None, **rot):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": _rot(dims, **rot),
         "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def _moe(experts, top, ff, shared):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    m["shared"] = None if shared is None else {"ff": shared}
    return m


def _cfg(vocab, width, layers, eps=1e-5):
    return {"architecture": "Gekapel", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{"type": "attention", "mixer": a, "mlp": m} for a, m in layers]}


CASES = {
    # shared keys across layers with windows of their own, a layer without feed-forward
    "mixed": _cfg(151, 96, [
        (_attn(6, 2, 32, 48, 13, 8, 0.31), _moe(5, 2, 40, 24)),
        (_attn(4, 4, 16, 16, 33, 16, 0.2, base=500.0), None),
        (_attn(3, 1, 48, 24, 17, 12, 0.17, factor=2.0, original=40), _moe(9, 3, 16, None)),
        (_attn(6, 2, 32, 48, 29, 8, 0.27, kv_from=0), _moe(4, 1, 24, 56)),
        (_attn(6, 2, 32, 48, 7, 8, 0.35, kv_from=0), _moe(3, 2, 8, 8)),
    ]),
    # nothing is a multiple of 8; every expert is chosen; a window of one token
    "odd": _cfg(37, 50, [
        (_attn(5, 5, 20, 12, 21, 6, 0.3, base=100.0, factor=8.0, low=0.5, high=2.0, original=64), _moe(7, 7, 18, 10)),
        (_attn(4, 2, 10, 30, 1, 10, 0.4), _moe(2, 1, 5, 3)),
        (_attn(5, 5, 20, 12, 40, 6, 0.2, kv_from=0, base=100.0, factor=8.0, low=0.5, high=2.0, original=64), _moe(6, 4, 13, None)),
    ], eps=3e-4),
    # big heads, more query heads per key/value head than one MMA tile has rows, a window beyond the sequences
    "wide": _cfg(64, 136, [
        (_attn(18, 1, 72, 136, 50, 72, 0.11), _moe(12, 3, 72, 64)),
        (_attn(2, 1, 192, 256, 19, 32, 0.07), _moe(3, 1, 200, 40)),
        (_attn(8, 2, 256, 64, 100000, 64, 0.06, base=1e6), _moe(4, 2, 32, 16)),
    ]),
}


def make_weights(cfg, seed=0):
    """bf16 tensors under the design's names."""
    g = torch.Generator().manual_seed(seed)

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain / cols ** 0.5

    def vec(n, mean, dev):
        return mean + dev * torch.randn(n, generator=g)

    H = cfg["width"]
    w = {"embed": torch.randn(cfg["vocab"], H, generator=g), "head": mat(cfg["vocab"], H, 1.0),
         "final.norm": vec(H, 1.0, 0.2), "final.norm.b": vec(H, 0.0, 0.2)}
    for i, lay in enumerate(cfg["layers"]):
        m, p = lay["mixer"], f"l{i}.mix."
        for n in ("norm1", "norm2") if lay["mlp"] is not None else ("norm1",):
            w[f"l{i}.{n}"], w[f"l{i}.{n}.b"] = vec(H, 0.8, 0.2), vec(H, 0.0, 0.2)
        w[p + "q"], w[p + "o"] = mat(m["heads"] * m["dim"], H), mat(H, m["heads"] * m["vdim"])
        w[p + "q.norm"] = vec(m["dim"], 1.5, 0.3)
        w[p + "sink"] = vec(m["heads"], 1.0, 1.0)
        if m.get("kv_from") is None:
            w[p + "k"], w[p + "v"] = mat(m["kv_heads"] * m["dim"], H), mat(m["kv_heads"] * m["vdim"], H)
            w[p + "k.norm"] = vec(m["dim"], 1.2, 0.3)
        if lay["mlp"] is None:
            continue
        mlp, p = lay["mlp"], f"l{i}.mlp."
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        w[p + "router"], w[p + "router.b"] = mat(E, H, 1.5), vec(E, 0.0, 1.0)
        for e in range(E):
            w[f"{p}e{e}.up"], w[f"{p}e{e}.down"] = mat(ff, H), mat(H, ff)
        if mlp["shared"] is not None:
            w[p + "shared.up"], w[p + "shared.down"] = mat(mlp["shared"]["ff"], H), mat(H, mlp["shared"]["ff"])
    return {n: t.to(torch.bfloat16) for n, t in w.items()}


def write_model(path, cfg, weights):
    """A model directory as a user has it."""
    from unillm_b200.weights.loaders import write_safetensors

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), weights)
    return str(path)


def load_model(cfg, weights):
    from unillm_b200.models import ALL_MODELS
    from unillm_b200.model_core import ModelWeights

    cls = ALL_MODELS["gekapel"]
    return cls.from_weights(cls.config_class.from_hf_config(cfg), ModelWeights(dict(weights)))


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def portions(n, sizes):
    """Cuts [0, n) into portions whose sizes cycle through ``sizes``."""
    out, at, k = [], 0, 0
    while at < n:
        s = min(sizes[k % len(sizes)], n - at)
        out.append((at, at + s))
        at, k = at + s, k + 1
    return out


def score(engine, toks, cuts, key="a"):
    """All logits of one sequence, fed in the given portions."""
    out = []
    for a, b in cuts:
        last = b == len(toks)
        out.append(engine.score_step([(key, toks[a:b], list(range(b - a)))], [key] if last else []).float().cpu())
    return torch.cat(out).double()


def row_error(got, want):
    """Root mean square difference per row (mean taken off), relative to the spread of the expected logits."""
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return (d ** 2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
