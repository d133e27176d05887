"""Small Nipulorn configurations and random weights for the tests, and helpers that run them through the engine.

The sizes differ from layer to layer and are picked so that nothing coincides by accident: widths, head, latent and value
sizes that are not multiples of 8, one tap and many taps, feed-forwards behind either mixer and behind none, one head and
more heads than one MMA tile has rows, latents larger than the width, rotations with and without scaling.  Queries are
large, so a softmax rests on few keys and a key that is wrongly seen or missed shows in the logits; decays reach from almost
none to almost everything within one token, so the recurrence remembers far tokens and forgets near ones.
"""
import json
import os

import torch


def _wkv(heads, dim, ff=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _latent(heads, dim, vdim, q_rank, kv_rank, rot_dim, scale, ff=None, base=10000.0, scaling=(4.0, 64, 16.0, 1.0)):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot_dim": rot_dim,
                      "scale": scale, "rot": rot},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _cfg(vocab, width, taps, layers, eps=1e-5, scale=3.0, logits=0.7):
    return {"architecture": "Nipulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"scale": scale}, "logit_scale": logits, "layers": layers}


# rank of the low-rank decay per wkv layer (a size that only the tensors give)
DECAY_RANKS = (6, 16, 1, 40)

CASES = {
    # both mixers, with and without feed-forwards
    "mixed": _cfg(151, 96, 4, [_wkv(3, 32, 72), _latent(5, 24, 40, 56, 48, 16, 0.21, 88), _wkv(2, 64), _latent(4, 16, 16, 32, 64, 8, 0.3)]),
    # nothing is a multiple of 8; an attention layer comes first
    "odd": _cfg(37, 50, 2, [_latent(3, 10, 14, 21, 18, 6, 0.35, 30, base=500.0, scaling=(2.0, 40, 8.0, 0.5)), _wkv(3, 20),
                            _wkv(1, 13, 45), _latent(7, 12, 9, 11, 20, 2, 0.3, scaling=None)], eps=3e-4, scale=1.0, logits=1.0),
    # big heads and latents, more heads than MMA rows, many taps
    "wide": _cfg(64, 136, 7, [_wkv(2, 128, 40), _latent(18, 40, 24, 72, 264, 40, 0.13), _latent(35, 16, 136, 200, 144, 24, 0.2, 24, base=1e6),
                              _latent(2, 72, 64, 24, 400, 64, 0.1)]),
    # one tap: no carried inputs; recurrences only
    "short": _cfg(96, 64, 1, [_wkv(4, 16, 32), _wkv(2, 40)]),
    # one tap and attention only: nothing is carried but the cache
    "plain": _cfg(40, 72, 1, [_latent(4, 24, 24, 24, 32, 8, 0.25, 48), _latent(2, 32, 48, 40, 96, 16, 0.2)]),
}


def make_weights(cfg, seed=0):
    """bf16 tensors under the design's names."""
    g = torch.Generator().manual_seed(seed)

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain / cols ** 0.5

    def vec(n, mean, dev):
        return mean + dev * torch.randn(n, generator=g)

    H = cfg["width"]
    w = {"embed": torch.randn(cfg["vocab"], H, generator=g) * 0.5, "final.norm": vec(H, 0.1, 0.2)}
    wkv = 0
    for i, lay in enumerate(cfg["layers"]):
        m, L, p = lay["mixer"], f"l{i}.", f"l{i}.mix."
        n, d = m["heads"], m["dim"]
        for k in ("1", "2") if lay["mlp"] is not None else ("1",):
            w[L + "norm" + k], w[L + "norm" + k + "b"] = vec(H, 0.1, 0.2), vec(H, -0.2, 0.2)
            w[L + "canon" + k] = 0.35 * torch.randn(H, cfg["canon"]["taps"], generator=g)
        if lay["type"] == "wkv":
            rank, wkv = DECAY_RANKS[wkv % len(DECAY_RANKS)], wkv + 1
            for c in "rkvgw":
                w[p + "mu." + c] = torch.rand(H, generator=g) * 1.4 - 0.2
            for c in "rkvg":
                w[p + c] = mat(n * d, H)
            w[p + "w1"], w[p + "w2"] = mat(rank, H, 2.0), mat(n * d, rank)
            w[p + "w0"] = torch.rand(n * d, generator=g) * 7.0 - 5.5
            w[p + "u"], w[p + "norm"], w[p + "o"] = torch.randn(n, d, generator=g), vec(n * d, 1.0, 0.3), mat(H, n * d)
        else:
            R = m["kv_rank"]
            w[p + "dq"], w[p + "dkv"] = mat(m["q_rank"], H), mat(R + m["rot_dim"], H)
            w[p + "dq.norm"], w[p + "dkv.norm"] = vec(m["q_rank"], 1.3, 0.3), vec(R, 1.1, 0.3)
            w[p + "uq"] = mat(n * (d + m["rot_dim"]), m["q_rank"], 2.0)
            w[p + "uk"], w[p + "uv"] = mat(n * d, R), mat(n * m["vdim"], R)
            w[p + "sink"], w[p + "o"] = vec(n, 1.0, 1.0), mat(H, n * m["vdim"])
        if lay["mlp"] is not None:
            ff = lay["mlp"]["ff"]
            w[L + "mlp.up"], w[L + "mlp.down"], w[L + "mlp.act"] = mat(ff, H, 1.5), mat(H, ff), \
                torch.tensor([-1.5, 1.5]) + 0.5 * torch.randn(2, generator=g)
    return {k: t.to(torch.bfloat16) for k, t in w.items()}


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

    cls = ALL_MODELS["nipulorn"]
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


def score_batch(engine, seqs, sizes, live_max=3):
    """Logits of several sequences fed in portions of their own sizes, ``live_max`` at a time; finished ones make room."""
    cuts = {k: portions(len(t), sizes[k]) for k, t in seqs.items()}
    queue, live, got = list(seqs), [], {k: [] for k in seqs}
    while queue or live:
        while queue and len(live) < live_max:
            live.append(queue.pop(0))
        step = [(k, cuts[k].pop(0)) for k in live]
        done = [k for k, (_, b) in step if b == len(seqs[k])]
        out = engine.score_step([(k, seqs[k][a:b], range(b - a)) for k, (a, b) in step], done).double().cpu()
        for k, (a, b) in step:
            got[k].append(out[:b - a])
            out = out[b - a:]
        live = [k for k in live if k not in done]
    return {k: torch.cat(v) for k, v in got.items()}


BATCH = {0: 61, 1: 7, 2: 33, 3: 1, 4: 48, 5: 16, 6: 2}
BATCH_SIZES = {0: [5, 1, 2], 1: [1], 2: [17, 1], 3: [1], 4: [2, 31], 5: [16], 6: [2]}


def row_error(got, want):
    """Root mean square difference per row (mean taken off), relative to the spread of the expected logits."""
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return (d ** 2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
