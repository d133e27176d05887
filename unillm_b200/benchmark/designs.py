"""Prefill and decode throughput of one design beside the closest existing family at equal size, and the same
comparison kernel by kernel (``python bench.py --design gekapel|nipulorn|bakasun|tasadra [--design-kernels]``).

Both models are random-weight stacks of a few layers with a real model's layer sizes, run by the same
``GpuModelRunner`` steps that serve requests: a prefill step is one batch of whole prompts, a decode step one token of
every sequence at a given context through the captured CUDA graph.  Device time of a step is the CUDA-event interval
around its launch (metadata upload, kernels, read-back of the samples); the layers' weights are larger than L2.

The kernel table replays every call of one step alone (CUDA graph, L2 flushed between calls, ``microbench.time_ms``) and
sets its time against the roofline of the call: the larger of its bytes over the copy bandwidth and its multiply-adds
over the bf16 matrix throughput (MEASURED_PEAKS.json).

The closest family to Gekapel is DeepSeek-MoE (routed experts plus always-on ones), here with Mistral's sliding window.
Its experts have a gate, so at equal size they are two thirds as wide.

Nipulorn's parts have two nearest relatives.  Whole steps are set beside Llama, the dense full-attention decoder of the same
runner, with its feed-forward as wide as makes the parameters equal; the recurrence is set beside RWKV-6's kernel (a model
of the whole-model path) at the same heads, tokens and state.  Arithmetic that is fp32 by design counts against the FMA
rate of the device instead of the matrix rate.

Bakasun's steps are set beside DeepSeek-MoE with Mistral's sliding window (the same gated experts and always-on expert, windowed
attention in every layer), its experts as wide as makes the parameters equal; its gated delta rule is set beside Nipulorn's
recurrence at the same heads, tokens and state.

Tasadra's steps are set beside Llama with its feed-forward as wide as makes the parameters equal, its delta rule with decays per
channel beside Bakasun's with decays per head at the same heads, tokens and state.
"""
from __future__ import annotations

import contextlib
import statistics
from typing import Dict, List, Optional

import torch

from ..engine.runner import GpuModelRunner, RunnerWeights, StepBatch
from ..models import configs as C
from ..models.families import BakasunModel, GekapelModel, NipulornModel, TasadraModel
from ..models.spec import DecoderSpec, MoESpec
from ..ops import cuda_ops as K
from .microbench import _peaks, time_ms

# per size: width, heads, kv heads, head dim, window, experts, top, expert width, shared width, vocabulary, layers
SIZES = {
    "1k": dict(width=1024, heads=16, kv=4, dim=64, window=256, experts=64, top=8, ff=384, shared=768, vocab=32000, layers=4),
    "2k": dict(width=2048, heads=16, kv=4, dim=128, window=512, experts=32, top=4, ff=1536, shared=3072, vocab=32000, layers=4),
    "4k": dict(width=4096, heads=32, kv=8, dim=128, window=1024, experts=16, top=2, ff=6144, shared=6144, vocab=32000, layers=4),
}
PREFILL = [(4, 2048), (1, 512)]            # (prompts, tokens each)
DECODE = [(1, 2048), (32, 2048), (256, 2048)]   # (sequences, context)


def gekapel_spec(z: dict) -> DecoderSpec:
    layers = []
    for i in range(z["layers"]):
        mx = {"heads": z["heads"], "kv_heads": z["kv"], "dim": z["dim"], "vdim": z["dim"], "mask": {"size": z["window"]},
              "rot": {"base": 10000.0, "dims": z["dim"] // 2,
                      "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 4096}}, "scale": z["dim"] ** -0.5}
        if i >= z["layers"] // 2:                       # the upper half reads the keys of the last layer that has some
            mx["kv_from"] = z["layers"] // 2 - 1
        layers.append({"type": "attention", "mixer": mx,
                       "mlp": {"kind": "moe", "router": {"experts": z["experts"], "top": z["top"]}, "expert": {"ff": z["ff"]},
                               "shared": {"ff": z["shared"]}}})
    return GekapelModel.spec_from_config(C.GekapelConfig(vocab_size=z["vocab"], hidden_size=z["width"],
                                                         num_hidden_layers=z["layers"], layers=layers))


def closest_spec(z: dict) -> DecoderSpec:
    ff = z["ff"] * 2 // 3
    return DecoderSpec(vocab_size=z["vocab"], hidden_size=z["width"], num_layers=z["layers"], num_heads=z["heads"],
                       num_kv_heads=z["kv"], head_dim=z["dim"], intermediate_size=ff, max_position_embeddings=8192,
                       window=z["window"],
                       moe=MoESpec(num_experts=z["experts"], top_k=z["top"], intermediate_size=ff, num_shared_experts=1,
                                   shared_intermediate_size=z["shared"] * 2 // 3))


# width, wkv heads and size, latent attention (heads, dim, vdim, q rank, kv rank, rotated), feed-forward, vocabulary, layers
# (three wkv layers, then one of latent attention with a feed-forward)
NIPULORN_SIZES = {
    "1k": dict(width=1024, wkv=16, wdim=64, heads=16, dim=64, vdim=64, q_rank=384, kv_rank=256, rot=32, ff=4096, vocab=32000, layers=4),
    "2k": dict(width=2048, wkv=32, wdim=64, heads=16, dim=128, vdim=128, q_rank=768, kv_rank=512, rot=64, ff=8192, vocab=32000, layers=4),
    "4k": dict(width=4096, wkv=64, wdim=64, heads=32, dim=128, vdim=128, q_rank=1536, kv_rank=512, rot=64, ff=16384, vocab=32000, layers=4),
}


def nipulorn_spec(z: dict) -> DecoderSpec:
    layers = []
    for i in range(z["layers"]):
        if i % 4 != 3:
            layers.append({"type": "wkv", "mixer": {"heads": z["wkv"], "dim": z["wdim"]}, "mlp": None})
            continue
        layers.append({"type": "latent_attention", "mlp": {"kind": "dense", "ff": z["ff"]},
                       "mixer": {"heads": z["heads"], "dim": z["dim"], "vdim": z["vdim"], "q_rank": z["q_rank"], "kv_rank": z["kv_rank"],
                                 "rot_dim": z["rot"], "scale": (z["dim"] + z["rot"]) ** -0.5,
                                 "rot": {"base": 10000.0, "dims": z["rot"],
                                         "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}})
    return NipulornModel.spec_from_config(C.NipulornConfig(vocab_size=z["vocab"], hidden_size=z["width"], num_hidden_layers=z["layers"],
                                                           canon_taps=4, logit_scale=0.5, embedding_scale=z["width"] ** 0.5, layers=layers))


def llama_spec(z: dict) -> DecoderSpec:
    """As many parameters in the layers, in a dense decoder with the same attention heads over full-size keys."""
    H, d, n = z["width"], z["dim"], z["layers"]
    hq, hkv = H // d, max(1, H // d // 4)
    wkv = 5 * H * z["wkv"] * z["wdim"] + 64 * (H + z["wkv"] * z["wdim"])
    lat = H * (z["q_rank"] + z["kv_rank"] + z["rot"]) + z["q_rank"] * z["heads"] * (d + z["rot"]) + \
        z["kv_rank"] * z["heads"] * (d + z["vdim"]) + H * z["heads"] * z["vdim"] + 2 * H * z["ff"]
    total = n // 4 * (3 * wkv + lat)
    attn = H * d * (hq + 2 * hkv) + H * hq * d
    ff = (total - n * attn) // (n * 3 * H) // 128 * 128
    return DecoderSpec(vocab_size=z["vocab"], hidden_size=H, num_layers=n, num_heads=hq, num_kv_heads=hkv, head_dim=d,
                       intermediate_size=ff, max_position_embeddings=8192, tie_embeddings=True)


# width, attention (heads, kv heads, size of a head, window), delta rule (heads, query / key heads, size), experts, expert width,
# shared width, vocabulary, layers (attention, two with both mixers, attention; a mixture of experts in each)
BAKASUN_SIZES = {
    "1k": dict(width=1024, heads=16, kv=4, dim=64, window=256, dh=16, dg=8, dd=64, experts=64, top=8, ff=256, shared=512, vocab=32000, layers=4),
    "2k": dict(width=2048, heads=16, kv=4, dim=128, window=512, dh=16, dg=8, dd=128, experts=32, top=4, ff=1024, shared=2048, vocab=32000, layers=4),
    "4k": dict(width=4096, heads=32, kv=8, dim=128, window=1024, dh=32, dg=16, dd=128, experts=16, top=2, ff=4096, shared=4096, vocab=32000, layers=4),
}


def bakasun_spec(z: dict) -> DecoderSpec:
    attn = {"heads": z["heads"], "kv_heads": z["kv"], "dim": z["dim"], "vdim": z["dim"], "mask": {"size": z["window"]},
            "rot": {"base": 10000.0, "dims": z["dim"]}, "scale": z["dim"] ** -0.5}
    left = dict(attn, softcap=30.0, rot={"base": 10000.0, "dims": z["dim"] // 2, "scaling": {"factor": 4.0}})
    right = {"heads": z["dh"], "kv_heads": z["dg"], "dim": z["dd"], "vdim": z["dd"], "conv": 4}
    mlp = {"kind": "moe", "router": {"experts": z["experts"], "top": z["top"], "groups": {"count": 4, "keep": 2}},
           "expert": {"ff": z["ff"]}, "shared": {"ff": z["shared"]}}
    both = {"left": left, "right": right, "left_scale": 0.7, "right_scale": 0.8}
    layers = [{"type": "parallel", "mixer": both, "mlp": mlp} if i % 4 in (1, 2) else {"type": "attention", "mixer": attn, "mlp": mlp}
              for i in range(z["layers"])]
    return BakasunModel.spec_from_config(C.BakasunConfig(vocab_size=z["vocab"], hidden_size=z["width"], num_hidden_layers=z["layers"],
                                                         layers=layers))


def windowed_moe_spec(z: dict) -> DecoderSpec:
    """As many parameters in the layers, in layers of windowed attention and a mixture of experts."""
    H, n = z["width"], z["layers"]
    delta = n // 2 * H * z["dd"] * (2 * z["dg"] + 3 * z["dh"])
    ff = z["ff"] + delta // (n * 3 * H * (z["experts"] + z["shared"] // z["ff"])) // 8 * 8
    return DecoderSpec(vocab_size=z["vocab"], hidden_size=H, num_layers=n, num_heads=z["heads"], num_kv_heads=z["kv"], head_dim=z["dim"],
                       intermediate_size=ff, max_position_embeddings=8192, window=z["window"],
                       moe=MoESpec(num_experts=z["experts"], top_k=z["top"], intermediate_size=ff, num_shared_experts=z["shared"] // z["ff"]))


# width, attention (heads, kv heads, size of a head), delta rule (heads, size), differential attention (heads, kv heads, size of a
# map's head; values are twice that), chunk, feed-forward, vocabulary, layers (attention, delta rule, differential, differential on
# the third layer's keys, and again)
TASADRA_SIZES = {
    "1k": dict(width=1024, heads=16, kv=4, dim=64, dh=16, dd=64, xh=8, xkv=2, xdim=64, chunk=1024, ff=4096, vocab=32000, layers=4),
    "2k": dict(width=2048, heads=16, kv=4, dim=128, dh=16, dd=128, xh=16, xkv=4, xdim=64, chunk=1024, ff=8192, vocab=32000, layers=4),
    "4k": dict(width=4096, heads=32, kv=8, dim=128, dh=32, dd=128, xh=32, xkv=8, xdim=64, chunk=1024, ff=16384, vocab=32000, layers=4),
}


def tasadra_spec(z: dict) -> DecoderSpec:
    layers = []
    for i in range(z["layers"]):
        if i % 4 == 0:
            kind = "attention"
            mx = {"heads": z["heads"], "kv_heads": z["kv"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5, "softcap": 50.0,
                  "rot": {"base": 10000.0, "dims": z["dim"], "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
        elif i % 4 == 1:
            kind, mx = "channel_delta", {"heads": z["dh"], "kv_heads": z["dh"], "dim": z["dd"], "vdim": z["dd"], "conv": 4}
        else:
            kind = "attention_2"
            mx = {"heads": z["xh"], "kv_heads": z["xkv"], "dim": z["xdim"], "vdim": 2 * z["xdim"], "scale": z["xdim"] ** -0.5, "diff": 0.5,
                  "mask": {"size": z["chunk"]}}
            if i % 4 == 3:
                mx["kv_from"] = i - 1
        layers.append({"type": kind, "mixer": mx, "mlp": {"kind": "dense", "ff": z["ff"]}})
    return TasadraModel.spec_from_config(C.TasadraConfig(vocab_size=z["vocab"], hidden_size=z["width"], num_hidden_layers=z["layers"],
                                                         residual_mult=0.5, layers=layers))


def plain_llama_spec(z: dict) -> DecoderSpec:
    """As many parameters in the layers, in a dense decoder with the attention heads of the first layer in every layer."""
    H, d, n, xv = z["width"], z["dim"], z["layers"], 2 * z["xdim"]
    attn = H * d * (2 * z["heads"] + 2 * z["kv"])
    delta = H * z["dd"] * 4 * z["dh"] + 2 * 64 * (H + z["dh"] * z["dd"])
    own = H * (3 * z["xh"] + 2 * z["xkv"]) * xv
    total = n // 4 * (attn + delta + 2 * own - H * 2 * z["xkv"] * xv) + n * 2 * H * z["ff"]
    ff = (total - n * attn) // (n * 3 * H) // 128 * 128
    return DecoderSpec(vocab_size=z["vocab"], hidden_size=H, num_layers=n, num_heads=z["heads"], num_kv_heads=z["kv"], head_dim=d,
                       intermediate_size=ff, max_position_embeddings=8192)


DESIGNS = {"gekapel": (SIZES, {"gekapel": gekapel_spec, "deepseek_moe + window": closest_spec}),
           "nipulorn": (NIPULORN_SIZES, {"nipulorn": nipulorn_spec, "llama": llama_spec}),
           "bakasun": (BAKASUN_SIZES, {"bakasun": bakasun_spec, "deepseek_moe + window": windowed_moe_spec}),
           "tasadra": (TASADRA_SIZES, {"tasadra": tasadra_spec, "llama": plain_llama_spec})}
FP32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12      # FMA pipe at the maximum clock


def _runner(spec: DecoderSpec, tokens: int, max_len: int, seqs: int) -> GpuModelRunner:
    w = RunnerWeights.random(spec, f"cuda:{torch.cuda.current_device()}", seed=7)
    return GpuModelRunner(spec, w, num_blocks=tokens // 16 + 8, max_num_seqs=max(seqs, 8), max_num_batched_tokens=8192,
                          max_model_len=max_len)


def _batch(spec: DecoderSpec, seqs: int, context: int, decode: bool, seed: int = 0) -> StepBatch:
    """Whole prompts of ``context`` tokens, or one token of every sequence at position ``context - 1``."""
    b = _token_batch(spec.vocab_size, seqs, context, decode, seed)
    if spec.has_state:
        b.state_in = [2 * s if decode else -1 for s in range(seqs)]
        b.state_out = [2 * s + 1 for s in range(seqs)]
    return b


def _token_batch(vocab: int, seqs: int, context: int, decode: bool, seed: int) -> StepBatch:
    g = torch.Generator().manual_seed(seed)
    nb = -(-context // 16)
    tables = [list(range(s * nb, (s + 1) * nb)) for s in range(seqs)]
    ids = torch.randint(0, vocab, (seqs * (1 if decode else context),), generator=g).tolist()
    if decode:
        pos = [context - 1] * seqs
        slots = [t[-1] * 16 + (context - 1) % 16 for t in tables]
        return StepBatch(ids, pos, slots, seqs, [context] * seqs, tables, [], list(range(seqs)))
    pos = list(range(context)) * seqs
    slots = [t[p // 16] * 16 + p % 16 for t in tables for p in range(context)]
    return StepBatch(ids, pos, slots, 0, [context] * seqs, tables, [context] * seqs, [(s + 1) * context - 1 for s in range(seqs)])


def step_ms(runner: GpuModelRunner, b: StepBatch, iters: int = 20, warmup: int = 4) -> Dict[str, float]:
    for _ in range(warmup):
        runner.execute(b)
    times = []
    for _ in range(iters):
        torch.cuda.synchronize()
        a, z = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        runner.launch(b)
        z.record()
        runner.fetch()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(z))
    return {"ms": round(statistics.median(times), 4), "ms_min": round(min(times), 4)}


# ------------------------------------------------------------------------------------------------
# kernel by kernel
# ------------------------------------------------------------------------------------------------
RECORDED = ("gemm_tn", "grouped_gemm", "norm", "residual_norm", "row_norm", "embed_residual", "embed_gather", "rope_kv_append",
            "attn_decode", "attn_prefill", "moe_route", "moe_gather", "moe_combine", "sample", "sublayer_in", "wkv_mixer", "delta_mixer",
            "gemm_stacked", "latent_rows", "latent_rotate", "gemm_heads", "attn_latent", "latent_gather", "attn_expanded",
            "stream_in", "map_rows", "attn_finish")


@contextlib.contextmanager
def _record(calls: list):
    """Collects the calls of the kernel front end made inside the block (outermost calls only)."""
    saved = {n: getattr(K, n) for n in RECORDED}
    depth = [0]

    def wrap(name, fn):
        def f(*a, **kw):
            depth[0] += 1
            try:
                r = fn(*a, **kw)
            finally:
                depth[0] -= 1
            if depth[0] == 0:
                calls.append((name, fn, a, kw, r))
            return r
        return f

    for n, fn in saved.items():
        setattr(K, n, wrap(n, fn))
    try:
        yield
    finally:
        for n, fn in saved.items():
            setattr(K, n, fn)


def _nbytes(*ts) -> int:
    return sum(t.numel() * t.element_size() for t in ts if isinstance(t, torch.Tensor))


def _cost(name: str, a, kw, r, b: StepBatch) -> tuple:
    """(label, bytes moved, flops of the matrix pipe[, flops of the fp32 pipe]) of one call, counting every operand once."""
    q_lens = [1] * b.num_decode + list(b.prefill_q_lens)
    pairs_all = sum(q * n - q * (q - 1) // 2 for q, n in zip(q_lens, b.seq_lens))
    if name == "sublayer_in":
        x, parts = a[0], a[1]
        if kw.get("conv") is None and kw.get("mu") is None:
            y, ex = kw.get("y"), kw.get("experts")
            if kw.get("rows") is not None:
                n = r.shape[0] / x.shape[0]
                k = kw["routing"].K if ex is not None else 0
                return "final norm", int(n * (_nbytes(x, y) + k * _nbytes(y if y is not None else x)) + _nbytes(r)), 0.0
            if y is None and ex is None:
                return "norm", _nbytes(x, r[1]), 0.0
            return ("norm + residual" + (" + expert sum" if ex is not None else "") + " + norm",
                    _nbytes(x, y, ex, r[1]) + (_nbytes(x) if y is not None or ex is not None else 0), 0.0)
        live = sum(p.n for p in parts)
        state = sum(2 * live * t[0].numel() * 4 for t in (kw.get("conv_state"), kw.get("shift_state")) if t is not None)
        return (f"norms + conv" + (" + mixes" if kw.get("mu") is not None else ""),
                _nbytes(x, kw.get("y"), r[1]) + (_nbytes(x) if kw.get("y") is not None else 0) + state, 0.0)
    if name == "wkv_mixer":
        rkvg, ww, u, st, parts = a[0], a[1], a[2], a[4], a[5]
        per = st[0].numel()
        live = sum(p.n for p in parts)
        reads = live if b.num_decode else 0              # prompts start from nothing
        return "wkv", _nbytes(rkvg, ww, r) + 4 * per * (live + reads), 0.0, 5.0 * rkvg.shape[1] * per
    if name == "stream_in":
        x, y, n = kw.get("x"), kw.get("y"), 0 if kw.get("mix") is None else kw["mix"].numel() - 1
        share = r.shape[0] / (x if x is not None else kw["ids"]).shape[0]
        reads = (_nbytes(x, y) if x is not None else _nbytes(r)) + n * (_nbytes(kw["streams"][0]) if n else 0)
        label = ("embedding" if x is None else "residual") + (f" + average of {n + 1}" if n else "") + " + norm"
        return (label + (" + shift" if kw.get("shift") is not None else "") + (" (last rows)" if kw.get("rows") is not None else ""),
                int(share * reads) + _nbytes(r, kw.get("x_res"), kw.get("x_out")), 0.0)
    if name == "map_rows":
        own = kw["num_heads"] * kw["maps"] * kw["dim"] if a[1] is None else a[0].shape[1]
        kv = 0 if a[1] is None else a[0].shape[1] - kw["num_heads"] * kw["maps"] * kw["dim"]
        return "rows of two maps" + (" + append" if kv else ""), _nbytes(r) + (own + kv) * a[0].shape[0] * a[0].element_size(), 0.0
    if name == "attn_finish":
        gate = kw["gate"].element_size() * r.shape[0] * (r.shape[1] if kw["gate_kind"] == "element" else kw["gate"].shape[1])
        return ("difference of maps + gate" if kw["maps"] == 2 else "rotation back + gate"), _nbytes(a[0], r) + gate, 0.0
    if name == "delta_mixer":
        proj, state, parts = a[0], a[7], a[8]
        per, conv = state[0].numel(), a[6][0].numel() if a[6] is not None else 0
        H = state.shape[1]
        used = a[2].shape[1] + H + (0 if kw.get("decay") is not None else H * state.shape[3] + H)
        live = sum(p.n for p in parts)
        reads = live if b.num_decode else 0              # prompts start from nothing
        return ("delta rule", proj.shape[0] * used * proj.element_size() + _nbytes(r, kw.get("decay"), kw.get("gate")) + 4 * (per + conv) * (live + reads), 0.0,
                6.0 * proj.shape[0] * per)
    if name == "gemm_stacked":
        x, w = a
        return f"stacked gemm {x.shape[0]}x[{x.shape[1]}x{w.shape[1]}x{w.shape[2]}]", _nbytes(x, w, r), 2.0 * x.shape[1] * w.numel()
    if name == "latent_rows":
        return "latent norms + rotation + append", 2 * _nbytes(a[0]), 0.0
    if name == "latent_rotate":
        return "query rotation", 2 * a[0].shape[0] * a[0].shape[1] * a[3] * a[0].element_size(), 0.0
    if name == "gemm_heads":
        return (f"head gemm {a[0].shape[1]}x[{a[0].shape[0]}x{a[1].shape[1]}x{a[1].shape[2]}]", _nbytes(*a), 2.0 * a[0].shape[0] * a[1].numel())
    if name == "attn_latent":
        q, kc = a[0], a[1]
        return (("attn_latent (prompt)" if kw.get("q_start") is not None else "attn_latent (decode)"),
                _nbytes(q, r) + sum(b.seq_lens) * kc.shape[3] * kc.element_size(), 2.0 * pairs_all * q.shape[1] * (kc.shape[3] + a[2]))
    if name == "latent_gather":
        return "gather of cached latents", 2 * _nbytes(r), 0.0
    if name == "attn_expanded":
        q, kv, lat, vd = a[0], a[1], a[2], a[3]
        return "attn_expanded", _nbytes(q, kv, r) + lat.shape[0] * 2 * (q.shape[2] - kv.shape[1] // q.shape[1] + vd), \
            2.0 * pairs_all * q.shape[1] * (q.shape[2] + vd)
    if name == "gemm_tn":
        x, w = a[0], a[1]
        return (f"gemm {x.shape[0]}x{w.shape[0]}x{w.shape[1]}", _nbytes(x, w, r, kw.get("residual")),
                2.0 * x.shape[0] * w.shape[0] * w.shape[1])
    if name == "grouped_gemm":
        x, w, rt = a[0], a[1], a[2]
        used = min(w.shape[0], int((rt.counts > 0).sum()))
        return (f"expert gemm {x.shape[0]}x{w.shape[1]}x{w.shape[2]} ({'up' if kw.get('act') else 'down'})",
                _nbytes(x, r) + used * _nbytes(w[0]), 2.0 * x.shape[0] * w.shape[1] * w.shape[2])
    if name in ("attn_decode", "attn_prefill"):
        q, kc, vc = a[0], a[1], a[2]
        win = kw.get("window") or 10 ** 9
        chunk = kw.get("chunk") or 0
        lens = b.seq_lens
        q_lens = [1] * b.num_decode + list(b.prefill_q_lens)
        row = (kc.shape[3] + vc.shape[3]) * kc.shape[1] * kc.element_size()
        keys = sum(min(n, win + ql - 1) for n, ql in zip(lens, q_lens))
        pairs = 0
        for n, ql in zip(lens, q_lens):
            first = n - ql + 1
            full = max(0, min(n, win) - first + 1) if first <= win else 0       # queries that see fewer keys than the window
            pairs += full * (first + first + full - 1) // 2 + (ql - full) * min(n, win)
        if chunk:                                        # the chunked attentions of these designs have two maps: half a row per query
            seen = [sum(p % chunk + 1 for p in range(n - ql, n)) for n, ql in zip(lens, q_lens)]
            keys = sum(n - (n - ql) // chunk * chunk for n, ql in zip(lens, q_lens))
            return name + " (chunks, two maps)", _nbytes(q) // 2 + _nbytes(r) + keys * row, 2.0 * sum(seen) * q.shape[1] * (kc.shape[3] // 2 + vc.shape[3])
        return name, _nbytes(q, r) + keys * row, 2.0 * pairs * q.shape[1] * (kc.shape[3] + vc.shape[3])
    if name == "residual_norm":
        x, y, ex = a[0], a[1], kw.get("experts")
        return ("norm + residual" + (" + expert sum" if ex is not None else "")), _nbytes(x, x, y, ex, r), 0.0
    if name == "moe_combine":
        return "expert sum + residual", _nbytes(a[0], kw.get("residual"), r), 0.0
    if name == "norm":
        return "norm", _nbytes(a[0], r), 0.0
    if name == "rope_kv_append":
        q = kw["num_q_heads"] * kw["head_dim"] / a[0].shape[1]
        kv = 1.0 - q
        return "rope + append", int(_nbytes(a[0]) * (2 * q + 2 * kv)), 0.0
    if name == "moe_route" and a[0] is None:
        return "route + sort (logits given)", _nbytes(kw["logits"], r.topk_ids, r.topk_w, r.sorted_rows, r.row_slot), 0.0
    if name == "moe_route":
        return "route + sort", _nbytes(a[0], a[1]), 2.0 * a[0].shape[0] * a[1].numel()
    if name == "moe_gather":
        return "gather", _nbytes(a[0], r), 0.0
    ts = [t for t in (*a, *(r if isinstance(r, tuple) else (r,))) if isinstance(t, torch.Tensor)]
    if name in ("embed_gather", "embed_residual"):
        rs = r if isinstance(r, tuple) else (r,)
        return "embedding", _nbytes(*rs) + _nbytes(rs[-1]), 0.0
    if name == "row_norm":
        return "row norm", _nbytes(r) + 4 * r.numel(), 0.0
    return name, _nbytes(*ts), 0.0


def kernel_rows(runner: GpuModelRunner, b: StepBatch) -> List[dict]:
    """One row per distinct kernel call of a step: calls, microseconds each, fraction of its roofline."""
    hbm, tf, _ = _peaks()
    calls: list = []
    with _record(calls):
        runner.forward_logits(b)
    torch.cuda.synchronize()
    rows: Dict[str, dict] = {}
    for name, fn, a, kw, r in calls:
        label, nbytes, flops, *f32 = _cost(name, a, kw, r, b)
        if label in rows:
            rows[label]["calls"] += 1
            continue
        ms, _ = time_ms(lambda: fn(*a, **kw))
        floor = max(nbytes / (hbm * 1e9), flops / (tf * 1e12), (f32[0] if f32 else 0.0) / (FP32_TFLOPS * 1e12)) * 1e6
        rows[label] = {"kernel": label, "calls": 1, "us": round(ms * 1e3, 2), "roofline_us": round(floor, 2),
                       "fraction": round(floor / (ms * 1e3), 3)}
    return list(rows.values())


def wkv6_row(z: dict, seqs: int, tokens: int) -> dict:
    """RWKV-6's recurrence kernel at a Nipulorn layer's heads, in the same units as the table above (its output is neither
    normalised nor gated, so it moves the gate's bytes less)."""
    from ..ops import recurrent as R

    hbm, _, _ = _peaks()
    H, D = z["wkv"], z["wdim"]
    g = torch.Generator(device="cuda").manual_seed(1)
    r, k, v = (torch.randn(seqs, tokens, H * D, generator=g, device="cuda").to(torch.bfloat16) for _ in range(3))
    w, u = torch.rand(seqs, tokens, H * D, generator=g, device="cuda") * 4 - 5, torch.randn(H * D, generator=g, device="cuda")
    st = torch.zeros(seqs, H, D, D, device="cuda")
    ms, _ = time_ms(lambda: R.wkv6(r, k, v, w, u, H, st))
    nbytes = _nbytes(r, k, v, w, r) + 2 * _nbytes(st)
    floor = max(nbytes / (hbm * 1e9), 5.0 * seqs * tokens * H * D * D / (FP32_TFLOPS * 1e12)) * 1e6
    return {"kernel": "wkv6 (RWKV-6)", "calls": 1, "us": round(ms * 1e3, 2), "roofline_us": round(floor, 2), "fraction": round(floor / (ms * 1e3), 3)}


def wkv_row(z: dict, seqs: int, tokens: int, decode: bool) -> dict:
    """Nipulorn's recurrence kernel at the heads and state of a Bakasun layer's delta rule, in the units of the table above."""
    hbm, _, _ = _peaks()
    H, D, T = z["dh"], z["dd"], seqs * tokens
    g = torch.Generator(device="cuda").manual_seed(1)
    rkvg = torch.randn(4, T, H * D, generator=g, device="cuda").to(torch.bfloat16)
    ww, u = torch.rand(T, H * D, generator=g, device="cuda") * 4 - 5, torch.randn(H, D, generator=g, device="cuda")
    st, nw = torch.zeros(2 * seqs, H, D, D, device="cuda"), torch.ones(H * D, device="cuda")
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    si, so = i32([2 * s if decode else -1 for s in range(seqs)]), i32([2 * s + 1 for s in range(seqs)])
    p = K.Portions(0, T, seqs, tokens, None if decode else i32([s * tokens for s in range(seqs + 1)]), si, so)
    ms, _ = time_ms(lambda: K.wkv_mixer(rkvg, ww, u, nw, st, [p], eps=1e-5))
    nbytes = _nbytes(rkvg, ww, rkvg[0]) + 4 * st[0].numel() * seqs * (2 if decode else 1)
    floor = max(nbytes / (hbm * 1e9), 5.0 * T * H * D * D / (FP32_TFLOPS * 1e12)) * 1e6
    return {"kernel": "wkv (Nipulorn)", "calls": 1, "us": round(ms * 1e3, 2), "roofline_us": round(floor, 2), "fraction": round(floor / (ms * 1e3), 3)}


def delta_row(z: dict, seqs: int, tokens: int, decode: bool) -> dict:
    """Bakasun's delta rule (one decay per head, full gate) at the heads and state of a Tasadra layer, in the units of the table
    above."""
    hbm, _, _ = _peaks()
    H, D, T = z["dh"], z["dd"], seqs * tokens
    g = torch.Generator(device="cuda").manual_seed(1)
    used = 4 * H * D + 2 * H
    proj = torch.randn(T, (used + 7) // 8 * 8, generator=g, device="cuda").to(torch.bfloat16)
    conv = torch.full((4, 3 * H * D), 0.3, device="cuda", dtype=torch.bfloat16)
    zero, st = torch.zeros(H, device="cuda"), torch.zeros(2 * seqs, H, D, D, device="cuda")
    cs = torch.zeros(2 * seqs, 3, 3 * H * D, device="cuda")
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    si, so = i32([2 * s if decode else -1 for s in range(seqs)]), i32([2 * s + 1 for s in range(seqs)])
    p = K.Portions(0, T, seqs, tokens, None if decode else i32([s * tokens for s in range(seqs + 1)]), si, so)
    nw = torch.ones(D, device="cuda")
    ms, _ = time_ms(lambda: K.delta_mixer(proj, 0, conv, zero, zero, nw, cs, st, [p], kv_heads=H, eps=1e-5))
    nbytes = T * (used + H * D) * 2 + 4 * (st[0].numel() + cs[0].numel()) * seqs * (2 if decode else 1)
    floor = max(nbytes / (hbm * 1e9), 6.0 * T * H * D * D / (FP32_TFLOPS * 1e12)) * 1e6
    return {"kernel": "delta rule (Bakasun)", "calls": 1, "us": round(ms * 1e3, 2), "roofline_us": round(floor, 2), "fraction": round(floor / (ms * 1e3), 3)}


def main(design: str = "gekapel", sizes: Optional[List[str]] = None, kernels: bool = False) -> List[dict]:
    out = []
    table, arms = DESIGNS[design]
    for size in sizes or list(table):
        z = table[size]
        for arm, make in arms.items():
            spec = make(z)
            tokens = max([n * c for n, c in PREFILL] + [n * c for n, c in DECODE])
            runner = _runner(spec, tokens, max(c for _, c in PREFILL + DECODE) + 16, max(n for n, _ in DECODE))
            for kind, cases in (("prefill", PREFILL), ("decode", DECODE)):
                for n, c in cases:
                    b = _batch(spec, n, c, kind == "decode")
                    t = step_ms(runner, b)
                    row = {"size": size, "model": arm, "layers": spec.num_layers, "params_m": round(runner.w.nbytes() / 2e6),
                           "step": kind, "sequences": n, "context": c, **t,
                           "tokens_per_s": round(len(b.token_ids) / t["ms"] * 1e3)}
                    out.append(row)
                    print(row, flush=True)
                    if kernels:
                        rows = kernel_rows(runner, b)
                        if design == "nipulorn" and arm != "nipulorn":
                            rows.append(wkv6_row(z, n, 1 if kind == "decode" else c))
                        if design == "bakasun" and arm != "bakasun":
                            rows.append(wkv_row(z, n, 1 if kind == "decode" else c, kind == "decode"))
                        if design == "tasadra" and arm != "tasadra":
                            rows.append(delta_row(z, n, 1 if kind == "decode" else c, kind == "decode"))
                        for k in rows:
                            out.append({"size": size, "model": arm, "step": kind, "sequences": n, "context": c, **k})
                            print("   ", k, flush=True)
            K.check_device_errors()
            del runner
            torch.cuda.empty_cache()
    return out
