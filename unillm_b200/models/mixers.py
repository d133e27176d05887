"""Sublayer parts of per-layer specs beyond plain attention: latent attention, the wkv recurrence, the gated delta rule, the
difference of two attention maps, the input convolution, the token shift and the xIELU activation, as PyTorch on any device --
the whole-model path and the CPU runner; the serving kernels are ``csrc/attn/attn_latent.cu``, ``csrc/attn/attn_finish.cu``,
``csrc/wkv/wkv_mixer.cu``, ``csrc/delta/delta_mixer.cu``, ``csrc/norm/sublayer_in.cu`` and ``csrc/norm/stream_in.cu``.

State that a sequence carries lives in a dictionary per layer (``st``); a missing entry stands for the start of a sequence.

Latent attention follows DeepSeek-V2 ("DeepSeek-V2: A Strong, Economical, and Efficient Mixture-of-Experts Language
Model"), the recurrence RWKV-6 (the reference's ``models_v2/rwkv6.rs:483-553`` in another parametrisation), the delta rule
with decay "Gated Delta Networks: Improving Mamba2 with Delta Rule" (Yang, Kautz, Hatamizadeh), the difference of maps
"Differential Transformer" (Ye et al.).
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch
import torch.nn.functional as F

from ..ops import recurrent as R
from ..tensor_core import ops_fn
from .spec import LayerSpec

MU = ("r", "k", "v", "g", "w")           # order of the token-shift mixes in the parameter ``mu``


def mixer_shapes(ls: LayerSpec, H: int) -> Dict[str, Tuple[int, ...]]:
    """Canonical parameters of a latent, wkv or delta mixer."""
    n, d = ls.num_heads, ls.head_dim
    if ls.mixer == "latent":
        return {"w_dqkv": (ls.q_rank + ls.kv_rank + ls.rot_dim, H), "q_a_norm": (ls.q_rank,), "kv_a_norm": (ls.kv_rank,),
                "w_uq": (ls.q_size, ls.q_rank), "w_uk": (n * d, ls.kv_rank), "w_uv": (n * ls.v_head_dim, ls.kv_rank),
                **({"sink": (n,)} if ls.sink else {}), "wo": (H, ls.o_size)}
    if ls.mixer == "wkv":
        C = n * d
        return {"mu": (5, H), "w_rkvg": (4, C, H), "w_d1": (ls.decay_rank, H), "w_d2": (C, ls.decay_rank), "d0": (C,),
                "u": (n, d), "o_norm": (C,), "wo": (H, C)}
    if ls.mixer == "delta":
        channels = n * d
        decay = {"w_a1": (ls.decay_rank, H), "w_a2": (channels, ls.decay_rank)} if ls.decay == "channel" else {"w_a": (n, H)}
        gate = {"w_g1": (ls.gate_rank, H), "w_g2": (ls.o_size, ls.gate_rank)} if ls.low_rank_gate else {"w_g": (ls.o_size, H)}
        return {"w_qkv": (ls.conv_rows, H), "conv": (ls.conv_rows, ls.conv_taps), "w_b": (n, H), **decay, "A_log": (n,),
                "dt_bias": (channels if ls.decay == "channel" else n,), **gate, "o_norm": (ls.v_head_dim,), "wo": (H, ls.o_size)}
    raise ValueError(f"no such mixer: {ls.mixer!r}")


def join_parts(parts, shape) -> torch.Tensor:
    """The parameter that several tensors make up: stacked where it has one axis more than they have, else concatenated."""
    if len(parts) == 1:
        return parts[0]
    return torch.stack(list(parts)) if len(shape) == parts[0].dim() + 1 else torch.cat(list(parts), 0)


def split_parts(t: torch.Tensor, ls: LayerSpec, name: str, n: int):
    """Inverse of ``join_parts`` for the parameters above."""
    if n == 1:
        return [t]
    if name == "w_dqkv":
        return list(t.split([ls.q_rank, ls.kv_rank + ls.rot_dim]))
    if name in ("w_qkv", "conv"):
        return list(t.split([ls.k_size, ls.k_size, ls.o_size]))
    return list(t.unbind(0))


def input_conv(h: torch.Tensor, w: torch.Tensor, st: dict, key: str) -> torch.Tensor:
    """h [B, T, H] plus its causal depthwise convolution with the taps w [H, n] (the last tap meets the token itself)."""
    n = w.shape[1] - 1
    if key not in st:
        st[key] = torch.zeros(h.shape[0], n, h.shape[2], dtype=h.dtype, device=h.device)
    return h + R.causal_dwconv1d(h, w, None, st[key])


def token_shift(h: torch.Tensor, mix: torch.Tensor, st: dict) -> torch.Tensor:
    """h [B, T, H]: every token's values mixed with those of the token before it."""
    first = st["shift"] if "shift" in st else torch.zeros(h.shape[0], h.shape[2], dtype=h.dtype, device=h.device)
    back = torch.cat([first[:, None], h[:, :-1]], 1)
    st["shift"] = h[:, -1].clone()
    return h + (back - h) * mix.to(h.dtype)


def before_sublayer(h: torch.Tensor, w: torch.Tensor, st: dict, key: str) -> torch.Tensor:
    """What stands between a norm and its sublayer: a token shift or an input convolution, by the parameter's name."""
    return token_shift(h, w, st) if key == "shift" else input_conv(h, w, st, key)


def wkv(p: Dict[str, torch.Tensor], L: str, ls: LayerSpec, h: torch.Tensor, st: dict, eps: float) -> torch.Tensor:
    """h [B, T, H] -> [B, T, heads * dim], before the output projection."""
    B, T, H = h.shape
    n, d = ls.num_heads, ls.head_dim
    first = st["shift"] if "shift" in st else torch.zeros(B, H, dtype=h.dtype, device=h.device)
    dx = torch.cat([first[:, None], h[:, :-1]], 1) - h
    st["shift"] = h[:, -1].clone()
    mix = [h + dx * m.to(h.dtype) for m in p[L + "mu"]]
    r, k, v, g = (ops_fn.linear(x, w) for x, w in zip(mix, p[L + "w_rkvg"]))
    low = torch.tanh(F.linear(mix[4].float(), p[L + "w_d1"].float()))
    ww = F.linear(low, p[L + "w_d2"].float()) + p[L + "d0"].float()          # decay = exp(-exp(ww))
    if "wkv" not in st:
        st["wkv"] = torch.zeros(B, n, d, d, dtype=torch.float32, device=h.device)
    y = R.wkv6(r, k, v, ww.contiguous(), p[L + "u"].float(), n, st["wkv"]).float().reshape(B, T, n, d)
    y = y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)
    return (y.reshape(B, T, n * d) * p[L + "o_norm"].float() * F.silu(g.float())).to(h.dtype)


def delta(p: Dict[str, torch.Tensor], L: str, ls: LayerSpec, h: torch.Tensor, st: dict, eps: float) -> torch.Tensor:
    """Gated delta rule: h [B, T, H] -> [B, T, heads * value size], before the output projection."""
    B, T, _ = h.shape
    n, g, dk, dv = ls.num_heads, ls.num_kv_heads, ls.head_dim, ls.v_head_dim
    y = ops_fn.linear(h, p[L + "w_qkv"]).float()
    if "conv" not in st:
        st["conv"] = torch.zeros(B, ls.conv_taps - 1, y.shape[2], dtype=torch.float32, device=h.device)
        st["delta"] = torch.zeros(B, n, dk, dv, dtype=torch.float32, device=h.device)
    y = F.silu(R.causal_dwconv1d(y, p[L + "conv"], None, st["conv"]))
    q, k, v = y.split([ls.k_size, ls.k_size, ls.o_size], dim=-1)
    unit = lambda x: x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)
    q, k = (unit(x.reshape(B, T, g, dk)).repeat_interleave(n // g, dim=2) for x in (q, k))
    beta = torch.sigmoid(ops_fn.linear(h, p[L + "w_b"]).float())
    if ls.decay == "channel":
        raw = F.linear(ops_fn.linear(h, p[L + "w_a1"]).float(), p[L + "w_a2"].float()) + p[L + "dt_bias"].float()
        keep = torch.exp(-torch.exp(p[L + "A_log"].float())[:, None] * F.softplus(raw).reshape(B, T, n, dk))
    else:
        keep = torch.exp(-torch.exp(p[L + "A_log"].float()) * F.softplus(ops_fn.linear(h, p[L + "w_a"]).float() + p[L + "dt_bias"].float()))
    o, st["delta"] = R.delta_rule(q * dk ** -0.5, k, v.reshape(B, T, n, dv), keep, beta, st["delta"])
    o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * p[L + "o_norm"].float()
    g = ops_fn.linear(ops_fn.linear(h, p[L + "w_g1"]), p[L + "w_g2"]) if ls.low_rank_gate else ops_fn.linear(h, p[L + "w_g"])
    return (o.reshape(B, T, n * dv) * ops_fn.activation(ls.gate_act)(g.float())).to(h.dtype)


def diff_lambda(ls: LayerSpec, lambdas: torch.Tensor) -> float:
    """The factor on the second map of a differential attention; ``lambdas`` [4, head_dim]: q and k of map 1, of map 2."""
    a = lambdas.detach().double().cpu()
    return float(torch.exp((a[0] * a[1]).sum()) - torch.exp((a[2] * a[3]).sum())) + ls.diff


def difference(ls: LayerSpec, lambdas: torch.Tensor, y: torch.Tensor, eps: float) -> torch.Tensor:
    """y [.., heads * 2, v size], the two maps of a head side by side -> [.., heads, v size]."""
    a1, a2 = y.unflatten(-2, (ls.num_heads, 2)).unbind(-2)
    o = a1 - diff_lambda(ls, lambdas) * a2
    return o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * (1.0 - ls.diff)


def latent_project(p: Dict[str, torch.Tensor], L: str, ls: LayerSpec, h: torch.Tensor, eps: float):
    """(queries [.., heads, dim + rot_dim], normalised latents [.., kv_rank], key part [.., 1, rot_dim]) before rotation."""
    cq, c, kr = ops_fn.linear(h, p[L + "w_dqkv"]).split([ls.q_rank, ls.kv_rank, ls.rot_dim], dim=-1)
    q = ops_fn.linear(ops_fn.rms_norm(cq.contiguous(), p[L + "q_a_norm"], eps), p[L + "w_uq"])
    c = ops_fn.rms_norm(c.contiguous(), p[L + "kv_a_norm"], eps)
    return q.reshape(*h.shape[:-1], ls.num_heads, ls.head_dim + ls.rot_dim), c, kr.unsqueeze(-2)


def latent_expand(p: Dict[str, torch.Tensor], L: str, ls: LayerSpec, rows: torch.Tensor):
    """Cached rows [.., S, kv_rank + rot_dim] -> keys [.., heads, S, dim + rot_dim] and values [.., heads, S, v size]."""
    c, kr = rows.split([ls.kv_rank, ls.rot_dim], dim=-1)
    lead = rows.shape[:-1]
    k = ops_fn.linear(c.contiguous(), p[L + "w_uk"]).reshape(*lead, ls.num_heads, ls.head_dim).transpose(-2, -3)
    v = ops_fn.linear(c.contiguous(), p[L + "w_uv"]).reshape(*lead, ls.num_heads, ls.v_head_dim).transpose(-2, -3)
    kr = kr.unsqueeze(-3).expand(*k.shape[:-1], ls.rot_dim)
    return torch.cat([k, kr], -1), v


def xielu_coefficients(act: torch.Tensor) -> Tuple[float, float]:
    """The two learned numbers as the activation uses them: softplus(p) in front of z^2, 1/2 + softplus(q) in front of the
    exponential part."""
    a = F.softplus(act.detach().double().cpu())
    return float(a[0]), float(a[1]) + 0.5


def xielu(z: torch.Tensor, act: torch.Tensor) -> torch.Tensor:
    """z > 0: a z^2 + z / 2; z <= 0: b (e^z - 1 - z) + z / 2."""
    a, b = xielu_coefficients(act)
    return torch.where(z > 0, a * z * z, b * (torch.expm1(z) - z)) + 0.5 * z
