"""``GpuModelRunner``: executes one engine step of a decoder model on one B200 with the hand-written
sm_100a kernels and a paged KV cache.

Per layer (tensor-parallel rank view):

    norm (K5)  ->  QKV GEMM (K1, tcgen05)  ->  RoPE + KV append (K6)  ->  paged attention (K3 prefill rows,
    K4 decode rows, optional cascade over a radix-shared prefix)  ->  o_proj GEMM with the residual add in
    its epilogue  ->  norm  ->  gate/up GEMM with SwiGLU in its epilogue (K2)  ->  down GEMM + residual

then final norm on the rows that are sampled, the (vocab-parallel) lm_head GEMM and the device sampler
(K8).  Token metadata for a step arrives as ONE packed int32 buffer copied from pinned host memory;
pure-decode steps are captured in CUDA graphs keyed by (padded batch, shared-prefix length).

Tensor parallelism (``TpContext``): column-parallel QKV / gate-up, row-parallel o / down, KV heads and
the vocabulary sharded.  With ``fused=True`` the two reductions per layer run inside the GEMM and norm
kernels over NVSwitch peer memory (GEMM epilogue pushes rows to the owning rank = reduce-scatter, the
norm kernel sums the partials, normalises its token shard and pushes it to every rank = all-gather,
and the next GEMM's TMA producer waits on the arrival counters); with ``fused=False`` the same math uses
NCCL all-reduce between library-style separate kernels -- the measured baseline.

Reference counterpart: the per-token loop of ``UniLLMBackend::generate`` / ``LlamaModelV2::forward_with_cache``
(``crates/runtime/src/benchmark/unillm_backend.rs:69-211``, ``models_v2/llama.rs:421-464, 654-680,
1027-1156``), which is batch-1, CPU-only and uses a contiguous cache.
"""
from __future__ import annotations

import dataclasses
import math
import os
import time
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from ..models.spec import DecoderSpec
from ..ops import cuda_ops as K
from ..precompute import alibi_slopes, rope_gain, rope_inv_freq
from ..types import InvalidInput, UnsupportedOperation


class DeviceStepError(RuntimeError):
    """A kernel of a launched step recorded a problem in the device error word (a bounded wait that gave up, an
    out-of-range block-table entry or slot): the step's sampled ids are garbage and must not be used."""

    NAMES = {1: "mbarrier wait timed out", 2: "flag wait timed out (peer or producer missing)",
             3: "index out of range", 4: "bad argument"}

    def __init__(self, code: int, detail: int):
        super().__init__(f"device error {code} ({self.NAMES.get(code, '?')}), detail {detail}")
        self.code, self.detail = code, detail


@dataclass
class StepBatch:
    """Host-side description of one engine step (built by the scheduler).

    Token rows are ordered: first the ``num_decode`` decode sequences (one row each), then the prefill
    chunks.  ``seq_lens`` is the KV length of each sequence after this step's tokens are appended."""

    token_ids: List[int]
    positions: List[int]
    slot_mapping: List[int]
    num_decode: int
    seq_lens: List[int]
    block_tables: List[List[int]]
    prefill_q_lens: List[int] = field(default_factory=list)
    sample_rows: List[int] = field(default_factory=list)
    shared_prefix_len: int = 0          # tokens of KV that ALL decode sequences share (whole blocks)
    prefill_shares_prefix: bool = False  # the prefill chunks start at or after that prefix and share its blocks too
    # sampling (per sampled row); None = greedy
    temperature: Optional[List[float]] = None
    top_p: Optional[List[float]] = None
    top_k: Optional[List[int]] = None
    seed: int = 0
    step: int = 0
    # per decode row: index (in sample order) of the PREVIOUS step's output that is this row's input token, or -1
    # when ``token_ids`` already holds it.  Lets a step be launched before the host has read the previous
    # step's samples.
    token_src: Optional[List[int]] = None
    # recurrent models, per sequence (decode rows, then prefill chunks): rows of the state tensors to read (-1: the
    # sequence starts, zero state) and to write (-1: none)
    state_in: Optional[List[int]] = None
    state_out: Optional[List[int]] = None


def shard_rows(w: torch.Tensor, rank: int, world: int) -> torch.Tensor:
    n = w.shape[0] // world
    return w[rank * n:(rank + 1) * n]


def shard_cols(w: torch.Tensor, rank: int, world: int) -> torch.Tensor:
    n = w.shape[1] // world
    return w[:, rank * n:(rank + 1) * n]


class QWeight:
    """A projection weight kept block-quantised on the device (ggml block layout, rows independent): what the
    reference keeps as ``QMatMul`` for ``*_proj`` / ``lm_head`` tensors of a GGUF checkpoint
    (``crates/runtime/src/weight_loader_core.rs:554-584``, used at ``models_v2/llama.rs:1184-1195``)."""

    __slots__ = ("blocks", "qtype", "shape")

    def __init__(self, blocks: torch.Tensor, qtype: int, shape):
        self.blocks, self.qtype, self.shape = blocks, qtype, tuple(shape)

    def nbytes(self) -> int:
        return self.blocks.numel()


QUANT_NAMES = {"q4_0": 2, "q8_0": 8, "q4_k": 12}


def _round8(n: int) -> int:
    return (n + 7) // 8 * 8


def _pad(t: torch.Tensor, dim: int, size: int) -> torch.Tensor:
    """``t`` with zeros appended along ``dim`` up to ``size`` entries."""
    n = size - t.shape[dim]
    if n == 0:
        return t
    shape = list(t.shape)
    shape[dim] = n
    return torch.cat([t, t.new_zeros(shape)], dim)


@dataclass(frozen=True)
class KernelHeads:
    """One layer's attention heads as this rank's kernels see them: head sizes are rounded up to multiples of 8 (16-byte
    rows); the pad entries of the projections are zero, so they add nothing to scores or outputs.

    Latent attention: one cache row of ``dk`` = kv_rank + rot elements whose first ``dv`` = kv_rank are the value; ``dim``,
    ``rot``, ``vdim`` and ``q_rank`` are the padded sizes around it.  wkv: ``dk`` x ``dv`` states, no cache row.

    With ``maps`` > 1 a key row holds the keys of all maps and every (head, map) is a query head of the kernels: ``hq`` counts
    those, ``dk`` is the whole row.  ``gate_rows``: rows of an output gate behind Q, K and V of the input projection."""

    hq: int
    hkv: int
    kv_lo: int
    dk: int
    dv: int
    own_kv: bool
    dim: int = 0
    rot: int = 0
    vdim: int = 0
    q_rank: int = 0
    delta: Optional["DeltaHeads"] = None         # of the layer's gated delta rule (beside the attention, or its only mixer)
    maps: int = 1
    gate_rows: int = 0

    @property
    def qkv_rows(self) -> int:
        return self.hq * (self.dk // self.maps) + (self.hkv * (self.dk + self.dv) if self.own_kv else 0)

    @property
    def cache_row(self) -> int:
        if not self.own_kv:
            return 0
        return self.dk if self.q_rank else self.hkv * (self.dk + self.dv)


@dataclass(frozen=True)
class DeltaHeads:
    """A gated delta rule as the kernels see it: ``hq`` heads of ``dk`` x ``dv`` states, ``hk`` query / key heads, head sizes
    rounded up to multiples of 8.  Its rows of the layer's input projection are [Q | K | V | gate | b | a], behind those of an
    attention it stands beside; its columns of the output projection follow that one's.  With low-rank decays per channel and a
    low-rank gate (``ra``, ``rg`` > 0, rounded up) they are [Q | K | V | b | first product of the decays | of the gate]."""

    hq: int
    hk: int
    dk: int
    dv: int
    taps: int
    row0: int
    col0: int
    ra: int = 0
    rg: int = 0

    @property
    def conv_rows(self) -> int:
        return 2 * self.hk * self.dk + self.hq * self.dv

    @property
    def low_col(self) -> int:
        """First column of the low-rank products."""
        return self.conv_rows + _round8(self.hq)

    @property
    def rows(self) -> int:
        if self.ra:
            return self.low_col + self.ra + self.rg
        return self.conv_rows + self.hq * self.dv + _round8(2 * self.hq)

    @property
    def cols(self) -> int:
        return self.hq * self.dv


class RunnerWeights:
    """Device weights of one rank in kernel layout (fused QKV / gate-up, TP-sharded), bf16 or fp32.  For per-layer specs, row
    sizes that are not multiples of 8 (model width, head sizes, feed-forward widths) are zero-padded to the next one."""

    def __init__(self, spec: DecoderSpec, params: Dict[str, torch.Tensor], device, rank: int = 0, world: int = 1,
                 expert_parallel: bool = False, dtype: torch.dtype = torch.bfloat16):
        self._init_layout(spec, rank, world, expert_parallel, dtype)
        s = spec
        H = self.width

        def dev(t):
            return t.to(device=device, dtype=dtype).contiguous()

        def heads(t, n, d, dp, lo, cnt):
            """Rows (or elements) of heads [lo, lo + cnt) of a [n * d, ...] tensor, every head padded to dp rows."""
            t = t.reshape(n, d, *t.shape[1:])[lo:lo + cnt]
            t = _pad(t, 1, dp)
            return t.reshape(cnt * dp, *t.shape[2:])

        self.t: Dict[str, torch.Tensor] = {}
        p = params
        self.t["embed"] = dev(_pad(p["embed"], 1, H))
        for n in ("embed_norm.w", "embed_norm.b", "final_norm.w", "final_norm.b"):
            if n in p:
                self.t[n] = dev(_pad(p[n], 0, H))
        if "final_norm.alpha" in p:
            self.slopes["final_norm"] = float(p["final_norm.alpha"])
        for n in ("pos_embed", "project_in", "project_out"):
            if n in p:
                self.t[n] = dev(p[n])
        lm = p["embed"] if s.tie_embeddings else p["lm_head"]
        self.t["lm_head"] = dev(_pad(shard_rows(lm, rank, world), 1, H)) if (world > 1 or not s.tie_embeddings) \
            else self.t["embed"]
        if "lm_head_bias" in p:
            self.t["lm_head_bias"] = dev(shard_rows(p["lm_head_bias"], rank, world))
        for i in range(s.num_layers):
            L = f"layers.{i}."
            ls, kh = s.layer(i), self.heads[i]
            for n in ("ln1.w", "ln1.b", "ln2.w", "ln2.b", "ln1b.w", "ln2b.w"):
                if L + n in p:
                    self.t[L + n] = dev(_pad(p[L + n], 0, H))
            for n in ("conv1", "conv2"):
                if L + n in p:                                # [taps, H]: neighbouring threads read neighbouring channels
                    self.t[L + n] = dev(_pad(p[L + n].t(), 1, H))
            self.slopes.update({L + n: float(p[L + n + ".alpha"]) for n in ("ln1", "ln2") if L + n + ".alpha" in p})
            if L + "shift" in p:
                self.t[L + "shift"] = dev(_pad(p[L + "shift"], 0, H))
            if L + "dwa" in p:
                self.t[L + "dwa"] = p[L + "dwa"].to(device=device, dtype=torch.float32).contiguous()
            if L + "lambdas" in p:
                from ..models.mixers import diff_lambda

                self.lams[i] = diff_lambda(ls, p[L + "lambdas"])
            if L + "act" in p:
                from ..models.mixers import xielu_coefficients

                self.act_params[i] = xielu_coefficients(p[L + "act"])
            if ls.mixer != "attention":
                self._mixer_weights(i, p, device, dev, heads)
                self._ff_weights(i, p, dev)
                continue
            for n, cnt in (("q_norm", ls.num_heads), ("k_norm", ls.num_kv_heads)):
                if L + n in p and s.qk_norm_kind(i) == "row":
                    self.t[L + n] = dev(heads(p[L + n], cnt, ls.head_dim, kh.dk, 0, cnt))
                elif L + n in p:
                    self.t[L + n] = dev(_pad(p[L + n], 0, kh.dk))
            if ls.fixed_sink is not None:
                self.t[L + "sink"] = torch.full((kh.hq,), ls.fixed_sink, dtype=torch.float32, device=device)
            if L + "sink" in p:
                self.t[L + "sink"] = p[L + "sink"][rank * kh.hq:(rank + 1) * kh.hq].to(device=device, dtype=torch.float32).contiguous()

            def fused_rows(t):
                parts = t.split([ls.q_size, ls.k_size, ls.v_size]) if kh.own_kv else (t,)
                n, d = ls.maps, kh.dk // ls.maps
                out = [heads(parts[0], ls.num_heads * n, ls.head_dim, d, rank * kh.hq, kh.hq)]
                if kh.own_kv:
                    out.append(heads(parts[1], ls.num_kv_heads * n, ls.head_dim, d, kh.kv_lo * n, kh.hkv * n))
                    out.append(heads(parts[2], ls.num_kv_heads, ls.v_head_dim, kh.dv, kh.kv_lo, kh.hkv))
                return torch.cat(out, 0)

            w_in = fused_rows(p[L + "wqkv"])
            if ls.out_gate:
                g = p[L + "w_og"]
                g = _pad(g, 0, kh.gate_rows) if ls.out_gate == "head" else heads(g, ls.num_heads, ls.v_head_dim, kh.dv, 0, ls.num_heads)
                w_in = torch.cat([w_in, g])
            self.t[L + "wqkv"] = dev(_pad(w_in, 1, H))
            if L + "bqkv" in p:
                self.t[L + "bqkv"] = dev(_pad(fused_rows(p[L + "bqkv"]), 0, kh.qkv_rows + kh.gate_rows))
            wo = p[L + "wo"].t()                              # [heads * v size, H]: sharded and padded like the head rows
            n = kh.hq // ls.maps
            self.t[L + "wo"] = dev(_pad(heads(wo, ls.num_heads, ls.v_head_dim, kh.dv, rank * n, n).t(), 0, H))
            if L + "bo" in p:
                self.t[L + "bo"] = dev(p[L + "bo"] if rank == 0 else torch.zeros_like(p[L + "bo"]))
            if kh.delta is not None:
                self._beside_weights(i, p, device, dev, heads)
            self._ff_weights(i, p, dev)

    def _ff_weights(self, i: int, p, dev) -> None:
        """Feed-forward of one layer, dense or a mixture."""
        self._dense_weights(i, p, dev)
        L, ls, H, rank, world = f"layers.{i}.", self.spec.layer(i), self.width, self.rank, self.world
        if L + "router" not in p:
            return
        # experts: tensor-parallel inside each expert here; expert-parallel layouts are built by MoeRunner
        m = ls.moe
        self.t[L + "router"] = dev(_pad(p[L + "router"], 1, H))
        if m.router_bias:
            self.t[L + "router_b"] = dev(p[L + "router_b"])
        if m.correction:
            self.t[L + "correction"] = dev(p[L + "correction"])
        if m.shared_gate:
            self.t[L + "shared_sg"] = dev(_pad(p[L + "shared_sg"], 1, H)).view(-1)
        self._router_full(L, m)

        def up_rows(t, r, w):
            """This rank's rows of an up (or [gate; up]) matrix [.., rows, H], each half padded to 8."""
            halves = t.chunk(2, -2) if m.gated else (t,)
            n = halves[0].shape[-2] // w
            cut = [_pad(h[..., r * n:(r + 1) * n, :], h.dim() - 2, self._round(n)) for h in halves]
            return _pad(torch.cat(cut, -2), t.dim() - 1, H)

        def down_cols(t, r, w):
            n = t.shape[-1] // w
            return _pad(_pad(t[..., r * n:(r + 1) * n], t.dim() - 1, self._round(n)), t.dim() - 2, H)

        gu, dn = p[L + "experts_gate_up"], p[L + "experts_down"]
        if self.ep:
            # expert parallel: whole experts [expert_lo, expert_lo + experts_local) live here
            lo, hi = self.expert_lo, self.expert_lo + self.experts_local
            self.t[L + "experts_gate_up"] = dev(up_rows(gu[lo:hi], 0, 1))
            self.t[L + "experts_down"] = dev(down_cols(dn[lo:hi], 0, 1))
        else:
            self.t[L + "experts_gate_up"] = dev(up_rows(gu, rank, world))
            self.t[L + "experts_down"] = dev(down_cols(dn, rank, world))
        if L + "shared_gate_up" in p:
            self.t[L + "shared_gate_up"] = dev(up_rows(p[L + "shared_gate_up"], rank, world))
            self.t[L + "shared_down"] = dev(down_cols(p[L + "shared_down"], rank, world))

    def _router_full(self, L: str, m) -> None:
        """Router rows and the shared expert's gate as one matrix of whole 8-row groups, for steps with many tokens."""
        if self.dtype != torch.bfloat16 or m.router_bias or self.ep:
            return
        rows = [self.t[L + "router"]] + ([self.t[L + "shared_sg"][None]] if m.shared_gate else [])
        w = torch.cat(rows)
        self.t[L + "router_full"] = _pad(w, 0, _round8(w.shape[0]))

    def _dense_weights(self, i: int, p, dev) -> None:
        """Dense feed-forward of one layer."""
        L, rank, world = f"layers.{i}.", self.rank, self.world
        if L + "w_gate_up" in p:
            halves = [shard_rows(t, rank, world) for t in p[L + "w_gate_up"].chunk(2, 0)]
            self.t[L + "w_gate_up"] = dev(_pad(torch.cat([_pad(t, 0, self._round(t.shape[0])) for t in halves], 0), 1, self.width))
        if L + "w_up" in p:
            up = shard_rows(p[L + "w_up"], rank, world)
            self.t[L + "w_up"] = dev(_pad(_pad(up, 0, self._round(up.shape[0])), 1, self.width))
            if L + "b_up" in p:
                self.t[L + "b_up"] = dev(_pad(shard_rows(p[L + "b_up"], rank, world), 0, self._round(up.shape[0])))
        if L + "w_down" in p:
            dn = shard_cols(p[L + "w_down"], rank, world)
            self.t[L + "w_down"] = dev(_pad(_pad(dn, 1, self._round(dn.shape[1])), 0, self.width))
            if L + "b_down" in p:
                self.t[L + "b_down"] = dev(_pad(p[L + "b_down"] if rank == 0 else torch.zeros_like(p[L + "b_down"]), 0, self.width))

    def _beside_weights(self, i: int, p, device, dev, heads) -> None:
        """The gated delta rule beside a layer's attention: one input and one output projection for both mixers.  The output
        projection's result is multiplied by the first mixer's factor, so the second one's norm weight carries the ratio."""
        L, ls, d = f"layers.{i}.", self.spec.layer(i), self.heads[i].delta
        sa, sb = ls.scales
        first = self.t.pop(L + "wqkv")
        w, wo = self._delta_weights(L + "beside.", ls.beside, d, p, L, device, heads, sb / sa if sa else sb)
        self.t[L + "w_in"] = torch.cat([first, dev(w)], 0)
        if L + "bqkv" in self.t:
            b = self.t.pop(L + "bqkv")
            self.t[L + "b_in"] = _pad(b, 0, b.shape[0] + d.rows)
        self.t[L + "wo"] = torch.cat([self.t[L + "wo"] * (1.0 if sa else 0.0), dev(wo)], 1).contiguous()

    def _delta_weights(self, src: str, ls, d: "DeltaHeads", p, L: str, device, heads, factor: float):
        """Parameters ``src`` of a gated delta rule into kernel layout; returns the rows of its input projection and its output
        projection."""
        t, H, n, g = self.t, self.width, ls.num_heads, ls.num_kv_heads

        def f32(x):
            return x.to(device=device, dtype=torch.float32).contiguous()

        def qkv_rows(x):
            q, k, v = x.split([ls.k_size, ls.k_size, ls.o_size])
            return torch.cat([heads(q, g, ls.head_dim, d.dk, 0, g), heads(k, g, ls.head_dim, d.dk, 0, g),
                              heads(v, n, ls.v_head_dim, d.dv, 0, n)])

        t[L + "delta_conv"] = qkv_rows(p[src + "conv"]).t().to(device=device, dtype=self.dtype).contiguous()
        t[L + "a_log"], t[L + "dt_bias"] = f32(p[src + "A_log"]), f32(p[src + "dt_bias"])
        t[L + "o_norm"] = f32(_pad(p[src + "o_norm"].float() * factor, 0, d.dv))
        wo = _pad(heads(p[src + "wo"].t(), n, ls.v_head_dim, d.dv, 0, n).t(), 0, H)
        if d.ra:
            low = lambda x, r: x.to(device=device, dtype=self.dtype).contiguous() if x.shape[1] == r else _pad(x, 1, r).to(device=device, dtype=self.dtype)
            t[L + "dt_bias"] = f32(heads(p[src + "dt_bias"], n, ls.head_dim, d.dk, 0, n))
            t[L + "w_a2"] = low(heads(p[src + "w_a2"], n, ls.head_dim, d.dk, 0, n), d.ra)
            t[L + "w_g2"] = low(heads(p[src + "w_g2"], n, ls.v_head_dim, d.dv, 0, n), d.rg)
            w = torch.cat([qkv_rows(p[src + "w_qkv"]), _pad(p[src + "w_b"], 0, _round8(n)), _pad(p[src + "w_a1"], 0, d.ra),
                           _pad(p[src + "w_g1"], 0, d.rg)])
            return _pad(w, 1, H), wo
        ba = torch.cat([p[src + "w_b"], p[src + "w_a"]])
        w = torch.cat([qkv_rows(p[src + "w_qkv"]), heads(p[src + "w_g"], n, ls.v_head_dim, d.dv, 0, n), _pad(ba, 0, _round8(2 * n))])
        return _pad(w, 1, H), wo

    def _mixer_weights(self, i: int, p, device, dev, heads) -> None:
        """Latent attention, wkv or delta parameters of one layer in kernel layout."""
        L, ls, kh, H = f"layers.{i}.", self.spec.layer(i), self.heads[i], self.width
        n, t = ls.num_heads, self.t

        def f32(x):
            return x.to(device=device, dtype=torch.float32).contiguous()

        def head_cols(w, d, dp):                              # [H, heads * d] -> [width, heads * dp]
            return dev(_pad(heads(w.t(), n, d, dp, 0, n).t(), 0, H))

        if ls.mixer == "delta":
            w, wo = self._delta_weights(L, ls, kh.delta, p, L, device, heads, 1.0)
            t[L + "w_in"], t[L + "wo"] = dev(w), dev(wo)
            return
        if ls.mixer == "wkv":
            d, dp, rank = ls.head_dim, kh.dk, self._round(ls.decay_rank)
            t[L + "mu"] = dev(_pad(p[L + "mu"], 1, H))
            t[L + "w_rkvg"] = dev(torch.stack([_pad(heads(w, n, d, dp, 0, n), 1, H) for w in p[L + "w_rkvg"]]))
            t[L + "w_d1"] = dev(_pad(_pad(p[L + "w_d1"], 0, rank), 1, H))
            t[L + "w_d2"] = dev(_pad(heads(p[L + "w_d2"], n, d, dp, 0, n), 1, rank))
            t[L + "d0"] = dev(heads(p[L + "d0"], n, d, dp, 0, n))
            t[L + "u"] = f32(_pad(p[L + "u"], 1, dp))
            t[L + "o_norm"] = f32(heads(p[L + "o_norm"], n, d, dp, 0, n))
            t[L + "wo"] = head_cols(p[L + "wo"], d, dp)
            return
        dq, dc, dr = p[L + "w_dqkv"].split([ls.q_rank, ls.kv_rank, ls.rot_dim])
        t[L + "w_dqkv"] = dev(_pad(torch.cat([_pad(dq, 0, kh.q_rank), _pad(dc, 0, kh.dv), _pad(dr, 0, kh.rot)]), 1, H))
        t[L + "q_a_norm"], t[L + "kv_a_norm"] = dev(_pad(p[L + "q_a_norm"], 0, kh.q_rank)), dev(_pad(p[L + "kv_a_norm"], 0, kh.dv))
        uq = p[L + "w_uq"].reshape(n, ls.head_dim + ls.rot_dim, ls.q_rank)
        uq = torch.cat([_pad(uq[:, :ls.head_dim], 1, kh.dim), _pad(uq[:, ls.head_dim:], 1, kh.rot)], 1)
        t[L + "w_uq"] = dev(_pad(uq.flatten(0, 1), 1, kh.q_rank))
        uk = _pad(_pad(p[L + "w_uk"].reshape(n, ls.head_dim, ls.kv_rank), 1, kh.dim), 2, kh.dv)
        uv = _pad(_pad(p[L + "w_uv"].reshape(n, ls.v_head_dim, ls.kv_rank), 1, kh.vdim), 2, kh.dv)
        t[L + "w_uk_t"] = dev(uk.transpose(1, 2))             # [heads, kv_rank, dim]: taken to the query side
        t[L + "w_uv"] = dev(uv)                               # [heads, vdim, kv_rank]
        if self.dtype == torch.bfloat16 and self.expandable(i):
            t[L + "w_ukv"] = dev(torch.cat([uk, uv], 1).flatten(0, 1))       # [heads * (dim + vdim), kv_rank]: long prompts
        if ls.sink:
            t[L + "sink"] = f32(p[L + "sink"])
        t[L + "wo"] = head_cols(p[L + "wo"], ls.v_head_dim, kh.vdim)

    def _init_layout(self, spec: DecoderSpec, rank: int, world: int, expert_parallel: bool, dtype=torch.bfloat16) -> None:
        """Everything that follows from the spec and the rank alone: head layout per layer, padded width, shard sizes."""
        self.spec, self.rank, self.world, self.dtype = spec, rank, world, dtype
        self._round = _round8 if spec.layers is not None else (lambda n: n)
        self._set_ep(expert_parallel)
        if spec.vocab_size % world != 0:
            raise InvalidInput(f"vocab {spec.vocab_size} not divisible by tensor parallel size {world}")
        self.vocab_shard = spec.vocab_size // world
        self.width = self._round(spec.hidden_size)
        self.heads: List[KernelHeads] = []
        self.act_params: Dict[int, Tuple[float, float]] = {}   # coefficients of activations with learned numbers, per layer
        self.slopes: Dict[str, float] = {}                     # of Dynamic Tanh norms, by the norm's name
        self.lams: Dict[int, float] = {}                       # factor on the second map of differential attentions, per layer
        r8 = self._round
        for i in range(spec.num_layers):
            ls = spec.layer(i)
            if ls.mixer != "attention" or spec.norm_placement == "both" or spec.norm == "tanh" or ls.maps > 1 or ls.out_gate or ls.value_rope:
                if world > 1:
                    raise UnsupportedOperation("latent attention, wkv and delta layers, output gates, rotated values, differential attention, "
                                               "Dynamic Tanh and norms on both sides of a sublayer: one rank")
            if ls.mixer == "delta":
                self.heads.append(KernelHeads(ls.num_heads, 0, 0, 8, 8, False, delta=self._delta_heads(ls, 0, 0)))
                continue
            if ls.mixer == "wkv":
                d = r8(ls.head_dim)
                self.heads.append(KernelHeads(ls.num_heads, 0, 0, d, d, False))
                continue
            if ls.mixer == "latent":
                rank_p, rot = r8(ls.kv_rank), r8(ls.rot_dim)
                self.heads.append(KernelHeads(ls.num_heads, 1, 0, rank_p + rot, rank_p, True, r8(ls.head_dim), rot,
                                              r8(ls.v_head_dim), r8(ls.q_rank)))
                continue
            if ls.num_heads % world != 0:
                raise InvalidInput(f"{ls.num_heads} heads not divisible by tensor parallel size {world}")
            if ls.moe is not None and not self.ep and (ls.moe.intermediate_size % world or ls.moe.shared_width % world):
                raise InvalidInput(f"layer {i}: expert widths not divisible by tensor parallel size {world}")
            hkv, kv_lo = self.kv_layout(ls.num_kv_heads, rank, world)
            dv = self._round(ls.v_head_dim)
            gate = {"": 0, "head": _round8(ls.num_heads), "element": ls.num_heads * dv}[ls.out_gate]
            kh = KernelHeads(ls.num_heads * ls.maps // world, hkv, kv_lo, self._round(ls.head_dim) * ls.maps, dv, ls.kv_from is None,
                             maps=ls.maps, gate_rows=gate)
            if ls.beside is not None:
                kh = dataclasses.replace(kh, delta=self._delta_heads(ls.beside, kh.qkv_rows, kh.hq * kh.dv))
            self.heads.append(kh)
        # uniform specs: one layout for all layers
        self.hq = self.heads[0].hq if self.heads else spec.num_heads // world
        self.hkv, self.kv_lo = (self.heads[0].hkv, self.heads[0].kv_lo) if self.heads else \
            self.kv_layout(spec.num_kv_heads, rank, world)

    @staticmethod
    def _delta_heads(ls, row0: int, col0: int) -> "DeltaHeads":
        if (ls.decay == "channel") != ls.low_rank_gate:
            raise UnsupportedOperation("delta rule: decays per channel go with a low-rank gate")
        ranks = (_round8(ls.decay_rank or 64), _round8(ls.gate_rank or 64)) if ls.low_rank_gate else (0, 0)
        return DeltaHeads(ls.num_heads, ls.num_kv_heads, _round8(ls.head_dim), _round8(ls.v_head_dim), ls.conv_taps, row0, col0, *ranks)

    def kv_bytes_per_token(self) -> int:
        """Cache bytes that one token takes on this rank over all layers that own keys and values."""
        e = torch.empty(0, dtype=self.dtype).element_size()
        return e * sum(k.cache_row for k in self.heads)

    def expandable(self, i: int) -> bool:
        """Layer ``i`` is latent attention of sizes that the tensor-core prompt kernel takes."""
        kh = self.heads[i]
        return self.spec.layer(i).mixer == "latent" and K.expanded_supported(kh.dim, kh.rot, kh.vdim)

    def state_bytes_per_seq(self) -> int:
        """Bytes of carried state of one live sequence (both halves of its slot)."""
        return 8 * sum(math.prod(shape) for _, shape in self.state_shapes())

    def state_shapes(self):
        """((layer, name), shape per state row) of everything that sequences carry from step to step, all fp32."""
        s, out = self.spec, []
        for i in range(s.num_layers):
            ls, kh = s.layer(i), self.heads[i]
            if s.input_conv:
                out += [((i, n), (s.input_conv - 1, self.width)) for n in (("conv1", "conv2") if ls.mlp is not None else ("conv1",))]
            if ls.mixer == "wkv" or s.token_shift:
                out.append(((i, "shift"), (self.width,)))
            if ls.mixer == "wkv":
                out.append(((i, "wkv"), (kh.hq, kh.dk, kh.dv)))
            d = kh.delta
            if d is not None:
                out += [((i, "delta_conv"), (d.taps - 1, d.conv_rows)), ((i, "delta"), (d.hq, d.dk, d.dv))]
        return out

    @staticmethod
    def kv_layout(num_kv_heads: int, rank: int, world: int) -> Tuple[int, int]:
        """(KV heads held by ``rank``, index of the first one).  When the ranks divide the KV heads every rank holds
        its share; when there are more ranks than KV heads (``world`` a multiple of them) every KV head is replicated
        on ``world / num_kv_heads`` consecutive ranks, whose query heads are exactly that head's group -- the
        reference expands grouped heads by copying them (``crates/runtime/src/models_v2/llama.rs:1073-1087``)."""
        if num_kv_heads % world == 0:
            n = num_kv_heads // world
            return n, rank * n
        if world % num_kv_heads == 0:
            return 1, rank // (world // num_kv_heads)
        raise UnsupportedOperation(f"{num_kv_heads} KV heads cannot be divided over or replicated on {world} ranks")

    def _set_ep(self, expert_parallel: bool) -> None:
        """Expert parallelism applies when asked for, with more than one rank and an expert count the ranks divide."""
        m = self.spec.moe
        self.ep = bool(expert_parallel and self.world > 1 and m is not None and m.num_experts % self.world == 0)
        self.experts_local = m.num_experts // self.world if self.ep else (m.num_experts if m is not None else 0)
        self.expert_lo = self.rank * self.experts_local if self.ep else 0

    @staticmethod
    def random(spec: DecoderSpec, device, rank: int = 0, world: int = 1, seed: int = 0,
               expert_parallel: bool = False) -> "RunnerWeights":
        """Random-init weights generated directly on the device, shard by shard (no host copy): the
        benchmark path for 8B-70B architectures.  Every rank draws the same full-size tensor for a given
        name from a per-tensor seed and keeps its shard, so TP=1 and TP=N hold the same model."""
        self = RunnerWeights.__new__(RunnerWeights)
        s = spec
        self._init_layout(spec, rank, world, expert_parallel)
        self.t = {}
        H, I = s.hidden_size, s.intermediate_size
        std = s.initializer_range
        counter = [0]

        def rnd(rows, cols, row0=0, nrows=None, col0=0, ncols=None):
            """Rows [row0, row0+nrows) x cols [col0, col0+ncols) of a virtual [rows, cols] N(0, std) matrix."""
            counter[0] += 1
            nrows = rows if nrows is None else nrows
            ncols = cols if ncols is None else ncols
            g = torch.Generator(device=device).manual_seed(seed * 1000003 + counter[0])
            # generate in row blocks so that a shard equals the same rows of the full matrix
            out = torch.empty(nrows, ncols, dtype=torch.bfloat16, device=device)
            blk = 1024
            for r in range(0, rows, blk):
                rr = min(blk, rows - r)
                lo, hi = max(r, row0), min(r + rr, row0 + nrows)
                g.manual_seed((seed * 1000003 + counter[0]) * 65537 + r)
                if lo >= hi:
                    continue
                full = torch.randn(rr, cols, generator=g, device=device, dtype=torch.float32) * std
                out[lo - row0:hi - row0] = full[lo - r:hi - r, col0:col0 + ncols].to(torch.bfloat16)
            return out

        ones = lambda n: torch.ones(n, dtype=torch.bfloat16, device=device)
        self.t["embed"] = rnd(s.vocab_size, H)
        self.t["final_norm.w"] = ones(H)
        vs = self.vocab_shard
        if s.tie_embeddings:
            self.t["lm_head"] = self.t["embed"][rank * vs:(rank + 1) * vs] if world > 1 else self.t["embed"]
        else:
            self.t["lm_head"] = rnd(s.vocab_size, H, rank * vs, vs)
        if s.layers is not None:
            self._random_layers(rnd, ones)
            return self
        qs, ks = s.q_size // world, self.hkv * s.head_dim
        k0 = self.kv_lo * s.head_dim
        for i in range(s.num_layers):
            L = f"layers.{i}."
            self.t[L + "ln1.w"], self.t[L + "ln2.w"] = ones(H), ones(H)
            q = rnd(s.q_size, H, rank * qs, qs)
            k = rnd(s.kv_size, H, k0, ks)
            v = rnd(s.kv_size, H, k0, ks)
            self.t[L + "wqkv"] = torch.cat([q, k, v], 0)
            self.t[L + "wo"] = rnd(H, s.q_size, 0, H, rank * qs, qs)
            if s.layer_is_moe(i):
                m = s.moe
                self.t[L + "router"] = rnd(m.num_experts, H)
                self._router_full(L, m)
                # tensor parallel inside every expert, or (expert parallel) whole experts of this rank
                Ie = m.intermediate_size if self.ep else m.intermediate_size // world
                c0 = 0 if self.ep else rank * Ie
                gu = torch.empty(self.experts_local, 2 * Ie, H, dtype=torch.bfloat16, device=device)
                dn = torch.empty(self.experts_local, H, Ie, dtype=torch.bfloat16, device=device)
                for e in range(m.num_experts):
                    mine = self.expert_lo <= e < self.expert_lo + self.experts_local
                    if not mine:
                        counter[0] += 3           # keep the per-tensor seeds aligned across ranks
                        continue
                    j = e - self.expert_lo
                    gu[j, :Ie] = rnd(m.intermediate_size, H, c0, Ie)
                    gu[j, Ie:] = rnd(m.intermediate_size, H, c0, Ie)
                    dn[j] = rnd(H, m.intermediate_size, 0, H, c0, Ie)
                self.t[L + "experts_gate_up"], self.t[L + "experts_down"] = gu, dn
                if m.num_shared_experts:
                    Is = m.shared_width // world
                    r0 = rank * Is
                    self.t[L + "shared_gate_up"] = torch.cat([rnd(m.shared_width, H, r0, Is) for _ in range(2 if m.gated else 1)], 0)
                    self.t[L + "shared_down"] = rnd(H, m.shared_width, 0, H, r0, Is)
            else:
                Is = I // world
                g = rnd(I, H, rank * Is, Is)
                u = rnd(I, H, rank * Is, Is)
                self.t[L + "w_gate_up"] = torch.cat([g, u], 0)
                self.t[L + "w_down"] = rnd(H, I, 0, H, rank * Is, Is)
        return self

    def _random_layers(self, rnd, ones) -> None:
        """Random weights of a per-layer spec on one rank, in kernel layout."""
        s, H = self.spec, self.width
        if self.world != 1 or H != s.hidden_size:
            raise UnsupportedOperation("random per-layer weights: one rank, width a multiple of 8")
        zeros = lambda n: torch.zeros_like(ones(n))
        if s.norm_bias:
            self.t["final_norm.b"] = zeros(H)
        if s.norm == "tanh":
            self.slopes = {n: 0.5 for n in ("final_norm", *(f"layers.{i}.{k}" for i in range(s.num_layers) for k in ("ln1", "ln2")))}
        for i, (kh, ls) in enumerate(zip(self.heads, s.layers)):
            L = f"layers.{i}."
            norm_w = zeros if s.norm_weight_offset_one else ones
            if s.token_shift:
                self.t[L + "shift"] = zeros(H) + 0.3
            if s.depth_average:
                self.t[L + "dwa"] = torch.cat([rnd(1, i + 1).view(-1), ones(1)]).float()
            if ls.maps > 1:
                self.lams[i] = ls.diff
            for n in ("ln1", "ln2") if s.norm_placement != "both" else ("ln1", "ln2", "ln1b", "ln2b"):
                self.t[L + n + ".w"] = norm_w(H)
                if s.norm_bias:
                    self.t[L + n + ".b"] = zeros(H)
            if s.input_conv:
                for n in ("conv1", "conv2"):
                    self.t[L + n] = rnd(s.input_conv, H)
            if ls.mlp == "dense":
                width = self._round(s.layer_intermediate(i))
                self.t[L + "w_up"], self.t[L + "w_down"] = rnd(width, H), rnd(H, width)
                if s.mlp_bias:
                    self.t[L + "b_up"], self.t[L + "b_down"] = zeros(width), zeros(H)
                if s.mlp == "gated":
                    self.t[L + "w_gate_up"] = torch.cat([self.t.pop(L + "w_up"), rnd(width, H)])
                if s.act == "xielu":
                    self.act_params[i] = (0.8, 1.3)
            d = kh.delta
            if d is not None:
                self.t[L + "delta_conv"] = rnd(d.taps, d.conv_rows) + 0.3
                self.t[L + "a_log"], self.t[L + "dt_bias"] = zeros(d.hq).float(), zeros(d.hq * (d.dk if d.ra else 1)).float() - 3.0
                self.t[L + "o_norm"] = ones(d.dv).float()
                if d.ra:
                    self.t[L + "w_a2"], self.t[L + "w_g2"] = rnd(d.hq * d.dk, d.ra), rnd(d.hq * d.dv, d.rg)
            if ls.mixer == "wkv":
                rank, C = self._round(ls.decay_rank or 64), kh.hq * kh.dk
                self.t[L + "mu"] = torch.full_like(rnd(5, H), 0.5)
                self.t[L + "w_rkvg"] = torch.stack([rnd(C, H) for _ in range(4)])
                self.t[L + "w_d1"], self.t[L + "w_d2"], self.t[L + "d0"] = rnd(rank, H), rnd(C, rank), zeros(C) - 2.0
                self.t[L + "u"], self.t[L + "o_norm"] = rnd(kh.hq, kh.dk).float(), ones(C).float()
                self.t[L + "wo"] = rnd(H, C)
                continue
            if ls.mixer == "latent":
                self.t[L + "w_dqkv"] = rnd(kh.q_rank + kh.dk, H)
                self.t[L + "q_a_norm"], self.t[L + "kv_a_norm"] = ones(kh.q_rank), ones(kh.dv)
                self.t[L + "w_uq"] = rnd(kh.hq * (kh.dim + kh.rot), kh.q_rank)
                self.t[L + "w_uk_t"] = rnd(kh.hq * kh.dv, kh.dim).view(kh.hq, kh.dv, kh.dim)
                self.t[L + "w_uv"] = rnd(kh.hq * kh.vdim, kh.dv).view(kh.hq, kh.vdim, kh.dv)
                if self.expandable(i):
                    self.t[L + "w_ukv"] = torch.cat([self.t[L + "w_uk_t"].transpose(1, 2), self.t[L + "w_uv"]], 1).flatten(0, 1).contiguous()
                self.t[L + "sink"], self.t[L + "wo"] = zeros(kh.hq).float(), rnd(H, kh.hq * kh.vdim)
                continue
            kind = s.qk_norm_kind(i)
            if ls.mixer == "delta":
                self.t[L + "w_in"], self.t[L + "wo"] = rnd(d.rows, H), rnd(H, d.cols)
            elif d is not None:
                self.t[L + "w_in"], self.t[L + "wo"] = rnd(kh.qkv_rows + d.rows, H), rnd(H, kh.hq * kh.dv + d.cols)
                if s.has_qkv_bias(i):
                    self.t[L + "b_in"] = zeros(kh.qkv_rows + d.rows)
            else:
                self.t[L + "wqkv"] = rnd(kh.qkv_rows + kh.gate_rows, H)
                self.t[L + "wo"] = rnd(H, kh.hq // kh.maps * kh.dv)
                if s.has_qkv_bias(i):
                    self.t[L + "bqkv"] = zeros(kh.qkv_rows + kh.gate_rows)
            if kind and ls.mixer == "attention":
                self.t[L + "q_norm"] = ones(kh.dk * (kh.hq if kind == "row" else 1))
                if kh.own_kv:
                    self.t[L + "k_norm"] = ones(kh.dk * (kh.hkv if kind == "row" else 1))
            if ls.sink or ls.fixed_sink is not None:
                self.t[L + "sink"] = zeros(kh.hq).float() + (ls.fixed_sink or 0.0)
            m = ls.moe
            if m is None:
                continue
            up = (2 if m.gated else 1) * self._round(m.intermediate_size)
            self.t[L + "router"] = rnd(m.num_experts, H)
            if m.router_bias:
                self.t[L + "router_b"] = zeros(m.num_experts)
            if m.correction:
                self.t[L + "correction"] = zeros(m.num_experts)
            if m.shared_gate:
                self.t[L + "shared_sg"] = rnd(1, H).view(-1)
            self._router_full(L, m)
            self.t[L + "experts_gate_up"] = torch.stack([rnd(up, H) for _ in range(m.num_experts)])
            self.t[L + "experts_down"] = torch.stack([rnd(H, self._round(m.intermediate_size)) for _ in range(m.num_experts)])
            if m.num_shared_experts:
                self.t[L + "shared_gate_up"] = rnd((2 if m.gated else 1) * self._round(m.shared_width), H)
                self.t[L + "shared_down"] = rnd(H, self._round(m.shared_width))

    def quantize(self, qtype="q4_k") -> "RunnerWeights":
        """Re-encodes every projection matrix (QKV, attention output, MLP, ``lm_head``; not embeddings, norms, routers
        or expert stacks) as ggml blocks of ``qtype`` on the device and drops the bf16 copy.  Decode-sized GEMMs
        (<= 8 token rows) then stream the blocks through the quantised GEMV kernel; larger ones expand the matrix into
        a scratch buffer first and run the tensor-core GEMM.  Rows are quantised independently along K, so sharded
        and fused matrices quantise like their parts.  Returns self."""
        from ..weights.gguf import BLOCK, quantize_blocks

        qt = QUANT_NAMES[qtype] if isinstance(qtype, str) else int(qtype)
        be = BLOCK[qt][0]
        tied = self.t.get("lm_head") is self.t.get("embed")
        for name, w in list(self.t.items()):
            leaf = name.rsplit(".", 1)[-1]
            if leaf not in ("wqkv", "wo", "w_gate_up", "w_up", "w_down", "lm_head") or isinstance(w, QWeight):
                continue
            if w.dim() != 2 or w.shape[1] % be or w.shape[1] % 8:
                continue                     # K is not a whole number of blocks: this matrix stays bf16
            if name == "lm_head" and tied:
                w = w.clone()                # the embedding keeps its bf16 table
            raw = quantize_blocks(w.float().cpu(), qt)
            self.t[name] = QWeight(torch.from_numpy(raw.copy()).to(w.device), qt, w.shape)
        self.quantized = qtype if isinstance(qtype, str) else str(qt)
        return self

    def dequantized_copy(self) -> "RunnerWeights":
        """The same weights with every quantised matrix expanded to bf16 (the values the quantised kernels compute
        with): the reference run for accuracy checks of the quantised path."""
        import copy

        from ..ops.quant import dequantize_cuda

        o = copy.copy(self)
        o.t = {k: (dequantize_cuda(v.blocks, v.qtype, v.shape) if isinstance(v, QWeight) else v) for k, v in self.t.items()}
        o.quantized = None
        return o

    def nbytes(self) -> int:
        seen, n = set(), 0
        for t in self.t.values():
            if isinstance(t, QWeight):
                n += t.nbytes()
                continue
            if t.data_ptr() not in seen:
                seen.add(t.data_ptr())
                n += t.numel() * t.element_size()
        return n


class TpContext:
    """Tensor-parallel plumbing of one rank: NCCL group for the baseline path, and (when fused) the
    symmetric buffers + counters that the fused kernels use.  ``world == 1`` needs none of it."""

    def __init__(self, rank: int = 0, world: int = 1, group=None, fused: bool = False):
        self.rank, self.world, self.group, self.fused = rank, world, group, fused and world > 1
        self.comm = None   # unillm_b200.dist.fused.FusedComm when fused

    def all_reduce(self, t: torch.Tensor) -> torch.Tensor:
        if self.world > 1:
            if self.comm is not None and self.comm.can_all_reduce(t):
                return self.comm.all_reduce(t)        # decode-sized message: one-shot exchange over peer memory
            import torch.distributed as dist

            dist.all_reduce(t, group=self.group)
        return t

    def all_gather_cat(self, t: torch.Tensor, dim: int = -1) -> torch.Tensor:
        if self.world == 1:
            return t
        import torch.distributed as dist

        outs = [torch.empty_like(t) for _ in range(self.world)]
        dist.all_gather(outs, t.contiguous(), group=self.group)
        return torch.cat(outs, dim=dim)


class StepPacker:
    """Packs a ``StepBatch`` into one int32 staging buffer (host-only logic, numpy views)."""

    def __init__(self, buf: torch.Tensor, max_blocks_per_seq: int, kv_pages: bool = False):
        self.meta_host = buf
        self.np = buf.numpy()
        self.META_INTS = buf.numel()
        self.max_blocks_per_seq = max_blocks_per_seq
        self.kv_pages = kv_pages

    @staticmethod
    def _bucket(n: int) -> int:
        b = 1
        while b < n:
            b <<= 1
        return b

    def pack(self, b: StepBatch, bucketed: bool = False, token_src: Optional[List[int]] = None):
        """Writes the step's integer metadata into the pinned buffer and returns the layout
        (name -> (offset, length)); one H2D copy moves all of it.

        With ``bucketed`` the batch is padded to a shape from a small set so that a captured CUDA graph
        can be replayed: decode rows to a power of two, prefill tokens to a multiple of 128 (the padding
        forms a dummy sequence that writes no KV), prefill sequences to a power of two (empty dummies),
        and every decode row plus the last row of every prefill sequence is sampled."""
        D = b.num_decode
        nseq = len(b.seq_lens)
        P = nseq - D
        mb = self.max_blocks_per_seq
        q_lens = list(b.prefill_q_lens)
        p_lens = list(b.seq_lens[D:])
        Tp = sum(q_lens)
        Dp, Pp, tpad = D, P, 0
        if bucketed:
            Dp = self._bucket(D) if D else 0
            if P:
                tpad = (-Tp) % 128
                Pp = self._bucket(P + (1 if tpad else 0))
                if tpad:
                    q_lens.append(tpad)
                    p_lens.append(tpad)
                q_lens += [0] * (Pp - len(q_lens))
                p_lens += [0] * (Pp - len(p_lens))
        pad = Dp - D
        h = self.np
        off = 0
        lay = {}

        def put(name, vals):
            nonlocal off
            n = len(vals)
            if off + n > self.META_INTS:
                raise InvalidInput("step metadata exceeds the staging buffer")
            if n:
                h[off:off + n] = vals
            lay[name] = (off, n)
            off += (n + 3) // 4 * 4     # keep every array 16-byte aligned

        # decode rows first (padded rows point at slot -1 / block 0 / length 1 so kernels stay in bounds)
        put("token_ids", b.token_ids[:D] + [0] * pad + b.token_ids[D:] + [0] * tpad)
        put("positions", b.positions[:D] + [0] * pad + b.positions[D:] + [0] * tpad)
        put("slot_mapping", b.slot_mapping[:D] + [-1] * pad + b.slot_mapping[D:] + [-1] * tpad)
        put("seq_lens_d", b.seq_lens[:D] + [1] * pad)
        if token_src is not None:
            # device index of each decode row's input token inside the previous step's sampled ids (-1 = uploaded)
            put("token_src", list(token_src[:D]) + [-1] * pad)
        nbt = (Dp + Pp) * mb
        if off + nbt > self.META_INTS:
            raise InvalidInput("step metadata exceeds the staging buffer")
        bt = h[off:off + nbt].reshape(Dp + Pp, mb)
        # only the entries below each sequence's length are ever read; rows of padded sequences are zeroed
        for i, row in enumerate(b.block_tables):
            bt[i if i < D else i + pad, :len(row)] = row
        if pad:
            bt[D:Dp, 0] = 0
        if Pp > P:
            bt[Dp + P:, :(128 // 16) + 1] = 0      # the dummy sequence is shorter than 128 tokens
        lay["block_tables"] = (off, nbt)
        off += (nbt + 3) // 4 * 4
        put("seq_lens_p", p_lens)
        qs = [0]
        for ql in q_lens:
            qs.append(qs[-1] + ql)
        put("q_start", qs)
        if self.kv_pages and Pp:
            # expanded prompts: where every sequence's rows start, in pages of 16, and a row count from a small set
            pages, pairs = [0], 0
            for n, q in zip(p_lens, q_lens):
                pages.append(pages[-1] + (n + 15) // 16)
                pairs += q * n - q * (q - 1) // 2
            put("kv_pages", pages)
            step = max(128, self._bucket(pages[-1] * 16) // 8)
            lay["_kv_rows"], lay["_kv_pairs"] = -(-pages[-1] * 16 // step) * step, pairs
        if b.state_in is not None:
            for name, v in (("state_in", b.state_in), ("state_out", b.state_out)):
                put(name, list(v[:D]) + [-1] * pad + list(v[D:]) + [-1] * (Pp - P))
        if bucketed:
            rows = list(range(Dp)) + [Dp + max(qs[j + 1] - 1, 0) for j in range(Pp)]
            sel = []
            for r in b.sample_rows:
                if r < D:
                    sel.append(r)
                else:
                    # r is the last row of some prefill sequence j: find it from the unpadded prefix sums
                    j = next(jj for jj in range(P) if D + qs[jj + 1] - 1 == r)
                    sel.append(Dp + j)
            lay["_sel"] = sel
        else:
            rows = [r if r < D else r + pad for r in b.sample_rows]
            lay["_sel"] = list(range(len(rows)))
        put("sample_rows", rows)
        lay["_T"], lay["_D"], lay["_Dp"], lay["_P"], lay["_S"] = Dp + Tp + tpad, D, Dp, Pp, len(rows)
        mq = max(q_lens) if q_lens else 0
        lay["_max_q"] = self._bucket(mq) if (bucketed and mq) else mq
        lay["_used"] = off
        return lay



class _OpTimer:
    def __init__(self, runner, name):
        self.r, self.name = runner, name

    def __enter__(self):
        if self.r.profile and not self.r._graph_mode:
            self.a = torch.cuda.Event(enable_timing=True)
            self.a.record()
        else:
            self.a = None

    def __exit__(self, *exc):
        if self.a is not None:
            b = torch.cuda.Event(enable_timing=True)
            b.record()
            self.r._prof_events.append((self.name, self.a, b))
        return False


class GpuModelRunner:
    META_INTS = 1 << 20   # capacity of the packed per-step metadata buffer (int32 words)

    def __init__(self, spec: DecoderSpec, weights: RunnerWeights, *, num_blocks: int, block_size: int = 16,
                 max_num_seqs: int = 256, max_num_batched_tokens: int = 8192, max_model_len: int = 8192,
                 tp: Optional[TpContext] = None, device=None, use_cuda_graphs: bool = True):
        if spec.norm not in ("rms", "layer", "tanh") or spec.post_ln or spec.embed_proj_dim:
            raise UnsupportedOperation("this spec is served by the generic model path, not the fused runner")
        tanh = spec.norm == "tanh"
        if tanh and (spec.norm_placement != "input" or not spec.residual_fp32 or not spec.norm_bias or not spec.final_norm or spec.pos == "learned"
                     or spec.embed_norm or spec.embed_scale != 1.0 or spec.parallel_residual or spec.input_conv
                     or any(spec.layer(i).mixer == "wkv" or spec.layer(i).mlp == "moe" for i in range(spec.num_layers))):
            raise UnsupportedOperation("Dynamic Tanh: in front of the sublayers of a 32-bit residual stream, no mixtures, wkv layers or convolutions")
        if not tanh and (spec.token_shift or spec.depth_average):
            raise UnsupportedOperation("token shifts and depth averages: behind Dynamic Tanh norms")
        if any(spec.layer(i).maps > 1 and (spec.layer(i).rotary_dim or spec.qk_norm_kind(i) or spec.layer(i).maps != 2) for i in range(spec.num_layers)):
            raise UnsupportedOperation("differential attention: two maps, no rotation, no query and key norms")
        if any(spec.layer(i).beside is not None and (spec.layer(i).out_gate or spec.layer(i).maps > 1 or spec.layer(i).value_rope or
                                                     spec.layer(i).beside.low_rank_gate) for i in range(spec.num_layers)):
            raise UnsupportedOperation("two mixers side by side: plain attention and a delta rule with one decay per head")
        if spec.norm_placement == "output" and (not spec.residual_fp32 or spec.pos == "learned" or spec.embed_norm
                                                or spec.residual_scale != 1.0 or spec.parallel_residual):
            raise UnsupportedOperation("norms on sublayer outputs: 32-bit residual stream, no learned positions")
        if spec.norm_placement == "both" and (not spec.residual_fp32 or spec.norm != "rms" or spec.norm_bias or spec.pos == "learned"
                                              or spec.embed_norm or spec.residual_scale != 1.0 or spec.parallel_residual
                                              or spec.mlp_bias or spec.o_bias
                                              or (spec.input_conv and any(spec.layer_is_moe(i) for i in range(spec.num_layers)))):
            raise UnsupportedOperation("norms on both sides of a sublayer: RMS, 32-bit residual stream, no mixtures behind convolutions")
        if spec.norm_placement != "both" and not tanh and (spec.input_conv or any(spec.layer(i).mixer != "attention" or spec.layer(i).beside is not None
                                                                     for i in range(spec.num_layers))):
            raise UnsupportedOperation("input convolutions, latent attention, wkv and delta layers: with norms on both sides of a sublayer")
        if spec.norm_placement == "input" and not tanh and (spec.residual_fp32 or weights.dtype != torch.bfloat16):
            raise UnsupportedOperation("a 32-bit residual stream or 32-bit weights: only with norms on sublayer outputs")
        self.spec, self.w = spec, weights
        self.tp = tp or TpContext()
        self.device = torch.device(device if device is not None else f"cuda:{torch.cuda.current_device()}")
        self.block_size, self.num_blocks = block_size, num_blocks
        self.max_num_seqs, self.max_tokens, self.max_model_len = max_num_seqs, max_num_batched_tokens, max_model_len
        self.max_blocks_per_seq = (max_model_len + block_size - 1) // block_size
        # NCCL collectives inside a captured graph stalled on this stack; the baseline path launches eagerly
        self.use_cuda_graphs = use_cuda_graphs and (self.tp.world == 1 or self.tp.fused)
        s, dev = spec, self.device
        self.layers = [s.layer(i) for i in range(s.num_layers)]
        # a window that no sequence can outgrow is full attention (and keeps the kernels for that)
        self.windows = [ls.window if 0 < ls.window < max_model_len else 0 for ls in self.layers]
        self.chunks = [ls.chunk if 0 < ls.chunk < max_model_len else 0 for ls in self.layers]
        self.k_cache: List[torch.Tensor] = []
        self.v_cache: List[torch.Tensor] = []
        for ls, kh in zip(self.layers, weights.heads):
            if ls.kv_from is not None:                   # attends to that layer's pages
                self.k_cache.append(self.k_cache[ls.kv_from])
                self.v_cache.append(self.v_cache[ls.kv_from])
                continue
            if not kh.own_kv:                            # no keys at all
                self.k_cache.append(None), self.v_cache.append(None)
                continue
            for cache, d in ((self.k_cache, kh.dk), (self.v_cache, 0 if ls.mixer == "latent" else kh.dv)):
                cache.append(torch.zeros(num_blocks, kh.hkv, block_size, d, dtype=weights.dtype, device=dev))
        # carried state: two rows per live sequence (a step reads one and writes the other)
        self.state: Dict[tuple, torch.Tensor] = {key: torch.zeros(2 * max_num_seqs, *shape, dtype=torch.float32, device=dev)
                                                 for key, shape in weights.state_shapes()}
        self._inv_freq: Dict[tuple, torch.Tensor] = {}   # rotation tables of per-layer specs
        self.alibi = None
        if s.pos == "alibi":
            sl = alibi_slopes(s.num_heads)
            self.alibi = sl[weights.rank * weights.hq:(weights.rank + 1) * weights.hq].to(dev)
        # packed metadata: pinned host staging + device mirror with fixed addresses (graph friendly)
        # two staging buffers: the next step may be packed while the copy of the previous one is still queued
        self.meta_hosts = [torch.zeros(self.META_INTS, dtype=torch.int32, pin_memory=True) for _ in range(2)]
        latent = any(ls.mixer == "latent" for ls in self.layers)
        self.packers = [StepPacker(h, self.max_blocks_per_seq, kv_pages=latent) for h in self.meta_hosts]
        self._flip = 0
        self.meta_dev = torch.empty(self.META_INTS, dtype=torch.int32, device=dev)
        self.fmeta_hosts = [torch.empty(4 * max_num_seqs, dtype=torch.float32, pin_memory=True) for _ in range(2)]
        self.fmeta_dev = torch.empty(4 * max_num_seqs, dtype=torch.float32, device=dev)
        self.out_ids_dev = torch.zeros(4 * max_num_seqs, dtype=torch.int32, device=dev)
        self.out_ids_hosts = [torch.zeros(4 * max_num_seqs, dtype=torch.int32, pin_memory=True) for _ in range(2)]
        # the per-device error word travels back with every step's sampled ids (same stream, no extra synchronisation)
        self.err_hosts = [torch.zeros(2, dtype=torch.int32, pin_memory=True) for _ in range(2)]
        self._out_events = [torch.cuda.Event(), torch.cuda.Event()]
        self._sel: List[int] = []
        self._handle = None
        self.attn_scratch = torch.empty(max_num_seqs * 16 * max((k.hq * (k.dv + 2) for k in weights.heads), default=0),
                                        dtype=torch.float32, device=dev)
        self.prefix_scratch = None     # workspace of the key-split shared-prefix pass, allocated on first use
        self._deq_scratch = None       # bf16 expansion of one quantised matrix at a time (quantised weights, > 8 rows)
        if getattr(weights, "quantized", None):
            big = max((int(v.shape[0]) * int(v.shape[1]) for v in weights.t.values() if isinstance(v, QWeight)), default=0)
            self._deq_scratch = torch.empty(big, dtype=torch.bfloat16, device=dev) if big else None
        self.overlap_suffix = os.environ.get("UB_ATTN_OVERLAP", "1") != "0"
        self._side = None
        self.graphs: Dict[tuple, tuple] = {}
        self.profile = False
        self._prof_events = []
        self._graph_mode = False
        self.launches = 0          # kernels of this library launched so far (counted on the host)
        self.captures = 0          # CUDA-graph captures so far (each costs an eager run, a synchronize and the capture)
        self.capture_new_graphs = True   # False: a step shape without a graph runs as plain launches instead
        self.eager_steps = 0       # graphable steps that ran as plain launches for that reason
        self.wait_s = 0.0          # host time spent blocked in fetch() waiting for the device
        self.fused_steps = 0       # tensor-parallel steps that ran the fused (peer-memory) path / the NCCL path
        self.unfused_steps = 0
        self.h2d_bytes = 0
        self.d2h_bytes = 0
        self._layout = None
        self._last_fused = False

    # ------------------------------------------------------------------------------------------
    # metadata packing
    # ------------------------------------------------------------------------------------------
    def _pack(self, b: StepBatch, bucketed: bool = False):
        src = None
        if b.token_src is not None:
            prev = self._sel            # sample order -> index in out_ids_dev, of the step launched before this one
            src = [prev[k] if k >= 0 else -1 for k in b.token_src]
        self._flip ^= 1
        pk = self.packers[self._flip]
        lay = pk.pack(b, bucketed, token_src=src)
        lay["_host"] = pk.meta_host
        self._choose_expansion(lay)
        return lay

    def _feed_sampled_ids(self, lay) -> None:
        """Decode rows whose input token was sampled by the previous step take it from the device buffer of that
        step's samples (the host may not have read them yet).  Runs right after the upload and outside the captured
        graph: the step itself then only reads its own metadata and can be replayed (graph capture runs it more
        than once) without seeing the samples it has just written."""
        if "token_src" not in lay:
            return
        src = self._view(lay, "token_src")
        d = self._view(lay, "token_ids")[:src.numel()]
        prev = self.out_ids_dev.index_select(0, src.clamp(min=0))
        d.copy_(torch.where(src >= 0, prev, d))

    def _view(self, lay, name):
        o, n = lay[name]
        return self.meta_dev[o:o + n]

    def _upload(self, lay):
        n = lay["_used"]
        self.meta_dev[:n].copy_(lay["_host"][:n], non_blocking=True)
        self.h2d_bytes += n * 4
        self._feed_sampled_ids(lay)

    # ------------------------------------------------------------------------------------------
    # layer math
    # ------------------------------------------------------------------------------------------
    def _prof(self, name: str):
        """Context manager timing one op with CUDA events when profiling is on (eager mode only)."""
        return _OpTimer(self, name)

    def profile_report(self) -> Dict[str, float]:
        """Milliseconds per op name accumulated since profiling was switched on (synchronises)."""
        torch.cuda.synchronize()
        out: Dict[str, float] = {}
        for name, a, b in self._prof_events:
            out[name] = out.get(name, 0.0) + a.elapsed_time(b)
        self._prof_events = []
        return out

    def _norm(self, x, name, residual=None, want_h=False):
        s, t = self.spec, self.w.t
        self.launches += 1
        with self._prof("norm"):
            return self._norm_impl(x, name, residual, want_h)

    def _norm_impl(self, x, name, residual=None, want_h=False):
        s, t = self.spec, self.w.t
        return K.norm(x, t[name + ".w"], bias=t.get(name + ".b"), residual=residual, eps=s.norm_eps,
                      kind="rms" if s.norm == "rms" else "layer", weight_offset_one=s.norm_weight_offset_one,
                      want_residual_out=want_h)

    def _gemm(self, x, w, tag="gemm", **kw):
        self.launches += 1
        with self._prof(f"{tag}[{x.shape[0]}x{w.shape[0]}x{w.shape[1]}]"):
            if isinstance(w, QWeight):
                return self._qgemm(x, w, **kw)
            return K.gemm_tn(x, w, **kw)

    def _qgemm(self, x, w: "QWeight", **kw):
        """GEMM against a block-quantised matrix.  Up to 8 token rows: the quantised GEMV kernel (the weight stream is
        4.5 - 8.5 bits per value) followed by the small epilogue kernels; more rows, or a fused collective: the matrix
        is expanded into the runner's scratch buffer and the tensor-core GEMM runs on that."""
        from ..ops import quant as Q

        M = x.shape[0]
        N_, Kd = w.shape
        plain = kw.get("rs") is None and kw.get("ag") is None and kw.get("out") is None
        if M <= 8 and plain and x.is_contiguous():
            y = Q.qgemv_cuda(w.blocks, x, N_, w.qtype)
            self.launches += 1
            dual = kw.get("dual_rows", 0)
            scale = kw.get("out_scale", 1.0)
            if dual:
                y = K.act_mul(y, kw.get("act") or "silu")
            else:
                if kw.get("bias") is not None or scale != 1.0:
                    yf = y.float() * scale
                    if kw.get("bias") is not None:
                        yf = yf + kw["bias"].float()
                    y = yf.to(torch.bfloat16)
                if kw.get("act"):
                    y = K.eltwise(y, kw["act"])
            if kw.get("residual") is not None:
                y = K.add(y, kw["residual"])
            if kw.get("out_dtype", torch.bfloat16) == torch.float32:
                y = y.float()
            return y
        need = N_ * Kd
        if self._deq_scratch is None or self._deq_scratch.numel() < need:
            self._deq_scratch = torch.empty(need, dtype=torch.bfloat16, device=self.device)
        dense = self._deq_scratch[:need].view(N_, Kd)
        Q.dequantize_cuda_into(w.blocks, w.qtype, dense)
        self.launches += 1
        return K.gemm_tn(x, dense, **kw)

    def _rope_append(self, i, qkv, pos, slots):
        """Head norms and rotation of q and k in place, keys and values into the cache (of a layer that owns some)."""
        s, t, ls, kh = self.spec, self.w.t, self.layers[i], self.w.heads[i]
        L = f"layers.{i}."
        kw = dict(theta=ls.rope_theta, llama3_scaling=ls.rope_llama3)
        if s.layers is not None:
            # frequencies from the host in 64 bits, and only for the layers' own rotation
            kw = dict(v_head_dim=kh.dv, norm_dim=ls.head_dim, v_inv_freq=self._value_rotation(ls) if ls.value_rope and kh.own_kv else None)
            if ls.rotary_dim > 0:
                kw["inv_freq"], kw["gain"] = self._rotation(ls)
        own = kh.own_kv
        with self._prof("rope_kv_append"):
            K.rope_kv_append(qkv, pos, slots if own else None, self.k_cache[i] if own else None,
                             self.v_cache[i] if own else None, num_q_heads=kh.hq, num_kv_heads=kh.hkv if own else 0,
                             head_dim=kh.dk, rotary_dim=ls.rotary_dim, pos_scale=s.rope_pos_scale,
                             interleaved=s.rope_interleaved, q_norm_w=t.get(L + "q_norm"), k_norm_w=t.get(L + "k_norm"),
                             norm_eps=s.norm_eps, k_cache_only=own, row_norm=s.qk_norm_kind(i) == "row", **kw)
        self.launches += 1

    def _attention_layer(self, i, h, pos, slots, lay, shared_prefix_len):
        """Attention of layer ``i`` on what it reads, up to the rows for its output projection."""
        t, ls, kh, L = self.w.t, self.layers[i], self.w.heads[i], f"layers.{i}."
        proj = self._gemm(h, t[L + "wqkv"], bias=t.get(L + "bqkv"))
        qkv = proj[:, :kh.qkv_rows] if kh.gate_rows else proj
        if kh.maps > 1:
            own = kh.own_kv
            with self._prof("map_rows"):
                qkv = K.map_rows(qkv, slots if own else None, self.k_cache[i] if own else None, self.v_cache[i] if own else None,
                                 num_heads=kh.hq // kh.maps, maps=kh.maps, dim=kh.dk // kh.maps).flatten(1)
            self.launches += 1
        else:
            self._rope_append(i, qkv, pos, slots)
        a = self._attention(i, qkv, lay, shared_prefix_len)
        if kh.maps == 1 and not ls.out_gate and not ls.value_rope:
            return a
        self.launches += 1
        with self._prof("attn_finish"):
            return K.attn_finish(a, kh.dv, gate=proj[:, kh.qkv_rows:] if kh.gate_rows else None, gate_kind=ls.out_gate, maps=kh.maps,
                                 lam=self.w.lams.get(i, 0.0), factor=1.0 - ls.diff, eps=self.spec.norm_eps, dv_real=ls.v_head_dim,
                                 positions=pos if ls.value_rope else None, inv_freq=self._value_rotation(ls) if ls.value_rope else None)

    def _attention(self, i, qkv, lay, shared_prefix_len, out=None):
        """qkv [T, q | k | v] already rotated and appended -> attention output [T, hq * Dv] (``out``: columns of a wider tensor)."""
        kh, ls = self.w.heads[i], self.layers[i]
        D, hq, hkv, window, chunk = kh.dk, kh.hq, kh.hkv, self.windows[i], self.chunks[i]
        sinks = self.w.t.get(f"layers.{i}.sink")
        T, Dp, P = lay["_T"], lay["_Dp"], lay["_P"]
        q = qkv[:, :hq * D].unflatten(1, (hq, D))          # strided view: row stride of the fused projection
        flat = torch.empty(T, hq * kh.dv, dtype=qkv.dtype, device=qkv.device) if out is None else out
        out = flat.unflatten(1, (hq, kh.dv))
        kc, vc = self.k_cache[i], self.v_cache[i]
        bt = self._view(lay, "block_tables").view(Dp + P, self.max_blocks_per_seq)
        scale = ls.scale if ls.scale is not None else 1.0 / math.sqrt(ls.head_dim)
        # the shared-prefix pass has no window, chunk, position bias or sink
        plain = window == 0 and chunk == 0 and self.alibi is None and sinks is None and not ls.softcap and kh.dk == kh.dv and qkv.dtype == torch.bfloat16
        cascade = plain and shared_prefix_len >= 4 * self.block_size and Dp >= 8
        # prefill rows join the cascade when their chunks start after the shared prefix and share its blocks
        pp = cascade and P > 0 and lay.get("_pp", False)
        if cascade:
            # one GEMM-shaped pass of all queries over the shared prefix blocks, one pass per sequence over the
            # unique suffixes, then a merge of the two partials
            R = T if pp else Dp
            # the suffix kernels fold the prefix partial into their output themselves (head dim 128, page 16);
            # otherwise a separate merge kernel combines the two partials
            fused = D == 128 and self.block_size == 16
            lse_a = torch.empty(R, hq, dtype=torch.float32, device=qkv.device)
            oa = torch.empty(R, hq, D, dtype=torch.bfloat16, device=qkv.device)
            kvs = self._prefix_splits(i, R, shared_prefix_len)
            with self._prof("attn_shared_prefix"):
                K.attn_prefill(q[:R], kc, vc, bt[:1], self._prefix_len_dev(shared_prefix_len), self._q_start_all(R),
                               R, scale=scale, causal=False, window=0, alibi_slopes=None, out=oa, lse=lse_a,
                               return_lse=True, kv_splits=kvs, scratch=self.prefix_scratch if kvs > 1 else None)
            if kvs > 1:
                self.launches += 1
            if fused:
                # The suffix pass of the prefill chunks is a handful of CTAs whose time is all latency; it runs beside
                # the decode rows' suffix pass on a second stream (both only read the prefix partial).
                side = self._side_stream() if (pp and self.overlap_suffix) else None
                if side is not None:
                    cur = torch.cuda.current_stream()
                    side.wait_stream(cur)
                    with torch.cuda.stream(side):
                        with self._prof("attn_prefill_suffix"):
                            K.attn_prefill(q[Dp:], kc, vc, bt[Dp:], self._view(lay, "seq_lens_p"),
                                           self._view(lay, "q_start"), lay["_max_q"], scale=scale, causal=True,
                                           kv_start=shared_prefix_len, out=out[Dp:], merge=(oa[Dp:], lse_a[Dp:]))
                    self.launches += 1
                with self._prof("attn_decode_suffix"):
                    K.attn_decode(q[:Dp], kc, vc, bt[:Dp], self._view(lay, "seq_lens_d"), scale=scale,
                                  kv_start=shared_prefix_len, out=out[:Dp], splits=1, merge=(oa[:Dp], lse_a[:Dp]))
                if side is not None:
                    cur.wait_stream(side)
                elif pp:
                    with self._prof("attn_prefill_suffix"):
                        K.attn_prefill(q[Dp:], kc, vc, bt[Dp:], self._view(lay, "seq_lens_p"), self._view(lay, "q_start"),
                                       lay["_max_q"], scale=scale, causal=True, kv_start=shared_prefix_len, out=out[Dp:],
                                       merge=(oa[Dp:], lse_a[Dp:]))
                    self.launches += 1
                self.launches += 2
            else:
                lse_b = torch.empty(R, hq, dtype=torch.float32, device=qkv.device)
                ob = torch.empty(R, hq, D, dtype=torch.bfloat16, device=qkv.device)
                with self._prof("attn_decode_suffix"):
                    K.attn_decode(q[:Dp], kc, vc, bt[:Dp], self._view(lay, "seq_lens_d"), scale=scale,
                                  kv_start=shared_prefix_len, out=ob[:Dp], lse=lse_b[:Dp], return_lse=True, splits=1)
                if pp:
                    with self._prof("attn_prefill_suffix"):
                        K.attn_prefill(q[Dp:], kc, vc, bt[Dp:], self._view(lay, "seq_lens_p"), self._view(lay, "q_start"),
                                       lay["_max_q"], scale=scale, causal=True, kv_start=shared_prefix_len, out=ob[Dp:],
                                       lse=lse_b[Dp:], return_lse=True)
                    self.launches += 1
                with self._prof("attn_merge"):
                    K.attn_merge(oa, lse_a, ob, lse_b, out=out[:R])
                self.launches += 3
        elif Dp > 0:
            with self._prof("attn_decode"):
                K.attn_decode(q[:Dp], kc, vc, bt[:Dp], self._view(lay, "seq_lens_d"), scale=scale, window=window,
                              alibi_slopes=self.alibi, sinks=sinks, softcap=ls.softcap, chunk=chunk, out=out[:Dp], scratch=self.attn_scratch,
                              max_seq_len=self.max_model_len if self._graph_mode else int(self._max_len_d))
            self.launches += 1
        if P > 0 and not pp:
            with self._prof("attn_prefill"):
                K.attn_prefill(q[Dp:], kc, vc, bt[Dp:], self._view(lay, "seq_lens_p"), self._view(lay, "q_start"),
                               lay["_max_q"], scale=scale, causal=True, window=window, alibi_slopes=self.alibi,
                               sinks=sinks, softcap=ls.softcap, chunk=chunk, out=out[Dp:])
            self.launches += 1
        return flat

    def _side_stream(self):
        if self._side is None:
            self._side = torch.cuda.Stream(device=self.device)
        return self._side

    PREFIX_SPLIT_ROWS = 160 * 128     # (query row, head) pairs x splits the key-split workspace can hold

    def _prefix_splits(self, i: int, R: int, prefix_len: int) -> int:
        """Key splits of the shared-prefix pass.  The pass has one CTA per 128 packed (token, head-of-group) rows and KV
        head; a tensor-parallel rank with one KV head and a few hundred rows would keep a fraction of the SMs busy while
        every CTA walks the whole prefix, so the key tiles are divided until about one wave of CTAs exists."""
        w = self.w.heads[i]
        if w.dk != 128 or self.block_size != 16:
            return 1
        G = w.hq // w.hkv
        if 128 % G:
            return 1
        ctas = -(-R // (128 // G)) * w.hkv
        n = min(prefix_len // 128, 148 // max(ctas, 1), 8)
        while n > 1 and n * R * w.hq > self.PREFIX_SPLIT_ROWS:
            n -= 1
        if n > 1 and self.prefix_scratch is None:
            self.prefix_scratch = torch.empty(K.attn_prefill_split_scratch_floats(self.PREFIX_SPLIT_ROWS, 1, 128, 1),
                                              dtype=torch.float32, device=self.device)
        return max(n, 1)

    def _prefix_len_dev(self, n: int) -> torch.Tensor:
        c = getattr(self, "_plen_cache", None)
        if c is None:
            c = self._plen_cache = {}
        if n not in c:
            c[n] = torch.tensor([n], dtype=torch.int32, device=self.device)
        return c[n]

    def _q_start_all(self, n: int) -> torch.Tensor:
        c = getattr(self, "_qsa_cache", None)
        if c is None:
            c = self._qsa_cache = {}
        if n not in c:
            c[n] = torch.tensor([0, n], dtype=torch.int32, device=self.device)
        return c[n]

    def _mlp(self, i, h, residual):
        s, t = self.spec, self.w.t
        L = f"layers.{i}."
        tp = self.tp
        if s.layer_is_moe(i):
            from .moe_runner import moe_forward

            return moe_forward(self, i, h, residual)
        if s.mlp == "gated":
            I = t[L + "w_gate_up"].shape[0] // 2
            a = self._gemm(h, t[L + "w_gate_up"], dual_rows=I, act=s.act)
        else:
            a = self._gemm(h, t[L + "w_up"], bias=t.get(L + "b_up"), act=s.act)
        if tp.world == 1:
            return self._gemm(a, t[L + "w_down"], bias=t.get(L + "b_down"), residual=residual)
        y = self._gemm(a, t[L + "w_down"], bias=t.get(L + "b_down"))
        tp.all_reduce(y)
        self.launches += 1
        return K.add(y, residual)

    def _forward_tokens(self, lay, shared_prefix_len: int) -> torch.Tensor:
        """Runs all layers on the packed step; returns the sampled token ids tensor (device, [S])."""
        s, t, tp = self.spec, self.w.t, self.tp
        T = lay["_T"]
        self._final_norm_done = False
        if self._fused_ok(T):
            self._last_fused = True
            return self._forward_tokens_fused(lay, shared_prefix_len)
        self._last_fused = False
        if s.norm_placement == "output":
            return self._forward_tokens_output_norm(lay, shared_prefix_len)
        if s.norm_placement == "both":
            return self._forward_tokens_both_norms(lay, shared_prefix_len)
        if s.norm == "tanh":
            return self._forward_tokens_stream(lay, shared_prefix_len)
        ids = self._view(lay, "token_ids")
        pos = self._view(lay, "positions")
        slots = self._view(lay, "slot_mapping")
        x = K.embed_gather(ids, t["embed"], scale=s.embed_scale)
        self.launches += 1
        if s.pos == "learned":
            x = x + t["pos_embed"][(pos + s.learned_pos_offset).long()]
        if s.embed_norm:
            x = K.norm(x, t["embed_norm.w"], bias=t["embed_norm.b"], eps=s.norm_eps, kind="layer")
        rs = s.residual_scale
        for i in range(s.num_layers):
            L = f"layers.{i}."
            h = self._norm(x, L + "ln1")
            a = self._attention_layer(i, h, pos, slots, lay, shared_prefix_len)
            if s.parallel_residual:
                m_in = h if s.parallel_shared_norm else self._norm(x, L + "ln2")
                o = self._gemm(a, t[L + "wo"], bias=t.get(L + "bo"))
                m = self._mlp_noresid(i, m_in)
                y = K.add(o, m)
                if tp.world > 1:
                    tp.all_reduce(y)
                x = K.add(x, y, 1.0, rs)
                self.launches += 2
                continue
            if tp.world == 1 and rs == 1.0:
                x = self._gemm(a, t[L + "wo"], bias=t.get(L + "bo"), residual=x)
            else:
                o = self._gemm(a, t[L + "wo"], bias=t.get(L + "bo"))
                tp.all_reduce(o)
                x = K.add(x, o, 1.0, rs)
                self.launches += 1
            h2 = self._norm(x, L + "ln2")
            if rs == 1.0:
                x = self._mlp(i, h2, x)
            else:
                m = self._mlp_noresid(i, h2)
                if tp.world > 1:
                    tp.all_reduce(m)
                x = K.add(x, m, 1.0, rs)
                self.launches += 1
        return x

    def _forward_tokens_output_norm(self, lay, shared_prefix_len: int) -> torch.Tensor:
        """Layers of the form ``x += norm(f(x))`` around a 32-bit residual stream.  ``h`` is the stream in the element type
        of the matrix products; the norm of a sublayer's output, the residual add and the next ``h`` are one kernel, which
        for a mixture-of-experts also sums the chosen experts' rows and the shared expert's."""
        s, t, tp = self.spec, self.w.t, self.tp
        pos, slots = self._view(lay, "positions"), self._view(lay, "slot_mapping")
        x, h = K.embed_residual(self._view(lay, "token_ids"), t["embed"], scale=s.embed_scale)
        self.launches += 1
        for i, ls in enumerate(self.layers):
            L = f"layers.{i}."
            a = self._attention_layer(i, h, pos, slots, lay, shared_prefix_len)
            y = self._gemm(a, t[L + "wo"], bias=t.get(L + "bo"))
            tp.all_reduce(y)
            h = self._residual_norm(x, y, L + "ln1")
            if ls.mlp == "moe":
                from .moe_runner import moe_branch

                y, experts, routing = moe_branch(self, i, h, router_x=x)
                h = self._residual_norm(x, y, L + "ln2", experts=experts, routing=routing)
            elif ls.mlp == "dense":
                y = self._mlp_noresid(i, h)
                tp.all_reduce(y)
                h = self._residual_norm(x, y, L + "ln2")
        return x

    def _forward_tokens_both_norms(self, lay, shared_prefix_len: int) -> torch.Tensor:
        """Layers of the form ``x += norm_b(f(conv(norm(x))))`` around a 32-bit residual stream.  Adding a sublayer's normed
        output (for a mixture-of-experts also its weighted sum), the next norm, its convolution over time and (in front of a wkv
        mixer) the token-shift mixes are one kernel; what it needs from earlier steps is in the sequences' state rows.  The last
        sublayer's output is added by the final norm, for the rows that are asked for."""
        s, t = self.spec, self.w.t
        pos, slots = self._view(lay, "positions"), self._view(lay, "slot_mapping")
        parts = self._portions(lay)
        x, _ = K.embed_residual(self._view(lay, "token_ids"), t["embed"], scale=s.embed_scale)
        self.launches += 1
        y: dict = {}                                         # the sublayer output that has not been added yet
        for i, ls in enumerate(self.layers):
            L = f"layers.{i}."
            x, h = self._sublayer_in(i, 1, x, parts, y)
            scale = 1.0
            if ls.mixer == "wkv":
                a = self._wkv(i, h, parts)
            elif ls.mixer == "latent":
                a = self._latent_attention(i, h, pos, slots, lay)
            else:
                a, scale = self._attention_and_delta(i, h, pos, slots, lay, parts, shared_prefix_len)
            y = dict(y=self._gemm(a, t[L + "wo"], out_scale=scale), y_weight=t[L + "ln1b.w"])
            if ls.mlp is None:
                continue
            x, h = self._sublayer_in(i, 2, x, parts, y)
            y = dict(y_weight=t[L + "ln2b.w"])
            if ls.mlp == "moe":
                from .moe_runner import moe_branch

                y["y"], y["experts"], y["routing"] = moe_branch(self, i, h, router_x=h)
            elif s.mlp == "gated":
                w = t[L + "w_gate_up"]
                y["y"] = self._gemm(self._gemm(h, w, dual_rows=w.shape[0] // 2, act=s.act), t[L + "w_down"])
            else:
                up = self._gemm(h, t[L + "w_up"], act=s.act, act_params=self.w.act_params.get(i))
                y["y"] = self._gemm(up, t[L + "w_down"])
        self._last_y = y
        return x

    def _forward_tokens_stream(self, lay, shared_prefix_len: int) -> torch.Tensor:
        """Layers of the form ``x += m f(norm(x))`` with a norm that needs no statistics, around a 32-bit residual stream.  Adding a
        sublayer's output, the average over depth behind a layer, the next norm and the token shift are one kernel; the embedding
        rows are gathered by the first of them, the last layer's output is added and averaged by the final norm, for the rows that
        are asked for."""
        s, t, m = self.spec, self.w.t, self.spec.residual_scale
        pos, slots = self._view(lay, "positions"), self._view(lay, "slot_mapping")
        parts = self._portions(lay)
        buf = lambda: torch.empty(lay["_T"], self.w.width, dtype=torch.float32, device=self.device)
        # results of the layers so far, the embedding first
        streams = torch.empty(s.num_layers, lay["_T"], self.w.width, dtype=torch.float32, device=self.device) if s.depth_average else None
        y: dict = dict(ids=self._view(lay, "token_ids"), table=t["embed"])
        for i, ls in enumerate(self.layers):
            L = f"layers.{i}."
            if streams is not None:
                y["x_res"] = streams[i]
            x = streams[0] if i == 0 and streams is not None else buf()
            if i > 0 or streams is None:
                y["x_out"] = x
            h = self._stream_in(L + "ln1", parts, shift=t.get(L + "shift"), shift_state=self.state.get((i, "shift")), **y)
            if ls.mixer == "latent":
                a = self._latent_attention(i, h, pos, slots, lay)
            elif ls.mixer == "delta":
                a, _ = self._attention_and_delta(i, h, pos, slots, lay, parts, shared_prefix_len)
            else:
                a = self._attention_layer(i, h, pos, slots, lay, shared_prefix_len)
            y = dict(x=x, y=self._gemm(a, t[L + "wo"], bias=t.get(L + "bo")), scale=m)
            if ls.mlp is not None:
                x = buf() if i == 0 and streams is not None else x
                h = self._stream_in(L + "ln2", (), x_out=x, **y)
                y = dict(x=x, y=self._mlp_noresid(i, h), scale=m)
            if streams is not None:
                y.update(streams=streams, mix=t[L + "dwa"])
        self._last_y = y
        return y["x"]

    def _stream_in(self, name, parts, **kw):
        t = self.w.t
        self.launches += len(parts) if kw.get("shift") is not None else 1
        with self._prof("stream_in"):
            return K.stream_in(parts, t[name + ".w"], t[name + ".b"], self.w.slopes[name], **kw)

    def _attention_and_delta(self, i, h, pos, slots, lay, parts, shared_prefix_len):
        """Attention, a gated delta rule, or both side by side on one input projection: (rows for the output projection, the
        factor on its result)."""
        t, L, ls, kh = self.w.t, f"layers.{i}.", self.layers[i], self.w.heads[i]
        d = kh.delta
        if d is None:
            return self._attention_layer(i, h, pos, slots, lay, shared_prefix_len), 1.0
        proj = self._gemm(h, t[L + "w_in"], bias=t.get(L + "b_in"))
        out = torch.empty(h.shape[0], d.col0 + d.cols, dtype=proj.dtype, device=proj.device)
        mx = ls
        if ls.beside is not None:
            mx = ls.beside
            qkv = proj[:, :d.row0]
            self._rope_append(i, qkv, pos, slots)
            self._attention(i, qkv, lay, shared_prefix_len, out=out[:, :d.col0])
        low = {}
        if d.ra:
            mid = proj[:, d.row0 + d.low_col:]
            low = dict(decay=self._gemm(mid[:, :d.ra], t[L + "w_a2"], out_dtype=torch.float32), gate=self._gemm(mid[:, d.ra:d.ra + d.rg], t[L + "w_g2"]))
        with self._prof("delta"):
            K.delta_mixer(proj, d.row0, t[L + "delta_conv"], t[L + "a_log"], t[L + "dt_bias"], t[L + "o_norm"],
                          self.state[(i, "delta_conv")], self.state[(i, "delta")], parts, kv_heads=d.hk, eps=self.spec.norm_eps,
                          dk_real=mx.head_dim, dv_real=mx.v_head_dim, out=out[:, d.col0:], gate_act=mx.gate_act, **low)
        self.launches += sum(1 if p.q_start is None else 4 for p in parts)
        if ls.beside is None:
            return out, 1.0
        return out, ls.scales[0] or 1.0

    def _portions(self, lay) -> List["K.Portions"]:
        """The step's rows as portions of sequences: one-token rows of decoding sequences, then pieces of prompts."""
        T, Dp, P = lay["_T"], lay["_Dp"], lay["_P"]
        si = so = None
        if "state_in" in lay:
            si, so = self._view(lay, "state_in"), self._view(lay, "state_out")
        cut = lambda t, a, b: None if t is None else t[a:b]
        out = []
        if Dp:
            out.append(K.Portions(0, Dp, Dp, 1, None, cut(si, 0, Dp), cut(so, 0, Dp)))
        if P:
            out.append(K.Portions(Dp, T - Dp, P, lay["_max_q"], self._view(lay, "q_start"), cut(si, Dp, Dp + P), cut(so, Dp, Dp + P)))
        return out

    def _sublayer_in(self, i, which, x, parts, y: dict):
        """``y``: the previous sublayer's output and norm weight, as keyword arguments of ``cuda_ops.sublayer_in``."""
        s, t, L = self.spec, self.w.t, f"layers.{i}."
        conv = f"conv{which}"
        mix = which == 1 and self.layers[i].mixer == "wkv"
        self.launches += len(parts) if s.input_conv or mix else 1
        with self._prof("sublayer_in"):
            return K.sublayer_in(x, parts, t[f"{L}ln{which}.w"], eps=s.norm_eps, conv=t.get(L + conv), conv_state=self.state.get((i, conv)),
                                 mu=t[L + "mu"] if mix else None, shift_state=self.state[(i, "shift")] if mix else None,
                                 width=s.hidden_size, offset_one=s.norm_weight_offset_one, **y)

    def _wkv(self, i, h, parts):
        """``h`` [5, T, width]: the mixes for receptance, key, value, gate and decay."""
        t, L, kh = self.w.t, f"layers.{i}.", self.w.heads[i]
        with self._prof(f"gemm_rkvg[4x{h.shape[1]}x{kh.hq * kh.dk}x{h.shape[2]}]"):
            rkvg = K.gemm_stacked(h[:4], t[L + "w_rkvg"])
        low = self._gemm(h[4], t[L + "w_d1"], act="tanh")
        ww = self._gemm(low, t[L + "w_d2"], bias=t[L + "d0"], out_dtype=torch.float32)
        self.launches += 1 + len(parts)
        with self._prof("wkv"):
            return K.wkv_mixer(rkvg, ww, t[L + "u"], t[L + "o_norm"], self.state[(i, "wkv")], parts, eps=self.spec.norm_eps,
                               norm_dim=self.layers[i].head_dim)

    def _latent_attention(self, i, h, pos, slots, lay):
        """Latent attention with the key matrices on the query side and the value matrices on the output side, over the
        cached latents themselves."""
        s, t, ls, kh, L = self.spec, self.w.t, self.layers[i], self.w.heads[i], f"layers.{i}."
        T, Dp, P = lay["_T"], lay["_Dp"], lay["_P"]
        freq, gain = self._rotation(ls)
        down = self._gemm(h, t[L + "w_dqkv"])
        with self._prof("latent_rows"):
            cq = K.latent_rows(down, pos, slots, self.k_cache[i], t[L + "q_a_norm"], t[L + "kv_a_norm"], freq, eps=s.norm_eps,
                               gain=gain, q_real=ls.q_rank, kv_real=ls.kv_rank)
        q = self._gemm(cq, t[L + "w_uq"]).view(T, kh.hq, kh.dim + kh.rot)
        bt = self._view(lay, "block_tables").view(Dp + P, self.max_blocks_per_seq)
        out = torch.empty(T, kh.hq, kh.vdim, dtype=q.dtype, device=q.device)
        kw = dict(scale=ls.scale, sinks=t.get(L + "sink"))
        if P and lay["_xp"][i]:
            self._latent_expanded(i, q[Dp:], pos[Dp:], bt[Dp:], lay, out[Dp:], freq, gain, kw)
            if not Dp:
                return out.view(T, kh.hq * kh.vdim)
            q, pos, full, T, P = q[:Dp], pos[:Dp], out, Dp, 0
            out = full[:Dp]
        else:
            full = out
        qa = torch.empty(T, kh.hq, kh.dk, dtype=q.dtype, device=q.device)
        lat = torch.empty(T, kh.hq, kh.dv, dtype=q.dtype, device=q.device)
        with self._prof("latent_query"):
            K.gemm_heads(q[..., :kh.dim], t[L + "w_uk_t"], qa[..., :kh.dv])
            K.latent_rotate(q, pos, freq, kh.rot, out=qa, gain=gain)
        if Dp:
            with self._prof("attn_latent_decode"):
                K.attn_latent(qa[:Dp], self.k_cache[i], kh.dv, bt[:Dp], self._view(lay, "seq_lens_d"), out=lat[:Dp],
                              scratch=self.attn_scratch, max_seq_len=self.max_model_len if self._graph_mode else int(self._max_len_d), **kw)
        if P:
            with self._prof("attn_latent_prefill"):
                K.attn_latent(qa[Dp:], self.k_cache[i], kh.dv, bt[Dp:], self._view(lay, "seq_lens_p"), out=lat[Dp:],
                              q_start=self._view(lay, "q_start"), max_q_len=lay["_max_q"], **kw)
        with self._prof("latent_value"):
            K.gemm_heads(lat, t[L + "w_uv"], out)
        self.launches += 4 + (Dp > 0) + (P > 0)
        return full.view(-1, kh.hq * kh.vdim)

    def _latent_expanded(self, i, q, pos, bt, lay, out, freq, gain, kw) -> None:
        """Prompt portions long enough to pay for it: keys and values of all heads are computed from the cached latents of
        their sequences, and the attention runs on those (a third of the multiply-adds of attention over the latents)."""
        t, kh, L = self.w.t, self.w.heads[i], f"layers.{i}."
        lens, pages = self._view(lay, "seq_lens_p"), self._view(lay, "kv_pages")
        with self._prof("latent_expand"):
            rows = K.latent_gather(self.k_cache[i], bt, lens, pages, lay["_kv_rows"])
            K.latent_rotate(q, pos, freq, kh.rot, gain=gain)
        kv = self._gemm(rows[:, :kh.dv], t[L + "w_ukv"])
        with self._prof("attn_expanded"):
            K.attn_expanded(q, kv, rows, kh.vdim, lens, self._view(lay, "q_start"), pages, lay["_max_q"], out=out, **kw)
        self.launches += 3

    def _choose_expansion(self, lay) -> None:
        """Per latent layer, whether this step's prompt portions attend to expanded keys and values: their multiply-adds saved
        (at about a third of the rate of the tensor-core kernel) against those of the expansion."""
        pairs, rows = lay.get("_kv_pairs", 0), lay.get("_kv_rows", 0)
        flags = []
        for i, kh in enumerate(self.w.heads):
            on = f"layers.{i}.w_ukv" in self.w.t and self.block_size == 16
            if on:
                on = pairs * 3 * max(2 * kh.dv - kh.dim - kh.vdim, 0) + pairs * 2 * (kh.dim + kh.rot + kh.vdim) > rows * kh.dv * (kh.dim + kh.vdim)
            flags.append(bool(on))
        lay["_xp"] = tuple(flags)
        if not any(flags):
            lay["_kv_rows"] = 0

    def _rotation(self, ls):
        """(device table of a layer's rotation frequencies, gain on cosine and sine)."""
        key = (ls.rotary_dim, ls.rope_theta, ls.rope_llama3, ls.rope_yarn, ls.rope_linear)
        if key not in self._inv_freq:
            self._inv_freq[key] = rope_inv_freq(*key).to(self.device)
        return self._inv_freq[key], rope_gain(ls.rope_yarn)

    def _value_rotation(self, ls):
        """Frequencies of a layer's rotated values: all their dimensions, no scaling."""
        key = (ls.v_head_dim, ls.rope_theta)
        if key not in self._inv_freq:
            self._inv_freq[key] = rope_inv_freq(*key).to(self.device)
        return self._inv_freq[key]

    def _residual_norm(self, x, y, name, **kw):
        s, t = self.spec, self.w.t
        self.launches += 1
        with self._prof("residual_norm"):
            return K.residual_norm(x, y, t[name + ".w"], t.get(name + ".b"), eps=s.norm_eps,
                                   kind="rms" if s.norm == "rms" else "layer", width=s.hidden_size,
                                   offset_one=s.norm_weight_offset_one, out=x if self.w.dtype == torch.float32 else None, **kw)

    # ------------------------------------------------------------------------------------------
    # fused tensor-parallel path (F1 / F3)
    # ------------------------------------------------------------------------------------------
    def _fused_ok(self, T: int) -> bool:
        s, tp = self.spec, self.tp
        return (tp.fused and tp.comm is not None and s.layers is None and s.norm_placement == "input" and T % tp.world == 0 and T // tp.world <= tp.comm.max_rows
                and not s.parallel_residual and s.residual_scale == 1.0 and s.pos != "learned"
                and not s.embed_norm and s.final_norm
                and (s.moe is None or (s.moe.num_shared_experts == 0 and not s.moe.dense_parallel)))

    def _forward_tokens_fused(self, lay, shared_prefix_len: int) -> torch.Tensor:
        """Same math as ``_forward_tokens`` with the residual stream sharded by token rows between the two
        GEMM pairs of every layer: o_proj / down_proj epilogues push rows to their owner (reduce-scatter),
        the norm kernel sums, normalises and pushes to everyone (all-gather), and the next GEMM waits on
        the arrival counters inside its TMA producer.  No NCCL call, no separate reduction kernel."""
        s, t, tp = self.spec, self.w.t, self.tp
        c, W, r = tp.comm, tp.world, tp.rank
        T = lay["_T"]
        R = T // W
        H = s.hidden_size
        ids = self._view(lay, "token_ids")
        pos = self._view(lay, "positions")
        slots = self._view(lay, "slot_mapping")
        x_full = K.embed_gather(ids, t["embed"], scale=s.embed_scale)
        self.launches += 1
        xr = x_full[r * R:(r + 1) * R]                      # this rank's rows of the residual stream
        h_full = self._norm(x_full, "layers.0.ln1")         # layer 0 normalises all rows locally
        kind = "rms" if s.norm == "rms" else "layer"
        dense = [i for i in range(s.num_layers) if not s.layer_is_moe(i)]
        I_loc = 0
        if dense:
            L0 = f"layers.{dense[0]}."
            I_loc = (t[L0 + "w_gate_up"].shape[0] // 2) if s.mlp == "gated" else t[L0 + "w_up"].shape[0]
        rs0_out = c.rs_local_tensor(0, R)
        rs1_out = c.rs_local_tensor(1, R)
        ag_args = None
        # whole experts per rank and a dispatch area in the symmetric buffer: route locally, send pairs, not all rows
        self._moe_sparse = bool(s.moe is not None and self.w.ep and c.has_moe_dispatch and
                                os.environ.get("UB_MOE_SPARSE", "1") != "0")
        for i in range(s.num_layers):
            L = f"layers.{i}."
            qkv = self._gemm(h_full, t[L + "wqkv"], bias=t.get(L + "bqkv"), ag=ag_args, tag="gemm_ag" if ag_args else "gemm")
            self._rope_append(i, qkv, pos, slots)
            a = self._attention(i, qkv, lay, shared_prefix_len)
            # o_proj: partial rows go straight to their owner's receive slot
            self._gemm(a, t[L + "wo"], bias=t.get(L + "bo"), out=rs0_out.view(W * R, H)[:T], rs=c.gemm_rs(0, R),
                       tag="gemm_rs")
            sparse = s.layer_is_moe(i) and self._moe_sparse
            if sparse:
                # F5 / F6: this rank normalises and routes its own rows only; each (token, expert) pair travels to the
                # rank of its expert and its weighted output comes back into slot k of the combine area
                from .moe_runner import moe_sparse

                with self._prof("norm_rs"):
                    h_own, xr = K.norm(rs0_out, t[L + "ln2.w"], bias=t.get(L + "ln2.b"), residual=xr, eps=s.norm_eps,
                                       kind=kind, weight_offset_one=s.norm_weight_offset_one, want_residual_out=True, T=R,
                                       rs=c.norm_rs(0, rows_per_rank=R), reset=c.reset_after_ag(1))
                self.launches += 1
                moe_sparse(self, i, h_own, c, R)
                last = i == s.num_layers - 1
                nname = "final_norm" if last else f"layers.{i + 1}.ln1"
                with self._prof("norm_rs_ag"):
                    _, xr = K.norm(c.moe_comb_tensor(R), t[nname + ".w"], bias=t.get(nname + ".b"), residual=xr,
                                   eps=s.norm_eps, kind=kind, weight_offset_one=s.norm_weight_offset_one,
                                   want_residual_out=True, no_out=True, T=R, rs=c.norm_comb(), ag=c.norm_ag(0),
                                   reset=c.reset_after_ag(0))
                self.launches += 1
                h_full = c.ag_local_tensor(0, T)
                ag_args = c.gemm_ag(0, R)
                continue
            # sum partials + residual, normalise own rows, push to every rank's gather area 1
            with self._prof("norm_rs_ag"):
                _, xr = K.norm(rs0_out, t[L + "ln2.w"], bias=t.get(L + "ln2.b"), residual=xr, eps=s.norm_eps, kind=kind,
                               weight_offset_one=s.norm_weight_offset_one, want_residual_out=True, no_out=True, T=R,
                               rs=c.norm_rs(0, rows_per_rank=R), ag=c.norm_ag(1), reset=c.reset_after_ag(1))
            self.launches += 1
            h2 = c.ag_local_tensor(1, T)
            if s.layer_is_moe(i):
                # F5: the all-gather of the normalised rows is the dispatch (every rank sees every token and keeps
                # the pairs of its own experts); F6: the combine kernel stores partial rows into their owners' slots
                from ..dist.fused import AG1
                from .moe_runner import moe_partial

                K.wait_flags(c.local_flag_ptr(AG1), W, 1, self.device)
                self.launches += 1
                moe_partial(self, i, h2, None, combine_rs=c.gemm_rs(1, R))
            else:
                if s.mlp == "gated":
                    act = self._gemm(h2, t[L + "w_gate_up"], dual_rows=I_loc, act=s.act, ag=c.gemm_ag(1, R), tag="gemm_ag")
                else:
                    act = self._gemm(h2, t[L + "w_up"], bias=t.get(L + "b_up"), act=s.act, ag=c.gemm_ag(1, R), tag="gemm_ag")
                self._gemm(act, t[L + "w_down"], bias=t.get(L + "b_down"), out=rs1_out.view(W * R, H)[:T],
                           rs=c.gemm_rs(1, R), tag="gemm_rs")
            last = i == s.num_layers - 1
            nname = "final_norm" if last else f"layers.{i + 1}.ln1"
            with self._prof("norm_rs_ag"):
                _, xr = K.norm(rs1_out, t[nname + ".w"], bias=t.get(nname + ".b"), residual=xr, eps=s.norm_eps, kind=kind,
                               weight_offset_one=s.norm_weight_offset_one, want_residual_out=True, no_out=True, T=R,
                               rs=c.norm_rs(1, rows_per_rank=R), ag=c.norm_ag(0), reset=c.reset_after_ag(0))
            self.launches += 1
            h_full = c.ag_local_tensor(0, T)
            ag_args = c.gemm_ag(0, R)
        # the final-normed rows of all ranks arrive in gather area 0; wait for them before the row gather
        from ..dist.fused import AG0

        K.wait_flags(c.local_flag_ptr(AG0), W, 1, self.device)
        self.launches += 1
        self._final_norm_done = True
        return h_full

    def _mlp_noresid(self, i, h, dense_only=False):
        s, t = self.spec, self.w.t
        L = f"layers.{i}."
        if s.layer_is_moe(i) and not dense_only:
            from .moe_runner import moe_partial

            return moe_partial(self, i, h, None)
        if s.mlp == "gated":
            I = t[L + "w_gate_up"].shape[0] // 2
            a = self._gemm(h, t[L + "w_gate_up"], dual_rows=I, act=s.act)
        else:
            a = self._gemm(h, t[L + "w_up"], bias=t.get(L + "b_up"), act=s.act)
        return self._gemm(a, t[L + "w_down"], bias=t.get(L + "b_down"))

    def _final_rows(self, x, lay) -> torch.Tensor:
        """Final-normed rows of the step whose logits are asked for."""
        s, t = self.spec, self.w.t
        rows = self._view(lay, "sample_rows")
        if s.norm_placement == "both":
            self.launches += 1
            with self._prof("norm"):
                return K.sublayer_in(x, (), t["final_norm.w"], eps=s.norm_eps, rows=rows, width=s.hidden_size,
                                     offset_one=s.norm_weight_offset_one, **self._last_y)
        if s.norm == "tanh":
            return self._stream_in("final_norm", (), rows=rows, **self._last_y)
        if s.residual_fp32:
            self.launches += 1
            with self._prof("norm"):
                return K.row_norm(x, t["final_norm.w"], t.get("final_norm.b"), eps=s.norm_eps, rows=rows,
                                  kind="rms" if s.norm == "rms" else "layer", width=s.hidden_size,
                                  offset_one=s.norm_weight_offset_one)
        xs = x.index_select(0, rows.long()) if lay["_S"] != x.shape[0] else x
        if s.final_norm and not self._final_norm_done:
            xs = self._norm(xs, "final_norm")
        return xs

    def _logits_and_sample(self, x, lay, b: Optional[StepBatch], fl) -> torch.Tensor:
        s, t, tp = self.spec, self.w.t, self.tp
        S = lay["_S"]
        xs = self._final_rows(x, lay)
        logits = self._gemm(xs, t["lm_head"], bias=t.get("lm_head_bias"), out_scale=s.logit_scale)
        out = self.out_ids_dev[:S]
        greedy = fl is None
        if tp.world == 1:
            if greedy:
                K.sample(logits, out_ids=out)
            else:
                K.sample(logits, temperature=fl["temperature"], top_p=fl["top_p"], top_k=fl["top_k"],
                         seed=fl["seed"], step=fl["step"], out_ids=out)
            self.launches += 1
            return out
        if greedy:
            ids, vals = K.sample(logits, vocab_offset=tp.rank * self.w.vocab_shard, return_vals=True)
            if tp.comm is not None and S <= 2048:
                tp.comm.argmax_merge(vals, ids, out)     # F4: exchange over peer memory, no NCCL call
                self.launches += 2
                return out
            allv = tp.all_gather_cat(vals[None], dim=0)
            alli = tp.all_gather_cat(ids[None], dim=0)
            K.argmax_merge(allv.contiguous(), alli.contiguous(), out=out)
            self.launches += 2
            return out
        kc = fl.get("cand_k", 0)
        if tp.comm is not None and kc and tp.comm.can_gather_pairs(S, kc) and os.environ.get("UB_SAMPLE_PAIRS", "1") != "0":
            # F4s: every shard hands in the best `kc` entries of each row (after temperature), the pairs are gathered
            # over peer memory and every rank draws the same token from them -- the whole-vocabulary logits stay put
            cv, ci = K.sample(logits, temperature=fl["temperature"], top_p=fl["top_p"], top_k=fl["top_k"], seed=fl["seed"],
                              step=fl["step"], vocab_offset=tp.rank * self.w.vocab_shard, candidates=kc)
            av, ai = tp.comm.gather_pairs(cv, ci)
            K.sample(av, temperature=fl["temperature"], top_p=fl["top_p"], top_k=fl["top_k"], seed=fl["seed"],
                     step=fl["step"], out_ids=out, id_map=ai)
            self.launches += 3
            return out
        if (tp.comm is not None and fl.get("whole_vocab") and tp.comm.can_gather_pairs(S, 1) and S <= 2048
                and os.environ.get("UB_SAMPLE_PAIRS", "1") != "0"):
            # F4s, temperature only: every shard reports its maximum and its mass, all ranks work out which shard the
            # draw falls into and where, that shard picks the token and the winner is merged like a greedy one
            st = K.sample(logits, temperature=fl["temperature"], seed=fl["seed"], step=fl["step"], stats=True)
            mv, sv = tp.comm.gather_pairs(st[:, :1].contiguous(), st[:, 1:].contiguous().view(torch.int32))
            owner, local = K.vocab_shard_targets(mv, sv.view(torch.float32), fl["uniform"])
            local = torch.where(owner == tp.rank, local, torch.full_like(local, -1.0)).contiguous()
            ids, vals = K.sample(logits, temperature=fl["temperature"], seed=fl["seed"], step=fl["step"],
                                 vocab_offset=tp.rank * self.w.vocab_shard, target=local, return_vals=True)
            tp.comm.argmax_merge(vals, ids, out)
            self.launches += 4
            return out
        full = tp.all_gather_cat(logits, dim=-1)
        K.sample(full, temperature=fl["temperature"], top_p=fl["top_p"], top_k=fl["top_k"], seed=fl["seed"],
                 step=fl["step"], out_ids=out)
        self.launches += 1
        return out

    # ------------------------------------------------------------------------------------------
    # step execution
    # ------------------------------------------------------------------------------------------
    @staticmethod
    def _bucket(n: int) -> int:
        b = 1
        while b < n:
            b <<= 1
        return b

    @staticmethod
    def candidate_count(temperature, top_k, top_p) -> int:
        """Candidates per row and vocabulary shard that a tensor-parallel draw has to exchange: the largest ``top_k`` of
        the batch, or the 1024 survivors that a top-p draw keeps; greedy rows need one.  0 = some row samples from the
        whole vocabulary (pure temperature), so the logits have to be gathered."""
        cand = 1
        for i, t in enumerate(temperature):
            if t <= 0:
                continue
            k = top_k[i] if top_k is not None and top_k[i] else 0
            p = top_p[i] if top_p is not None else 1.0
            k = min(k, 1024) if k > 0 else (1024 if p < 1.0 else 0)
            if k == 0:
                return 0
            cand = max(cand, k)
        return cand

    def _sampling_tensors(self, b: StepBatch, S: int):
        if b.temperature is None or all(t <= 0 for t in b.temperature):
            return None
        f = self.fmeta_hosts[self._flip]
        f[:S] = torch.as_tensor(b.temperature, dtype=torch.float32)
        f[S:2 * S] = torch.as_tensor(b.top_p if b.top_p is not None else [1.0] * S, dtype=torch.float32)
        self.fmeta_dev[:2 * S].copy_(f[:2 * S], non_blocking=True)
        self.h2d_bytes += 8 * S
        tk = None
        if b.top_k is not None and any(k and k > 0 for k in b.top_k):
            tk = torch.as_tensor([k or 0 for k in b.top_k], dtype=torch.int32).to(self.device, non_blocking=True)
            self.h2d_bytes += 4 * S
        cand = self.candidate_count(b.temperature, b.top_k, b.top_p)
        # temperature-only rows everywhere: the draw from the whole vocabulary can be split over the shards; it needs the
        # uniform number of every row (the device sampler's Philox stream, evaluated here)
        whole = cand == 0 and all(t > 0 for t in b.temperature) and (b.top_k is None or not any(b.top_k)) and \
            (b.top_p is None or all(p >= 1.0 for p in b.top_p)) and self.tp.world > 1
        uni = None
        if whole:
            from ..sampling import philox_uniform

            uni = torch.tensor([philox_uniform(b.seed, b.step, r) for r in range(S)], dtype=torch.float32).to(self.device)
        return {"temperature": self.fmeta_dev[:S], "top_p": self.fmeta_dev[S:2 * S], "top_k": tk, "seed": b.seed,
                "step": b.step, "cand_k": cand, "whole_vocab": whole, "uniform": uni}

    MAX_GRAPHS = 96

    def launch(self, b: StepBatch) -> int:
        """Uploads the step's metadata and enqueues all kernels on the current stream.  Returns the number of
        sampled rows; ``fetch`` reads them back."""
        D = b.num_decode
        if len(b.token_ids) > self.max_tokens + self.max_num_seqs:
            raise InvalidInput("step exceeds max_num_batched_tokens")
        greedy = b.temperature is None or all(t <= 0 for t in b.temperature)
        graphable = self.use_cuda_graphs and greedy and len(b.token_ids) > 0
        self._max_len_d = max(b.seq_lens[:D]) if D else 0
        if graphable:
            lay = self._pack(b, bucketed=True)
            lay["_pp"] = b.prefill_shares_prefix
            key = (lay["_Dp"], lay["_P"], lay["_T"], lay["_max_q"], b.shared_prefix_len, b.prefill_shares_prefix, lay["_xp"],
                   lay.get("_kv_rows", 0))
            g = self.graphs.get(key)
            self._graph_mode = True
            self._upload(lay)
            if g is None and self.capture_new_graphs and len(self.graphs) < self.MAX_GRAPHS:
                # one eager run (sets kernel attributes, warms the allocator), then capture
                self._forward_and_sample(lay, b.shared_prefix_len, None)
                torch.cuda.current_stream().synchronize()
                before = self.launches
                graph = torch.cuda.CUDAGraph()
                with torch.cuda.graph(graph):
                    self._forward_and_sample(lay, b.shared_prefix_len, None)
                g = self.graphs[key] = (graph, self.launches - before, self._last_fused)
                self.captures += 1
            if g is not None:
                g[0].replay()
                self.launches += g[1]
                self._count_step(g[2])
            else:
                # a shape without a graph while captures are off (or the graph table is full): the padded step runs
                # as plain launches -- slower than a replay, but without the synchronisation a capture needs
                self._forward_and_sample(lay, b.shared_prefix_len, None)
                self._count_step(self._last_fused)
                self.eager_steps += 1
            return self._queue_readback(lay["_sel"])
        self._graph_mode = False
        lay = self._pack(b, bucketed=False)
        lay["_pp"] = b.prefill_shares_prefix
        self._upload(lay)
        fl = None if greedy else self._sampling_tensors(b, lay["_S"])
        self._forward_and_sample(lay, b.shared_prefix_len, fl)
        self._count_step(self._last_fused)
        return self._queue_readback(lay["_sel"])

    def _count_step(self, fused: bool) -> None:
        if self.tp.world > 1:
            if fused:
                self.fused_steps += 1
            else:
                self.unfused_steps += 1

    def _queue_readback(self, sel: List[int]) -> int:
        """Queues the device -> pinned host copy of the sampled ids behind the step and records an event; the
        returned handle of ``pending()`` stays valid while one later step is launched."""
        self._sel = sel
        n = (max(sel) + 1) if sel else 0
        host, ev, err = self.out_ids_hosts[self._flip], self._out_events[self._flip], self.err_hosts[self._flip]
        if n:
            host[:n].copy_(self.out_ids_dev[:n], non_blocking=True)
            self.d2h_bytes += 4 * n
        err.copy_(K.err_word(self.device), non_blocking=True)
        self.d2h_bytes += 8
        ev.record()
        self._handle = (ev, host, n, sel, err)
        return len(sel)

    def pending(self):
        """Handle of the step launched last; pass it to ``fetch`` after launching the next step."""
        return self._handle

    def _forward_and_sample(self, lay, shared_prefix_len, fl):
        x = self._forward_tokens(lay, shared_prefix_len)
        if lay["_S"] > 0:
            self._logits_and_sample(x, lay, None, fl)

    def fetch(self, handle=None) -> List[int]:
        """Waits for a launched step (the last one by default) and returns its sampled ids from pinned memory."""
        ev, host, n, sel, err = handle if handle is not None else self._handle
        t0 = time.perf_counter()
        ev.synchronize()
        self.wait_s += time.perf_counter() - t0
        code, detail = err.tolist()
        if code != 0:
            raise DeviceStepError(code, detail)
        if not sel:
            return []
        vals = host[:n].tolist()
        return [vals[i] for i in sel]

    def execute(self, b: StepBatch) -> List[int]:
        self.launch(b)
        return self.fetch()

    def reset_after_error(self) -> None:
        """After a ``DeviceStepError``: waits for the device, clears the error word and (tensor parallel, fused path)
        zeroes the arrival counters on every rank -- a collective call, every rank of the group has to make it."""
        torch.cuda.synchronize(self.device)
        K.err_word(self.device).zero_()
        K.gemm_streamk_reset(self.device)
        for e in self.err_hosts:
            e.zero_()
        if self.tp.comm is not None:
            self.tp.comm.reset()
        torch.cuda.synchronize(self.device)

    def kv_cache_bytes(self) -> int:
        own = [i for i, ls in enumerate(self.layers) if ls.has_kv]
        return sum(c[i].numel() * c[i].element_size() for c in (self.k_cache, self.v_cache) for i in own)

    def forward_logits(self, b: StepBatch) -> torch.Tensor:
        """Runs a step as plain launches without sampling: fp32 logits [len(b.sample_rows), vocab shard] of any of its
        rows (an empty list just appends to the cache)."""
        self._graph_mode = False
        self._max_len_d = max(b.seq_lens[:b.num_decode]) if b.num_decode else 0
        lay = self._pack(b, bucketed=False)
        lay["_pp"] = b.prefill_shares_prefix
        self._upload(lay)
        x = self._forward_tokens(lay, b.shared_prefix_len)
        if lay["_S"] == 0:
            return torch.empty(0, self.w.vocab_shard, dtype=torch.float32, device=self.device)
        return self._gemm(self._final_rows(x, lay), self.w.t["lm_head"], bias=self.w.t.get("lm_head_bias"),
                          out_scale=self.spec.logit_scale, out_dtype=torch.float32)

    logits_for = forward_logits

    def raise_on_device_error(self) -> None:
        """Waits for the work launched so far and raises if a kernel recorded an error."""
        code, detail = K.err_word(self.device).tolist()
        if code != 0:
            raise DeviceStepError(code, detail)
