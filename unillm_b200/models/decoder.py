"""``DecoderModel``: the parametric decoder-only transformer behind most of the model zoo.

Parameters live in a flat dict under canonical names (``embed``, ``layers.{i}.wqkv``, ``layers.{i}.wo``,
``layers.{i}.w_gate_up`` ...).  Q, K and V are always fused into one ``[(Hq + 2 Hkv) * D, H]`` matrix and
gate / up into one ``[2 I, H]`` matrix at load time -- one GEMM each on the device -- whatever packing
the family uses on disk; ``KeyScheme`` describes the on-disk names and ``export_hf`` writes them back.

``forward`` / ``forward_with_cache`` here are the straightforward PyTorch statement of the math and
serve as the numerical oracle (fp32 on CPU) and as the generic path for long-tail families; the
serving engine runs the same parameters through the fused sm_100a kernels with a paged KV cache
(``unillm_b200.engine.runner``).

Reference: ``crates/runtime/src/models_v2/llama.rs`` -- ``forward`` ``:203-236``, ``forward_with_cache``
``:421-464``, layer ``:631-680``, attention ``:921-1156``, MLP ``:1274-1297``, weight loading ``:175-201,
682-747``; the other families as cited in ``unillm_b200/models/families.py``.
"""
from __future__ import annotations

import dataclasses
import math
from typing import Dict, List, Optional

import torch
import torch.nn.functional as F

from ..kv_cache import KVCache
from ..model_core import Model, ModelInputs, ModelOutputs, ModelWeights, WeightMetadata
from ..precompute import RoPECache, alibi_slopes, apply_rope
from ..tensor_core import ops_fn
from ..types import InvalidInput, LoadingError
from . import mixers as MX
from .spec import DecoderSpec, KeyScheme, LayerSpec, MoESpec


def _f(x):
    return x.float() if x.dtype in (torch.bfloat16, torch.float16) else x


class DecoderModel(Model):
    """Subclasses set ``config_class``, ``scheme`` and implement ``spec_from_config``."""

    scheme: KeyScheme = KeyScheme()

    def __init__(self, config, reference_quirks: bool = False):
        super().__init__(config)
        self.spec: DecoderSpec = self.spec_from_config(config)
        self.reference_quirks = reference_quirks
        self.p: Dict[str, torch.Tensor] = {}
        self._rope: Optional[Dict[tuple, RoPECache]] = None
        self._alibi: Optional[torch.Tensor] = None

    @classmethod
    def spec_from_config(cls, config) -> DecoderSpec:  # pragma: no cover - abstract
        raise NotImplementedError

    # ------------------------------------------------------------------------------------------
    # parameter inventory
    # ------------------------------------------------------------------------------------------
    def param_shapes(self) -> Dict[str, tuple]:
        s = self.spec
        H = s.hidden_size
        E = s.embed_proj_dim or H
        shp: Dict[str, tuple] = {"embed": (s.vocab_size, E)}
        if s.embed_proj_dim:
            shp["project_in"] = (H, E)
            shp["project_out"] = (E, H)
        if s.pos == "learned":
            shp["pos_embed"] = (s.max_position_embeddings + s.learned_pos_offset, H)
        if s.embed_norm:
            shp["embed_norm.w"] = (H,)
            shp["embed_norm.b"] = (H,)
        for i in range(s.num_layers):
            L = f"layers.{i}."
            ls = s.layer(i)
            shp[L + "ln1.w"] = (H,)
            if s.norm_bias:
                shp[L + "ln1.b"] = (H,)
            if not (s.parallel_residual and s.parallel_shared_norm) and ls.mlp is not None:
                shp[L + "ln2.w"] = (H,)
                if s.norm_bias:
                    shp[L + "ln2.b"] = (H,)
            if s.norm == "tanh":
                shp.update({L + n + ".alpha": () for n in ("ln1", "ln2") if L + n + ".w" in shp})
            if s.token_shift:
                shp[L + "shift"] = (H,)
            if s.depth_average:
                shp[L + "dwa"] = (i + 2,)
            if s.norm_placement == "both":
                shp[L + "ln1b.w"] = (H,)
                if ls.mlp is not None:
                    shp[L + "ln2b.w"] = (H,)
            if s.input_conv:
                shp[L + "conv1"] = (H, s.input_conv)
                if ls.mlp is not None:
                    shp[L + "conv2"] = (H, s.input_conv)
            if ls.mixer != "attention":
                shp.update({L + n: t for n, t in MX.mixer_shapes(ls, H).items()})
            else:
                shp[L + "wqkv"] = (ls.qkv_size, H)
                if s.has_qkv_bias(i):
                    shp[L + "bqkv"] = (ls.qkv_size,)
                kind = s.qk_norm_kind(i)
                if kind:
                    shp[L + "q_norm"] = (ls.q_size if kind == "row" else ls.head_dim,)
                    if ls.kv_from is None:
                        shp[L + "k_norm"] = (ls.k_size if kind == "row" else ls.head_dim,)
                if ls.sink:
                    shp[L + "sink"] = (ls.num_heads,)
                if ls.out_gate:
                    shp[L + "w_og"] = (ls.gate_size, H)
                if ls.maps == 2:
                    shp[L + "lambdas"] = (4, ls.head_dim)
                shp[L + "wo"] = (H, ls.o_size)
                if s.o_bias:
                    shp[L + "bo"] = (H,)
            if ls.beside is not None:
                shp.update({L + "beside." + n: t for n, t in MX.mixer_shapes(ls.beside, H).items()})
            moe = ls.mlp == "moe"
            if ls.mlp == "dense" or (moe and ls.moe.dense_parallel):
                I = s.layer_intermediate(i)
                if s.act == "xielu":
                    shp[L + "act"] = (2,)
                if s.mlp == "gated":
                    shp[L + "w_gate_up"] = (2 * I, H)
                else:
                    shp[L + "w_up"] = (I, H)
                    if s.mlp_bias:
                        shp[L + "b_up"] = (I,)
                shp[L + "w_down"] = (H, I)
                if s.mlp_bias:
                    shp[L + "b_down"] = (H,)
            if moe:
                m = ls.moe
                shp[L + "router"] = (m.num_experts, H)
                if m.router_bias:
                    shp[L + "router_b"] = (m.num_experts,)
                if m.correction:
                    shp[L + "correction"] = (m.num_experts,)
                shp[L + "experts_gate_up"] = (m.num_experts, (2 if m.gated else 1) * m.intermediate_size, H)
                shp[L + "experts_down"] = (m.num_experts, H, m.intermediate_size)
                if m.num_shared_experts:
                    Is = m.shared_width
                    shp[L + "shared_gate_up"] = ((2 if m.gated else 1) * Is, H)
                    shp[L + "shared_down"] = (H, Is)
                    if m.shared_gate:
                        shp[L + "shared_sg"] = (1, H)
        if s.final_norm:
            shp["final_norm.w"] = (H,)
            if s.norm_bias:
                shp["final_norm.b"] = (H,)
            if s.norm == "tanh":
                shp["final_norm.alpha"] = ()
        if not s.tie_embeddings:
            shp["lm_head"] = (s.vocab_size, E)
        if s.lm_head_bias:
            shp["lm_head_bias"] = (s.vocab_size,)
        return shp

    def _init_params(self, init="zeros", seed=0, dtype=torch.float32, device=torch.device("cpu")):
        g = torch.Generator(device="cpu").manual_seed(seed)
        std = self.spec.initializer_range
        self.p = {}
        for name, shape in self.param_shapes().items():
            is_norm_w = name.endswith((".w", "q_norm", "k_norm")) and len(shape) == 1
            if init == "zeros":
                t = torch.zeros(shape, dtype=dtype)
            elif name.endswith(("q_norm", "k_norm")) and self.spec.layers is not None:
                t = torch.ones(shape, dtype=dtype)
            elif name.endswith(".alpha"):
                t = torch.full(shape, 0.5, dtype=dtype)
            elif name.endswith(".dwa"):                                      # the layer's own result
                t = torch.zeros(shape, dtype=dtype)
                t[-1] = 1.0
            elif is_norm_w:
                t = torch.zeros(shape, dtype=dtype) if self.spec.norm_weight_offset_one else torch.ones(shape, dtype=dtype)
            elif name.endswith(("q_a_norm", "kv_a_norm", "o_norm")):         # weights that are not stored around zero
                t = torch.ones(shape, dtype=dtype)
            elif name.endswith((".b", "bqkv", "bo", "b_up", "b_down", "lm_head_bias", "router_b", "sink", "correction", "A_log", "dt_bias")):
                t = torch.zeros(shape, dtype=dtype)
            else:
                t = (torch.randn(shape, generator=g, dtype=torch.float32) * std).to(dtype)
            self.p[name] = t.to(device)
        self.device, self.dtype = device, dtype
        self._rope = self._alibi = None

    # ------------------------------------------------------------------------------------------
    # loading from / exporting to the family's on-disk names
    # ------------------------------------------------------------------------------------------
    def _find(self, w: ModelWeights, prefixes, names, suffix=".weight"):
        """First present alias; block-quantised (GGUF) tensors are dequantised on the way in."""
        suffix = {".weight": self.scheme.weight_suffix, ".bias": self.scheme.bias_suffix}.get(suffix, suffix)
        for pre in prefixes:
            for n in names:
                t = w.get(pre + n + suffix)
                if t is not None:
                    return t
                q = w.get_quantized(pre + n + suffix)
                if q is not None:
                    return q.dequantize()
        return None

    def _complete_spec(self, weights: ModelWeights) -> DecoderSpec:
        """The spec with the sizes that only the tensors' shapes give (the ranks of low-rank decays and gates)."""
        s = self.spec
        if s.layers is None:
            return s
        layers = list(s.layers)
        for i, ls in enumerate(layers):
            need = {}
            if ls.mixer == "wkv":
                need["decay_rank"] = "w_d1"
            if ls.mixer == "delta" and ls.decay == "channel":
                need["decay_rank"] = "w_a1"
            if ls.mixer == "delta" and ls.low_rank_gate:
                need["gate_rank"] = "w_g1"
            for rank, name in need.items():
                if getattr(ls, rank):
                    continue
                t = self._find(weights, tuple(p.format(i=i) for p in self.scheme.layer), self.scheme.mixers[ls.mixer][name])
                if t is None:
                    raise LoadingError(f"{type(self).__name__}: missing weight layer {i} {name}")
                layers[i] = dataclasses.replace(layers[i], **{rank: t.shape[0]})
        return dataclasses.replace(s, layers=tuple(layers))

    def _side(self, names, i: int, second: bool = False):
        """A mixer's tensor names in layer ``i``: another prefix where two mixers stand side by side."""
        if self.spec.layer(i).beside is None or self.scheme.sides is None:
            return tuple(names)
        old, new = self.scheme.sides[0], self.scheme.sides[2 if second else 1]
        return tuple(new + n[len(old):] if n.startswith(old) else n for n in names)

    def _load_mixer(self, weights: ModelWeights, i: int, ls: LayerSpec, pre, out: Dict[str, torch.Tensor], second: bool = False) -> None:
        """Parameters of a layer's mixer that is not plain attention, each put together from the tensors the scheme names."""
        for name, shape in MX.mixer_shapes(ls, self.spec.hidden_size).items():
            names = self._side(self.scheme.mixers[ls.mixer][name], i, second)
            parts = [self._find(weights, pre, (n,)) for n in names]
            if any(t is None for t in parts):
                raise LoadingError(f"{type(self).__name__}: missing weight layer {i} {name} {names}")
            out[f"layers.{i}.{'beside.' if second else ''}{name}"] = MX.join_parts(parts, shape)

    def _load(self, weights: ModelWeights, dtype=None, device=None):
        self.spec = self._complete_spec(weights)
        s, k = self.spec, self.scheme
        dtype = dtype or torch.float32
        dev = torch.device(device) if device is not None else torch.device("cpu")
        shapes = self.param_shapes()
        out: Dict[str, torch.Tensor] = {}

        def T(t):
            return t.t() if (k.transposed and t is not None and t.dim() == 2) else t

        def need(t, what):
            if t is None:
                raise LoadingError(f"{type(self).__name__}: missing weight {what}")
            return t

        def deq(name_candidates):
            # quantised GGUF tensors are dequantised here; the engine re-quantises on demand
            for n in name_candidates:
                q = weights.get_quantized(n)
                if q is not None:
                    return q.dequantize()
            return None

        root = ("",)
        out["embed"] = need(self._find(weights, root, k.embed), "embedding " + str(k.embed))
        if s.embed_proj_dim:
            out["project_in"] = need(self._find(weights, root, k.project_in), "project_in")
            out["project_out"] = need(self._find(weights, root, k.project_out), "project_out")
        if s.pos == "learned":
            out["pos_embed"] = need(self._find(weights, root, k.pos_embed), "position embedding")
        if s.embed_norm:
            out["embed_norm.w"] = need(self._find(weights, root, k.embed_norm), "embed norm")
            b = self._find(weights, root, k.embed_norm, ".bias")
            out["embed_norm.b"] = b if b is not None else torch.zeros(s.hidden_size)
        for i in range(s.num_layers):
            L = f"layers.{i}."
            ls = s.layer(i)
            pre = tuple(p.format(i=i) for p in k.layer)
            out[L + "ln1.w"] = need(self._find(weights, pre, k.ln1), f"layer {i} ln1")
            if s.norm_bias:
                b = self._find(weights, pre, k.ln1, ".bias")
                out[L + "ln1.b"] = b if b is not None else torch.zeros(s.hidden_size)
            if L + "ln2.w" in shapes:
                t = self._find(weights, pre, k.ln2)
                out[L + "ln2.w"] = t if t is not None else out[L + "ln1.w"].clone()
                if s.norm_bias:
                    b = self._find(weights, pre, k.ln2, ".bias")
                    out[L + "ln2.b"] = b if b is not None else torch.zeros(s.hidden_size)
            for n, names in (("ln1", k.ln1), ("ln2", k.ln2)):
                if L + n + ".alpha" in shapes:
                    out[L + n + ".alpha"] = need(self._find_slope(weights, pre, names), f"layer {i} {n} slope")
            for n, names in (("shift", k.shift), ("dwa", k.depth_average), ("ln1b.w", k.ln1b), ("ln2b.w", k.ln2b), ("conv1", k.conv1), ("conv2", k.conv2), ("act", k.act)):
                if L + n in shapes:
                    out[L + n] = need(self._find(weights, pre, names), f"layer {i} {n}")
            # ---- mixer ----
            if ls.mixer != "attention":
                self._load_mixer(weights, i, ls, pre, out)
            else:
                self._load_attention(weights, i, pre, out, T, need, deq)
            if ls.beside is not None:
                self._load_mixer(weights, i, ls.beside, pre, out, second=True)
            # ---- MLP ----
            moe = ls.mlp == "moe"
            if ls.mlp == "dense" or (moe and ls.moe.dense_parallel):
                if s.mlp == "gated":
                    gu = T(self._find(weights, pre, k.gate_up)) if k.gate_up else None
                    if gu is None:
                        g = T(self._find(weights, pre, k.gate))
                        u = T(self._find(weights, pre, k.up))
                        if g is None:
                            g = deq([p + n + ".weight" for p in pre for n in k.gate])
                            u = deq([p + n + ".weight" for p in pre for n in k.up])
                        gu = torch.cat([need(g, f"layer {i} gate_proj"), need(u, f"layer {i} up_proj")], dim=0)
                    out[L + "w_gate_up"] = gu
                else:
                    out[L + "w_up"] = need(T(self._find(weights, pre, k.up)), f"layer {i} fc1")
                    if s.mlp_bias:
                        b = self._find(weights, pre, k.up, ".bias")
                        out[L + "b_up"] = b if b is not None else torch.zeros(s.layer_intermediate(i))
                dn = T(self._find(weights, pre, k.down))
                if dn is None:
                    dn = deq([p + n + ".weight" for p in pre for n in k.down])
                out[L + "w_down"] = need(dn, f"layer {i} down_proj")
                if s.mlp_bias:
                    b = self._find(weights, pre, k.down, ".bias")
                    out[L + "b_down"] = b if b is not None else torch.zeros(s.hidden_size)
            if moe:
                m = ls.moe
                out[L + "router"] = need(self._find(weights, pre, k.router), f"layer {i} router")
                if m.router_bias:
                    out[L + "router_b"] = need(self._find(weights, pre, k.router, ".bias"), f"layer {i} router bias")
                if m.correction:
                    out[L + "correction"] = need(self._find(weights, pre, k.correction), f"layer {i} router correction")
                gus, dns = [], []
                for e in range(m.num_experts):
                    epre = tuple(p + x.format(e=e) for p in pre for x in k.expert)
                    g = self._find(weights, epre, k.e_gate)
                    u = self._find(weights, epre, k.e_up) if m.gated else None
                    d = self._find(weights, epre, k.e_down)
                    need(g, f"layer {i} expert {e} gate"), need(d, f"layer {i} expert {e} down")
                    gus.append(torch.cat([g, need(u, f"layer {i} expert {e} up")], 0) if m.gated else g)
                    dns.append(d)
                out[L + "experts_gate_up"] = torch.stack(gus)
                out[L + "experts_down"] = torch.stack(dns)
                if m.num_shared_experts:
                    g = need(self._find(weights, pre, k.shared_gate), "shared gate")
                    if m.gated:
                        g = torch.cat([g, need(self._find(weights, pre, k.shared_up), "shared up")], 0)
                    out[L + "shared_gate_up"] = g
                    out[L + "shared_down"] = need(self._find(weights, pre, k.shared_down), "shared down")
                    if m.shared_gate:
                        out[L + "shared_sg"] = need(self._find(weights, pre, k.shared_sg), f"layer {i} gate of the shared expert")
        if s.final_norm:
            out["final_norm.w"] = need(self._find(weights, root, k.final_norm), "final norm")
            if s.norm_bias:
                b = self._find(weights, root, k.final_norm, ".bias")
                out["final_norm.b"] = b if b is not None else torch.zeros(s.hidden_size)
            if s.norm == "tanh":
                out["final_norm.alpha"] = need(self._find_slope(weights, root, k.final_norm), "final norm slope")
        if not s.tie_embeddings:
            lm = self._find(weights, root, k.lm_head)
            if lm is None:
                lm = deq([n + ".weight" for n in k.lm_head])
            out["lm_head"] = lm if lm is not None else out["embed"]
        if s.lm_head_bias:
            b = self._find(weights, root, k.lm_head, ".bias")
            out["lm_head_bias"] = b if b is not None else torch.zeros(s.vocab_size)
        for name, shape in shapes.items():
            if name not in out:
                raise LoadingError(f"internal: parameter {name} was not produced by the loader")
            if tuple(out[name].shape) != tuple(shape):
                raise LoadingError(f"{name}: expected shape {tuple(shape)}, file has {tuple(out[name].shape)}")
        self.p = {n: t.to(device=dev, dtype=dtype).contiguous() for n, t in out.items() if n in shapes}
        self.device, self.dtype = dev, dtype
        self._rope = self._alibi = None

    def _find_slope(self, weights: ModelWeights, pre, names):
        """The scalar slope of a Dynamic Tanh (stored with or without an axis)."""
        t = self._find(weights, pre, tuple(n + self.scheme.alpha_suffix for n in names))
        return None if t is None else t.reshape(())

    def _load_attention(self, weights: ModelWeights, i: int, pre, out: Dict[str, torch.Tensor], T, need, deq) -> None:
        """Projections, head norms and sinks of one layer's attention."""
        s, k, ls = self.spec, self.scheme, self.spec.layer(i)
        L = f"layers.{i}."
        nq, nk, nv, no, nqn, nkn, nsink = (self._side(n, i) for n in (k.q, k.k, k.v, k.o, k.q_norm, k.k_norm, k.sink))
        packed = T(self._find(weights, pre, k.qkv)) if k.qkv else None
        pb = self._find(weights, pre, k.qkv, ".bias") if k.qkv else None
        if packed is not None:
            out[L + "wqkv"], bq = self._unpack_qkv(packed, pb)
        else:
            q = T(self._find(weights, pre, nq))
            kk = T(self._find(weights, pre, nk))
            v = T(self._find(weights, pre, nv))
            if q is None:
                names = [p + n + ".weight" for p in pre for n in nq]
                q, kk, v = deq(names), deq([n.replace(nq[0], nk[0]) for n in names]), \
                    deq([n.replace(nq[0], nv[0]) for n in names])
            need(q, f"layer {i} q_proj")
            if ls.kv_from is None:
                need(kk, f"layer {i} k_proj"), need(v, f"layer {i} v_proj")
                out[L + "wqkv"] = torch.cat([q, kk, v], dim=0)
            else:
                out[L + "wqkv"] = q
            bq = None
            qb = self._find(weights, pre, nq, ".bias")
            if qb is not None:
                kb = self._find(weights, pre, nk, ".bias")
                vb = self._find(weights, pre, nv, ".bias")
                bq = torch.cat([qb, kb if kb is not None else torch.zeros(ls.k_size),
                                vb if vb is not None else torch.zeros(ls.v_size)])
        if s.has_qkv_bias(i):
            out[L + "bqkv"] = bq if bq is not None else torch.zeros(ls.qkv_size)
        if s.qk_norm_kind(i):
            out[L + "q_norm"] = need(self._find(weights, pre, nqn), "q_norm")
            if ls.kv_from is None:
                out[L + "k_norm"] = need(self._find(weights, pre, nkn), "k_norm")
        if ls.sink:
            out[L + "sink"] = need(self._find(weights, pre, nsink, ""), f"layer {i} sinks")
        if ls.out_gate:
            out[L + "w_og"] = need(self._find(weights, pre, k.out_gate), f"layer {i} output gate")
        if ls.maps == 2:
            out[L + "lambdas"] = torch.stack([need(self._find(weights, pre, (n,)), f"layer {i} {n}") for n in k.lambdas])
        wo = T(self._find(weights, pre, no))
        if wo is None:
            wo = deq([p + n + ".weight" for p in pre for n in no])
        out[L + "wo"] = need(wo, f"layer {i} o_proj")
        if s.o_bias:
            b = self._find(weights, pre, no, ".bias")
            out[L + "bo"] = b if b is not None else torch.zeros(s.hidden_size)

    def _unpack_qkv(self, w: torch.Tensor, b: Optional[torch.Tensor]):
        """On-disk packed QKV -> canonical [Q; K; V] row order."""
        s, lay = self.spec, self.scheme.qkv_layout
        D, Hq, Hkv = s.head_dim, s.num_heads, s.num_kv_heads
        if lay == "concat":
            return w, b
        if lay == "per_head":        # [h][q, k, v] (GPT-NeoX, BLOOM); MHA only
            wr = w.reshape(Hq, 3, D, -1)
            w2 = torch.cat([wr[:, 0].reshape(Hq * D, -1), wr[:, 1].reshape(Hq * D, -1), wr[:, 2].reshape(Hq * D, -1)])
            b2 = None
            if b is not None:
                br = b.reshape(Hq, 3, D)
                b2 = torch.cat([br[:, 0].reshape(-1), br[:, 1].reshape(-1), br[:, 2].reshape(-1)])
            return w2, b2
        if lay == "grouped":         # [kv group][G q heads, k, v] (Falcon new decoder architecture)
            G = Hq // Hkv
            wr = w.reshape(Hkv, G + 2, D, -1)
            w2 = torch.cat([wr[:, :G].reshape(Hq * D, -1), wr[:, G].reshape(Hkv * D, -1), wr[:, G + 1].reshape(Hkv * D, -1)])
            b2 = None
            if b is not None:
                br = b.reshape(Hkv, G + 2, D)
                b2 = torch.cat([br[:, :G].reshape(-1), br[:, G].reshape(-1), br[:, G + 1].reshape(-1)])
            return w2, b2
        raise LoadingError(f"unknown qkv layout {lay}")

    def _pack_qkv(self, w: torch.Tensor) -> torch.Tensor:
        """Inverse of ``_unpack_qkv`` for weights (used by ``export_hf``)."""
        s, lay = self.spec, self.scheme.qkv_layout
        D, Hq, Hkv = s.head_dim, s.num_heads, s.num_kv_heads
        if lay == "concat":
            return w
        q, k, v = w[:Hq * D], w[Hq * D:Hq * D + Hkv * D], w[Hq * D + Hkv * D:]
        if lay == "per_head":
            return torch.stack([q.reshape(Hq, D, -1), k.reshape(Hq, D, -1), v.reshape(Hq, D, -1)], 1).reshape(3 * Hq * D, -1)
        G = Hq // Hkv
        return torch.cat([q.reshape(Hkv, G, D, -1), k.reshape(Hkv, 1, D, -1), v.reshape(Hkv, 1, D, -1)], 1).reshape((Hq + 2 * Hkv) * D, -1)

    def export_hf(self) -> ModelWeights:
        """Parameters under the family's on-disk names (first alias of each scheme entry)."""
        s, k = self.spec, self.scheme
        out: Dict[str, torch.Tensor] = {}
        WS, BS = k.weight_suffix, k.bias_suffix

        def T(t):
            return t.t().contiguous() if k.transposed and t.dim() == 2 else t

        out[k.embed[0] + WS] = self.p["embed"]
        if s.embed_proj_dim:
            out[k.project_in[0] + WS] = self.p["project_in"]
            out[k.project_out[0] + WS] = self.p["project_out"]
        if s.pos == "learned":
            out[k.pos_embed[0] + WS] = self.p["pos_embed"]
        if s.embed_norm:
            out[k.embed_norm[0] + WS] = self.p["embed_norm.w"]
            out[k.embed_norm[0] + BS] = self.p["embed_norm.b"]
        for i in range(s.num_layers):
            L, pre = f"layers.{i}.", k.layer[0].format(i=i)
            ls = s.layer(i)
            out[pre + k.ln1[0] + WS] = self.p[L + "ln1.w"]
            if s.norm_bias:
                out[pre + k.ln1[0] + BS] = self.p[L + "ln1.b"]
            if L + "ln2.w" in self.p:
                out[pre + k.ln2[0] + WS] = self.p[L + "ln2.w"]
                if s.norm_bias:
                    out[pre + k.ln2[0] + BS] = self.p[L + "ln2.b"]
            for n, names in (("ln1", k.ln1), ("ln2", k.ln2)):
                if L + n + ".alpha" in self.p:
                    out[pre + names[0] + k.alpha_suffix + WS] = self.p[L + n + ".alpha"]
            for n, names, suffix in (("shift", k.shift, WS), ("dwa", k.depth_average, WS), ("ln1b.w", k.ln1b, WS), ("ln2b.w", k.ln2b, WS), ("conv1", k.conv1, WS), ("conv2", k.conv2, WS),
                                     ("act", k.act, WS)):
                if L + n in self.p:
                    out[pre + names[0] + suffix] = self.p[L + n]
            side = lambda names: self._side(names, i)[0]
            for mx, at in zip(ls.mixers, ("", "beside.")):
                if mx.mixer == "attention":
                    continue
                for n in MX.mixer_shapes(mx, s.hidden_size):
                    names = self._side(k.mixers[mx.mixer][n], i, bool(at))
                    for name, t in zip(names, MX.split_parts(self.p[L + at + n], mx, n, len(names))):
                        out[pre + name + WS] = t
            if ls.mixer == "attention":
                wqkv = self.p[L + "wqkv"]
                if k.qkv:
                    out[pre + k.qkv[0] + WS] = T(self._pack_qkv(wqkv))
                    if s.qkv_bias:
                        out[pre + k.qkv[0] + BS] = self._pack_qkv(self.p[L + "bqkv"][:, None])[:, 0]
                elif ls.kv_from is not None:
                    out[pre + side(k.q) + WS] = T(wqkv)
                else:
                    q, kk, v = wqkv.split([ls.q_size, ls.k_size, ls.v_size])
                    out[pre + side(k.q) + WS], out[pre + side(k.k) + WS], out[pre + side(k.v) + WS] = T(q), T(kk), T(v)
                    if s.has_qkv_bias(i):
                        qb, kb, vb = self.p[L + "bqkv"].split([ls.q_size, ls.k_size, ls.v_size])
                        out[pre + side(k.q) + BS], out[pre + side(k.k) + BS], out[pre + side(k.v) + BS] = qb, kb, vb
                if s.qk_norm_kind(i):
                    out[pre + side(k.q_norm) + WS] = self.p[L + "q_norm"]
                    if ls.kv_from is None:
                        out[pre + side(k.k_norm) + WS] = self.p[L + "k_norm"]
                if ls.sink:
                    out[pre + side(k.sink)] = self.p[L + "sink"]
                if ls.out_gate:
                    out[pre + k.out_gate[0] + WS] = self.p[L + "w_og"]
                if ls.maps == 2:
                    out.update({pre + n + WS: t for n, t in zip(k.lambdas, self.p[L + "lambdas"].unbind(0))})
                out[pre + side(k.o) + WS] = T(self.p[L + "wo"])
                if s.o_bias:
                    out[pre + side(k.o) + BS] = self.p[L + "bo"]
            if L + "w_gate_up" in self.p:
                if k.gate_up:
                    out[pre + k.gate_up[0] + WS] = T(self.p[L + "w_gate_up"])
                else:
                    g, u = self.p[L + "w_gate_up"].chunk(2, 0)
                    out[pre + k.gate[0] + WS], out[pre + k.up[0] + WS] = T(g), T(u)
            if L + "w_up" in self.p:
                out[pre + k.up[0] + WS] = T(self.p[L + "w_up"])
                if s.mlp_bias:
                    out[pre + k.up[0] + BS] = self.p[L + "b_up"]
            if L + "w_down" in self.p:
                out[pre + k.down[0] + WS] = T(self.p[L + "w_down"])
                if s.mlp_bias:
                    out[pre + k.down[0] + BS] = self.p[L + "b_down"]
            if L + "router" in self.p:
                m = ls.moe
                out[pre + k.router[0] + WS] = self.p[L + "router"]
                if m.router_bias:
                    out[pre + k.router[0] + BS] = self.p[L + "router_b"]
                if m.correction:
                    out[pre + k.correction[0] + WS] = self.p[L + "correction"]
                for e in range(m.num_experts):
                    ep = pre + k.expert[0].format(e=e)
                    gu = self.p[L + "experts_gate_up"][e]
                    if m.gated:
                        g, u = gu.chunk(2, 0)
                        out[ep + k.e_gate[0] + WS], out[ep + k.e_up[0] + WS] = g, u
                    else:
                        out[ep + k.e_gate[0] + WS] = gu
                    out[ep + k.e_down[0] + WS] = self.p[L + "experts_down"][e]
                if m.num_shared_experts:
                    if m.gated:
                        g, u = self.p[L + "shared_gate_up"].chunk(2, 0)
                        out[pre + k.shared_gate[0] + WS], out[pre + k.shared_up[0] + WS] = g, u
                    else:
                        out[pre + k.shared_gate[0] + WS] = self.p[L + "shared_gate_up"]
                    out[pre + k.shared_down[0] + WS] = self.p[L + "shared_down"]
                    if m.shared_gate:
                        out[pre + k.shared_sg[0] + WS] = self.p[L + "shared_sg"]
        if s.final_norm:
            out[k.final_norm[0] + WS] = self.p["final_norm.w"]
            if s.norm_bias:
                out[k.final_norm[0] + BS] = self.p["final_norm.b"]
            if s.norm == "tanh":
                out[k.final_norm[0] + k.alpha_suffix + WS] = self.p["final_norm.alpha"]
        if not s.tie_embeddings:
            out[k.lm_head[0] + WS] = self.p["lm_head"]
        if s.lm_head_bias:
            out[k.lm_head[0] + BS] = self.p["lm_head_bias"]
        md = WeightMetadata(architecture=type(self._config).__name__, total_params=sum(t.numel() for t in out.values()),
                            format="memory", dtype=str(self.dtype))
        return ModelWeights({n: t.contiguous() for n, t in out.items()}, md)

    def parameters(self) -> Dict[str, torch.Tensor]:
        return self.p

    def _move(self, dev, dtype):
        self.p = {n: (t.to(device=dev, dtype=dtype) if dtype is not None else t.to(dev)) for n, t in self.p.items()}
        self._rope = self._alibi = None

    # ------------------------------------------------------------------------------------------
    # math
    # ------------------------------------------------------------------------------------------
    def _norm(self, x, name, layer_level=True):
        s = self.spec
        w, b = self.p[name + ".w"], self.p.get(name + ".b")
        eps = s.norm_eps
        if self.reference_quirks:
            if layer_level and s.ref_layer_eps is not None:
                eps = s.ref_layer_eps
            if s.ref_ln_star:
                return ops_fn.layer_norm(x, w, None, eps)
        if s.norm == "tanh":
            return (torch.tanh(_f(self.p[name + ".alpha"]) * _f(x)) * _f(w) + _f(b)).to(x.dtype)
        if s.norm == "layer":
            return ops_fn.layer_norm(x, w, b, eps)
        if s.norm_weight_offset_one:
            return ops_fn.rms_norm(x, (w.float() + 1.0).to(w.dtype), eps)
        return ops_fn.rms_norm(x, w, eps)

    def _rope_cache(self, need_len: int, ls: Optional[LayerSpec] = None) -> RoPECache:
        """Tables of one rotation; layers with the same rotation share them."""
        s = self.spec
        ls = ls or s.layer(0)
        key = (ls.rotary_dim, ls.rope_theta, ls.rope_llama3, ls.rope_yarn, ls.rope_linear)
        if self._rope is None:
            self._rope = {}
        c = self._rope.get(key)
        if c is None or c.max_seq_len < need_len or c.cos.device != self.device:
            n = max(need_len, min(s.max_position_embeddings, 8192))
            c = self._rope[key] = RoPECache(ls.head_dim, n, ls.rope_theta, rotary_dim=ls.rotary_dim,
                                            position_scale=s.rope_pos_scale, llama3=ls.rope_llama3, yarn=ls.rope_yarn,
                                            linear=ls.rope_linear, device=self.device)
        return c

    def _value_rope(self, need_len: int, ls: LayerSpec) -> RoPECache:
        """Tables of the rotation of a layer's values: all their dimensions, no scaling."""
        return self._rope_cache(need_len, dataclasses.replace(ls, head_dim=ls.v_head_dim, rotary_dim=ls.v_head_dim, rope_llama3=None,
                                                              rope_yarn=None, rope_linear=1.0))

    def _project_qkv(self, i: int, h: torch.Tensor):
        """(q, k, v) of layer ``i`` as [..., heads, size] before rotation, normalised where the design has it; k and v
        are None when the layer reads another layer's.  With two maps a head's two queries (keys) lie side by side."""
        s, ls = self.spec, self.spec.layer(i)
        L = f"layers.{i}."
        qkv = ops_fn.linear(h, self.p[L + "wqkv"], self.p.get(L + "bqkv"))
        lead = h.shape[:-1]
        k = v = None
        kind = s.qk_norm_kind(i)
        if ls.kv_from is None:
            q, k, v = qkv.split([ls.q_size, ls.k_size, ls.v_size], dim=-1)
            if kind == "row":
                k = ops_fn.rms_norm(k.contiguous(), self.p[L + "k_norm"], s.norm_eps)
            k = k.reshape(*lead, ls.num_kv_heads * ls.maps, ls.head_dim)
            v = v.reshape(*lead, ls.num_kv_heads, ls.v_head_dim)
        else:
            q = qkv
        if kind == "row":
            q = ops_fn.rms_norm(q.contiguous(), self.p[L + "q_norm"], s.norm_eps)
        q = q.reshape(*lead, ls.num_heads * ls.maps, ls.head_dim)
        if kind == "head":
            q = ops_fn.rms_norm(q, self.p[L + "q_norm"], s.norm_eps)
            if k is not None:
                k = ops_fn.rms_norm(k, self.p[L + "k_norm"], s.norm_eps)
        return q, k, v

    def _latent_rows(self, i: int, h: torch.Tensor, rope):
        """Rotated queries [.., heads, head_dim + rot_dim] and the rows to be cached [.., kv_rank + rot_dim] of a latent layer."""
        s, ls = self.spec, self.spec.layer(i)
        q, c, kr = MX.latent_project(self.p, f"layers.{i}.", ls, h, s.norm_eps)
        if rope is not None:
            qn, qr = q.split([ls.head_dim, ls.rot_dim], dim=-1)
            q = torch.cat([qn, apply_rope(qr, *rope, ls.rotary_dim, s.rope_interleaved)], -1)
            kr = apply_rope(kr, *rope, ls.rotary_dim, s.rope_interleaved)
        return q, torch.cat([c, kr.squeeze(-2)], -1)

    def mixer(self, i: int, h: torch.Tensor, past: int, cache: Optional[KVCache], shared: dict, st: dict) -> torch.Tensor:
        """The first sublayer of layer ``i`` on whole sequences; ``st`` is the layer's carried state."""
        ls, L = self.spec.layer(i), f"layers.{i}."
        if ls.mixer == "wkv":
            return ops_fn.linear(MX.wkv(self.p, L, ls, h, st, self.spec.norm_eps), self.p[L + "wo"])
        if ls.mixer == "delta":
            return self._delta(i, h, st)
        a = self._attention(i, h, past, cache, shared)
        return a if ls.beside is None else self._side_by_side(i, a, self._delta(i, h, st))

    def _delta(self, i: int, h: torch.Tensor, st: dict) -> torch.Tensor:
        """Gated delta rule of layer ``i`` (its only mixer, or the one beside another) with its output projection."""
        ls, L = self.spec.layer(i), f"layers.{i}."
        if ls.beside is not None:
            ls, L = ls.beside, L + "beside."
        return ops_fn.linear(MX.delta(self.p, L, ls, h, st, self.spec.norm_eps), self.p[L + "wo"])

    def _side_by_side(self, i: int, a: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
        sa, sb = self.spec.layer(i).scales
        return (sa * _f(a) + sb * _f(b)).to(a.dtype)

    def _attend(self, i: int, q, k, v, bias):
        """q [B, Hq, T, Dk], k / v [B, Hkv, S, ...] in fp32, additive ``bias`` [T, S] or [Hq, T, S] -> [B, Hq, T, Dv]; with two
        maps per head q, k and the result have twice the heads."""
        ls = self.spec.layer(i)
        g = ls.num_heads // ls.num_kv_heads
        if ls.maps > 1:
            k = k.unflatten(1, (ls.num_kv_heads, ls.maps)).repeat_interleave(g, dim=1).flatten(1, 2)
            v = v.repeat_interleave(g * ls.maps, dim=1)
        elif g > 1:
            k, v = k.repeat_interleave(g, dim=1), v.repeat_interleave(g, dim=1)
        scale = ls.scale if ls.scale is not None else 1.0 / math.sqrt(ls.head_dim)
        if not ls.sink and ls.fixed_sink is None and not ls.softcap:
            return F.scaled_dot_product_attention(q, k, v, attn_mask=bias, scale=scale)
        sc = torch.matmul(q, k.transpose(-1, -2)) * scale
        if ls.softcap:
            sc = ls.softcap * torch.tanh(sc / ls.softcap)
        sc = sc + bias
        if ls.sink:
            sink = self.p[f"layers.{i}.sink"].to(sc).reshape(-1, 1, 1).expand(*sc.shape[:-1], 1)
        elif ls.fixed_sink is not None:
            sink = torch.full((*sc.shape[:-1], 1), ls.fixed_sink, dtype=sc.dtype, device=sc.device)
        else:
            return torch.matmul(torch.softmax(sc, dim=-1), v)
        # the sink is one more column of the softmax that has no value
        p = torch.softmax(torch.cat([sc, sink], dim=-1), dim=-1)[..., :-1]
        return torch.matmul(p, v)

    def _finish_attention(self, i: int, y: torch.Tensor, h: torch.Tensor, vrope) -> torch.Tensor:
        """y [.., T, heads, Dv] of the attention over what the layer read, h [.., T, H] -> rows for the output projection: values
        turned back, maps subtracted, output gate."""
        s, ls, L = self.spec, self.spec.layer(i), f"layers.{i}."
        if ls.maps == 2:
            y = MX.difference(ls, self.p[L + "lambdas"], _f(y), s.norm_eps)
        if vrope is not None:
            y = apply_rope(y, vrope[0], -vrope[1], ls.v_head_dim, s.rope_interleaved)
        if ls.out_gate:
            g = torch.sigmoid(_f(ops_fn.linear(h, self.p[L + "w_og"])))
            y = _f(y) * (g.unsqueeze(-1) if ls.out_gate == "head" else g.unflatten(-1, (ls.num_heads, ls.v_head_dim)))
        return y.flatten(-2).to(h.dtype)

    def _attention(self, i: int, h: torch.Tensor, past: int, cache: Optional[KVCache], shared: dict) -> torch.Tensor:
        s, ls = self.spec, self.spec.layer(i)
        L = f"layers.{i}."
        B, T, _ = h.shape
        rope = self._rope_cache(past + T, ls).get_range(past, past + T) if ls.rotary_dim > 0 else None
        vrope = self._value_rope(past + T, ls).get_range(past, past + T) if ls.value_rope else None
        if ls.mixer == "latent":
            q, rows = self._latent_rows(i, h, rope)
            rows = rows[:, None]                              # one row of width kv_rank + rot_dim for all heads
            if cache is not None:
                cache.layer(i).append(rows, rows[..., :0])
                rows, _ = cache.layer(i).get_kv()
            k, v = MX.latent_expand(self.p, L, ls, rows[:, 0])
        else:
            q, k, v = self._project_qkv(i, h)
            if rope is not None:
                q = apply_rope(q, *rope, ls.rotary_dim, s.rope_interleaved)
                if k is not None:
                    k = apply_rope(k, *rope, ls.rotary_dim, s.rope_interleaved)
            if vrope is not None and v is not None:
                v = apply_rope(v, *vrope, ls.v_head_dim, s.rope_interleaved)
        if ls.mixer == "latent":
            pass
        elif ls.kv_from is not None:
            k, v = shared[ls.kv_from]
        else:
            k, v = k.transpose(1, 2), v.transpose(1, 2)      # [B, Hkv, T, D]
            if cache is not None:
                lc = cache.layer(i)
                lc.append(k, v)
                k, v = lc.get_kv()
            shared[i] = (k, v)
        q = q.transpose(1, 2)                             # [B, Hq, T, D]
        S = k.shape[2]
        qpos = torch.arange(past, past + T, device=h.device)[:, None]
        kpos = torch.arange(S, device=h.device)[None, :]
        vis = kpos <= qpos
        if ls.window > 0:
            vis = vis & (kpos > qpos - ls.window)
        if ls.chunk > 0:
            vis = vis & (kpos // ls.chunk == qpos // ls.chunk)
        bias = torch.zeros(T, S, device=h.device, dtype=torch.float32).masked_fill(~vis, float("-inf"))
        if s.pos == "alibi":
            if self._alibi is None or self._alibi.device != h.device:
                self._alibi = alibi_slopes(s.num_heads).to(h.device)
            bias = bias[None] + self._alibi[:, None, None] * (kpos - qpos)[None].float()
        y = self._attend(i, _f(q), _f(k), _f(v), bias)
        y = self._finish_attention(i, y.transpose(1, 2), h, vrope)
        return ops_fn.linear(y, self.p[L + "wo"], self.p.get(L + "bo"))

    def _dense_mlp(self, x, w_gate_up=None, w_up=None, b_up=None, w_down=None, b_down=None, act="silu", act_p=None):
        if w_gate_up is not None:
            gu = ops_fn.linear(x, w_gate_up)
            g, u = gu.chunk(2, dim=-1)
            hdn = (ops_fn.activation(act)(_f(g)) * _f(u)).to(x.dtype)
        else:
            z = _f(ops_fn.linear(x, w_up, b_up))
            hdn = (MX.xielu(z, act_p) if act == "xielu" else ops_fn.activation(act)(z)).to(x.dtype)
        return ops_fn.linear(hdn, w_down, b_down)

    def _moe(self, i: int, x: torch.Tensor) -> torch.Tensor:
        m = self.spec.layer(i).moe
        L = f"layers.{i}."
        shape = x.shape
        x2 = x.reshape(-1, shape[-1])
        rb = self.p.get(L + "router_b")
        logits = F.linear(_f(x2), _f(self.p[L + "router"]), None if rb is None else _f(rb))
        if m.correction or m.groups > 1:
            sc = torch.softmax(logits, dim=-1)
            choice = sc + _f(self.p[L + "correction"]) if m.correction else sc
            if m.keep_groups < m.groups:
                best = choice.reshape(-1, m.groups, m.num_experts // m.groups).amax(-1).topk(m.keep_groups, dim=-1).indices
                shut = torch.ones(choice.shape[0], m.groups, dtype=torch.bool, device=x.device).scatter_(1, best, False)
                choice = choice.masked_fill(shut.repeat_interleave(m.num_experts // m.groups, dim=1), float("-inf"))
            idx = choice.topk(m.top_k, dim=-1).indices
            w = sc.gather(1, idx)
            if m.normalize_topk:
                w = w / (w.sum(-1, keepdim=True) + 1e-20)
        elif m.normalize_topk:
            v, idx = torch.topk(logits, m.top_k, dim=-1)
            w = torch.softmax(v, dim=-1)
        else:
            w, idx = torch.topk(torch.softmax(logits, dim=-1), m.top_k, dim=-1)
        out = torch.zeros(x2.shape, dtype=torch.float32, device=x.device)
        gu, dn = self.p[L + "experts_gate_up"], self.p[L + "experts_down"]
        for e in range(m.num_experts):
            tok, slot = (idx == e).nonzero(as_tuple=True)
            if tok.numel() == 0:
                continue
            if m.gated:
                y = self._dense_mlp(x2[tok], w_gate_up=gu[e], w_down=dn[e], act=m.act)
            else:
                y = self._dense_mlp(x2[tok], w_up=gu[e], w_down=dn[e], act=m.act)
            out.index_add_(0, tok, _f(y) * w[tok, slot].unsqueeze(-1))
        if m.num_shared_experts:
            w = self.p[L + "shared_gate_up"]
            y = _f(self._dense_mlp(x2, w_gate_up=w if m.gated else None, w_up=None if m.gated else w,
                                   w_down=self.p[L + "shared_down"], act=m.act))
            if m.shared_gate:
                y = y * torch.sigmoid(F.linear(_f(x2), _f(self.p[L + "shared_sg"])))
            out = out + y
        return out.to(x.dtype).reshape(shape)

    def _mlp(self, i: int, x: torch.Tensor) -> torch.Tensor:
        s = self.spec
        L = f"layers.{i}."
        y = None
        if L + "w_down" in self.p:
            y = self._dense_mlp(x, self.p.get(L + "w_gate_up"), self.p.get(L + "w_up"), self.p.get(L + "b_up"),
                                self.p[L + "w_down"], self.p.get(L + "b_down"), s.act, self.p.get(L + "act"))
        if s.layer_is_moe(i):
            mo = self._moe(i, x)
            y = mo if y is None else y + mo
        return y

    def block(self, i: int, x: torch.Tensor, attention, conv=None) -> torch.Tensor:
        """One layer around ``attention(h)``: where the norms sit and how the sublayers join the residual stream.
        ``conv(h, name)`` puts the input convolution of that name (or the token shift) in front of a sublayer."""
        s = self.spec
        L = f"layers.{i}."
        rs = s.residual_scale
        if s.post_ln:
            x = self._norm(x + attention(x) * rs, L + "ln1")
            return self._norm(x + self._mlp(i, x) * rs, L + "ln2")
        if s.norm_placement == "output":
            x = x + self._norm(attention(x), L + "ln1") * rs
            return x if s.layer(i).mlp is None else x + self._norm(self._mlp(i, x), L + "ln2") * rs
        if s.norm_placement == "both":
            h = self._norm(x, L + "ln1")
            x = x + self._norm(attention(conv(h, "conv1") if s.input_conv else h), L + "ln1b") * rs
            if s.layer(i).mlp is None:
                return x
            h = self._norm(x, L + "ln2")
            return x + self._norm(self._mlp(i, conv(h, "conv2") if s.input_conv else h), L + "ln2b") * rs
        h = self._norm(x, L + "ln1")
        a = attention(conv(h, "shift") if s.token_shift else h)
        if s.parallel_residual:
            m_in = h if s.parallel_shared_norm else self._norm(x, L + "ln2")
            return x + (a + self._mlp(i, m_in)) * rs
        x = x + a * rs
        return x if s.layer(i).mlp is None else x + self._mlp(i, self._norm(x, L + "ln2")) * rs

    def after_layer(self, i: int, x: torch.Tensor, streams: List[torch.Tensor]) -> torch.Tensor:
        """What goes on behind layer ``i``, whose result is ``x``; ``streams`` collects the results."""
        if not self.spec.depth_average:
            return x
        streams.append(x)
        return sum(w * t.to(w.dtype) for w, t in zip(_f(self.p[f"layers.{i}.dwa"]), streams)).to(x.dtype)

    def hidden_states(self, input_ids: torch.Tensor, cache: Optional[KVCache] = None,
                      inputs_embeds: Optional[torch.Tensor] = None) -> torch.Tensor:
        s = self.spec
        if input_ids is not None and input_ids.dim() != 2:
            raise InvalidInput("input_ids must be [batch, seq]")
        past = cache.seq_len() if cache is not None else 0
        if inputs_embeds is None:
            if int(input_ids.max()) >= s.vocab_size or int(input_ids.min()) < 0:
                raise InvalidInput("token id out of range")
            x = ops_fn.embedding(input_ids.to(self.device), self.p["embed"])
            if s.embed_proj_dim:
                x = ops_fn.linear(x, self.p["project_in"])
            if s.embed_scale != 1.0:
                x = (_f(x) * s.embed_scale).to(x.dtype)
        else:
            x = inputs_embeds
        T = x.shape[1]
        if s.pos == "learned":
            pos = torch.arange(past, past + T, device=self.device) + s.learned_pos_offset
            x = x + self.p["pos_embed"][pos][None]
        if s.embed_norm:
            x = ops_fn.layer_norm(x, self.p["embed_norm.w"], self.p["embed_norm.b"], s.norm_eps)
        streams = [x]                         # for the depth average
        shared: dict = {}                     # keys and values of this call's layers, for those that read an earlier one's
        for i in range(s.num_layers):
            st: dict = cache.layer(i).state if cache is not None else {}
            x = self.block(i, x, lambda h, i=i, st=st: self.mixer(i, h, past, cache, shared, st),
                           lambda h, n, i=i, st=st: MX.before_sublayer(h, self.p[f"layers.{i}.{n}"], st, n))
            x = self.after_layer(i, x, streams)
        if cache is not None:
            cache.set_seq_len(past + T)
        if s.final_norm:
            x = self._norm(x, "final_norm", layer_level=False)
        return x

    def lm_logits(self, x: torch.Tensor) -> torch.Tensor:
        s = self.spec
        if s.embed_proj_dim:
            x = ops_fn.linear(x, self.p["project_out"])
        w = self.p["embed"] if s.tie_embeddings else self.p["lm_head"]
        y = ops_fn.linear(x, w, self.p.get("lm_head_bias"))
        if s.logit_scale != 1.0:
            y = (_f(y) * s.logit_scale).to(y.dtype)
        return y

    def forward(self, inputs: ModelInputs) -> ModelOutputs:
        if inputs.input_ids is None:
            raise InvalidInput(f"{type(self).__name__} takes text inputs")
        x = self.hidden_states(inputs.input_ids)
        return ModelOutputs.from_logits(self.lm_logits(x), hidden_states=x)

    def new_cache(self, max_seq_len: Optional[int] = None) -> KVCache:
        return KVCache(self.spec.num_layers, max_seq_len or max(2048, min(self.spec.max_position_embeddings, 8192)))

    def forward_with_cache(self, input_ids: torch.Tensor, cache: Optional[KVCache] = None) -> torch.Tensor:
        """Logits ``[B, T_new, V]`` for the new tokens only; keys / values are appended to ``cache``."""
        if input_ids.dim() == 1:
            input_ids = input_ids[None]
        return self.lm_logits(self.hidden_states(input_ids, cache))

    def generate_with_cache(self, prompt: str, config=None) -> str:
        return self.generate(prompt, config)
