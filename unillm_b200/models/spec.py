"""``DecoderSpec``: one parametric description of a decoder-only transformer block stack, and
``KeyScheme``: how a family names its tensors on disk.

Thirty-odd of the reference's 47 model files (``crates/runtime/src/models_v2/*.rs``) are the same
pre-norm decoder with small variations; instead of one copy of the code per family, each family
supplies a config -> ``DecoderSpec`` function and a ``KeyScheme``.  The variation axes are exactly the
ones the reference's files differ in: norm kind and bias, rotary variant (full / partial / theta /
linear or Llama-3 scaling / interleaved), ALiBi, learned positions, sliding window, QKV packing,
residual topology (sequential / parallel, shared or separate norms, post-LN), MLP kind (gated /
plain, activation), biases, embedding / logit / residual / attention scalings, tied embeddings, and
mixture-of-experts (experts, top-k, shared experts, dense-parallel MLP, leading dense layers).

Designs whose layers differ from one another (head counts, head sizes, windows, rotations, feed-forward sizes, layers
without a feed-forward, layers that read another layer's keys and values, layers with another mixer than attention) list
a ``LayerSpec`` per layer; ``DecoderSpec.layer(i)`` answers for every spec, so the loaders and runners ask it instead of
the uniform fields.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional, Tuple


@dataclass
class MoESpec:
    num_experts: int = 8
    top_k: int = 2
    intermediate_size: int = 14336       # per-expert FFN width
    normalize_topk: bool = True          # softmax over the k selected logits (Mixtral); else softmax over all E
    num_shared_experts: int = 0          # always-on experts (DeepSeek-MoE); width = num_shared * intermediate_size
    dense_parallel: bool = False         # Arctic: dense MLP output + MoE output
    first_k_dense: int = 0               # leading layers that use the dense MLP instead of MoE
    act: str = "silu"
    gated: bool = True                   # False: down(act(up x)) experts (and shared experts)
    router_bias: bool = False            # logits = W x + b
    shared_intermediate_size: Optional[int] = None   # width of the always-on expert; None: num_shared * intermediate_size
    correction: bool = False             # experts are chosen by softmax(logits) + correction, weighted without it
    groups: int = 1                      # equal groups of neighbouring experts; only those of the ``keep_groups`` groups with
    keep_groups: int = 1                 # the largest score in them can be chosen
    shared_gate: bool = False            # the always-on expert's output is multiplied by sigmoid(w . x), one number per token

    @property
    def shared_width(self) -> int:
        if self.shared_intermediate_size is not None:
            return self.shared_intermediate_size
        return self.num_shared_experts * self.intermediate_size


@dataclass(frozen=True)
class LayerSpec:
    """What one layer's sublayers look like.  ``kv_from``: the layer has no key / value projections and attends to the
    cached keys and values of that earlier layer (its own queries, window, scale and sinks).  ``mlp``: "dense", "moe" or
    None (no feed-forward).

    ``mixer``: "attention"; "latent" (multi-head latent attention: queries through a normalised latent of ``q_rank``, keys
    and values of all heads from one cached, normalised latent of ``kv_rank`` and one cached rotated key part of
    ``rot_dim`` shared by the heads; ``head_dim`` is the unrotated key size); "wkv" (RWKV-6 style recurrence with a
    ``head_dim`` x ``head_dim`` state per head, five token-shift mixes and a low-rank decay of ``decay_rank``); or "delta"
    (gated delta rule with a ``head_dim`` x ``v_head_dim`` state per head, queries and keys of ``num_kv_heads`` heads, and
    causal convolutions of ``conv_taps`` taps on queries, keys and values; ``decay="channel"``: every row of the state decays at
    its own rate, through a low-rank map of ``decay_rank``; ``low_rank_gate``: the output gate is a product of rank ``gate_rank``).

    ``maps`` = 2: differential attention, two softmax maps per head over the same values (query and key rows lie head by head as
    [map 1, map 2]); o = (a1 - lambda a2) / rms * (1 - ``diff``) with one learned lambda per layer.

    ``beside``: a second mixer that reads the same input; the first one's output times ``scales[0]`` and the second one's
    times ``scales[1]`` are added."""

    num_heads: int
    num_kv_heads: int
    head_dim: int                        # query / key size
    v_head_dim: int
    window: int = 0                      # keys p - window + 1 .. p; 0 = all
    chunk: int = 0                       # keys of the query's own chunk of this many positions, counted from 0; 0 = all
    scale: Optional[float] = None        # None = 1/sqrt(head_dim)
    rotary_dim: int = 0
    rope_theta: float = 10000.0
    rope_llama3: Optional[Tuple[float, float, float, float]] = None
    rope_yarn: Optional[Tuple[float, float, float, float]] = None   # (factor, original_ctx, fast turns, slow turns)
    kv_from: Optional[int] = None
    rope_linear: float = 1.0             # frequencies are divided by this
    sink: bool = False                   # one learned logit per head in the softmax denominator
    fixed_sink: Optional[float] = None   # a constant logit there instead
    softcap: float = 0.0                 # scores become softcap * tanh(score / softcap); 0 = as they are
    qkv_bias: Optional[bool] = None      # None = as the model says
    qk_norm: Optional[str] = None        # "head", "row" (over the whole projection), "" = none; None = as the model says
    mlp: Optional[str] = "dense"
    moe: Optional[MoESpec] = None
    mixer: str = "attention"
    q_rank: int = 0
    kv_rank: int = 0
    rot_dim: int = 0
    decay_rank: int = 0
    intermediate_size: Optional[int] = None   # dense feed-forward width (None: the model's)
    conv_taps: int = 0
    decay: str = "head"                  # delta: one decay per "head", or one per "channel" of its keys
    low_rank_gate: bool = False
    gate_rank: int = 0
    gate_act: str = "silu"               # delta: activation of the output gate
    value_rope: bool = False             # values turn by their position over all their dimensions, outputs turn back by the query's
    out_gate: str = ""                   # the attention's output times sigmoid(W h): "head" = one number per head, "element", "" = none
    maps: int = 1
    diff: float = 0.0
    beside: Optional["LayerSpec"] = None
    scales: Tuple[float, float] = (1.0, 1.0)

    @property
    def has_kv(self) -> bool:
        """The layer owns cache rows."""
        return self.mixer not in ("wkv", "delta") and self.kv_from is None

    @property
    def mixers(self) -> Tuple["LayerSpec", ...]:
        return (self,) if self.beside is None else (self, self.beside)

    @property
    def conv_rows(self) -> int:
        """Channels of a delta mixer's convolutions: [Q; K; V]."""
        return 2 * self.k_size + self.o_size

    @property
    def cache_row(self) -> int:
        """Cache elements per token of a layer that owns some: keys and values, or the latent and its rotated part."""
        return self.kv_rank + self.rot_dim if self.mixer == "latent" else self.k_size + self.v_size

    @property
    def q_size(self) -> int:
        return self.num_heads * self.maps * (self.head_dim + self.rot_dim)

    @property
    def k_size(self) -> int:
        return self.num_kv_heads * self.maps * self.head_dim

    @property
    def v_size(self) -> int:
        return self.num_kv_heads * self.v_head_dim

    @property
    def o_size(self) -> int:
        return self.num_heads * self.v_head_dim

    @property
    def gate_size(self) -> int:
        """Rows of the attention's output gate."""
        return {"": 0, "head": self.num_heads, "element": self.o_size}[self.out_gate]

    @property
    def qkv_size(self) -> int:
        """Rows of the fused projection: [Q; K; V], or Q alone for a layer that reads another layer's keys."""
        return self.q_size if self.kv_from is not None else self.q_size + self.k_size + self.v_size


@dataclass
class DecoderSpec:
    vocab_size: int = 32000
    hidden_size: int = 4096
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 32
    head_dim: int = 128
    intermediate_size: int = 11008
    max_position_embeddings: int = 2048
    # norms
    norm: str = "rms"                    # "rms" | "layer" | "tanh" (Dynamic Tanh: tanh(alpha x) w + b, no statistics)
    norm_eps: float = 1e-6
    norm_bias: bool = False
    norm_weight_offset_one: bool = False  # Gemma: y * (1 + w)
    final_norm: bool = True
    embed_norm: bool = False             # BLOOM word_embeddings_layernorm
    qk_norm: bool = False
    # positions
    pos: str = "rope"                    # "rope" | "learned" | "alibi" | "none"
    rope_theta: float = 10000.0
    rotary_dim: Optional[int] = None     # None = head_dim
    rope_interleaved: bool = False       # GPT-J style adjacent pairs
    rope_pos_scale: float = 1.0          # linear scaling: position * scale
    rope_llama3: Optional[Tuple[float, float, float, float]] = None  # (factor, low, high, original_ctx)
    learned_pos_offset: int = 0          # OPT stores positions shifted by 2
    window: int = 0                      # sliding-window size, 0 = full attention
    # projections
    qkv_bias: bool = False
    o_bias: bool = False
    mlp_bias: bool = False
    lm_head_bias: bool = False
    mlp: str = "gated"                   # "gated" (act(gate) * up) | "plain" (act(fc1))
    act: str = "silu"
    # topology
    parallel_residual: bool = False      # x + attn(n1(x)) + mlp(n2(x))
    parallel_shared_norm: bool = False   # ... with mlp reading n1(x) (GPT-J, Phi, Falcon-7B)
    post_ln: bool = False                # OPT-350m style: norm after the residual add
    norm_placement: str = "input"        # "input": x + f(norm(x)) | "output": x + norm(f(x)), sublayers read x itself |
    #                                      "both": x + norm_b(f(norm(x)))
    input_conv: int = 0                  # taps of the causal depthwise convolution added to what every sublayer reads (0: none)
    token_shift: bool = False            # a mixer reads h + (h of the previous token - h) * shift, per channel
    depth_average: bool = False          # what leaves layer i is a learned weighted sum of the embedding and all layers' results
    residual_fp32: bool = False          # the residual stream is kept in 32 bits between the layers
    layers: Optional[Tuple[LayerSpec, ...]] = None   # per-layer description; None: all layers as the fields above say
    # scalings
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    residual_scale: float = 1.0
    attn_scale: Optional[float] = None   # None = 1/sqrt(head_dim)
    tie_embeddings: bool = False
    embed_proj_dim: Optional[int] = None  # OPT word_embed_proj_dim != hidden: project_in / project_out
    moe: Optional[MoESpec] = None
    # behaviour of the reference implementation that differs from the published architecture;
    # applied only when a model is built with reference_quirks=True
    ref_ln_star: bool = False            # uses mean-subtracting layer_norm(x, w, None) where the family has RMSNorm
    ref_layer_eps: Optional[float] = None  # eps hard-coded inside layers (llama.rs:633,642 uses 1e-6)
    initializer_range: float = 0.02

    @property
    def q_size(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    @property
    def rd(self) -> int:
        return self.head_dim if self.rotary_dim is None else self.rotary_dim

    def layer(self, i: int) -> LayerSpec:
        if self.layers is not None:
            return self.layers[i]
        return LayerSpec(num_heads=self.num_heads, num_kv_heads=self.num_kv_heads, head_dim=self.head_dim,
                         v_head_dim=self.head_dim, window=self.window, scale=self.attn_scale,
                         rotary_dim=self.rd if self.pos == "rope" else 0, rope_theta=self.rope_theta,
                         rope_llama3=self.rope_llama3, mlp="moe" if self.layer_is_moe(i) else "dense",
                         moe=self.moe if self.layer_is_moe(i) else None)

    def layer_is_moe(self, i: int) -> bool:
        if self.layers is not None:
            return self.layers[i].mlp == "moe"
        return self.moe is not None and i >= self.moe.first_k_dense

    @property
    def kv_elements_per_token(self) -> int:
        """Cache elements that one token takes over all layers that own keys and values."""
        return sum(self.layer(i).cache_row for i in self.kv_layers)

    @property
    def kv_layers(self) -> Tuple[int, ...]:
        """Layers that own cache rows (the others read one of these, or have no keys)."""
        return tuple(i for i in range(self.num_layers) if self.layer(i).has_kv)

    def qk_norm_kind(self, i: int) -> str:
        kind = self.layer(i).qk_norm
        return ("head" if self.qk_norm else "") if kind is None else kind

    def has_qkv_bias(self, i: int) -> bool:
        b = self.layer(i).qkv_bias
        return self.qkv_bias if b is None else b

    def layer_intermediate(self, i: int) -> int:
        n = self.layer(i).intermediate_size
        return self.intermediate_size if n is None else n

    @property
    def state_elements(self) -> int:
        """fp32 elements of state that one sequence carries from token to token besides cache rows: the last inputs of the
        convolutions, the previous token's input of the wkv layers and of token shifts, and the recurrent state of the wkv and delta mixers."""
        n = 0
        for i in range(self.num_layers):
            ls = self.layer(i)
            if self.input_conv:
                n += (self.input_conv - 1) * self.hidden_size * (2 if ls.mlp is not None else 1)
            if self.token_shift:
                n += self.hidden_size
            if ls.mixer == "wkv":
                n += self.hidden_size + ls.num_heads * ls.head_dim * ls.head_dim
            for mx in ls.mixers:
                if mx.mixer == "delta":
                    n += (mx.conv_taps - 1) * mx.conv_rows + mx.num_heads * mx.head_dim * mx.v_head_dim
        return n

    @property
    def has_state(self) -> bool:
        """Sequences carry state that cannot be rebuilt from cached blocks (so prompts cannot skip a cached prefix)."""
        return self.state_elements > 0


@dataclass
class KeyScheme:
    """Tensor names of one family.  Every entry is a tuple of aliases, tried in order; layer-level
    names are relative to ``layer.format(i=...)``.  ``weight_suffix`` / ``bias_suffix`` are appended (sinks have none)."""

    embed: Tuple[str, ...] = ("model.embed_tokens",)
    pos_embed: Tuple[str, ...] = ()
    embed_norm: Tuple[str, ...] = ()
    project_in: Tuple[str, ...] = ()
    project_out: Tuple[str, ...] = ()
    layer: Tuple[str, ...] = ("model.layers.{i}.",)
    ln1: Tuple[str, ...] = ("input_layernorm",)
    ln2: Tuple[str, ...] = ("post_attention_layernorm",)
    q: Tuple[str, ...] = ("self_attn.q_proj",)
    k: Tuple[str, ...] = ("self_attn.k_proj",)
    v: Tuple[str, ...] = ("self_attn.v_proj",)
    qkv: Tuple[str, ...] = ()
    qkv_layout: str = "concat"           # "concat" [Q;K;V] | "per_head" [h][q,k,v] | "grouped" [kv group][G q, k, v]
    q_norm: Tuple[str, ...] = ("self_attn.q_norm",)
    k_norm: Tuple[str, ...] = ("self_attn.k_norm",)
    o: Tuple[str, ...] = ("self_attn.o_proj",)
    gate: Tuple[str, ...] = ("mlp.gate_proj",)
    up: Tuple[str, ...] = ("mlp.up_proj",)
    down: Tuple[str, ...] = ("mlp.down_proj",)
    gate_up: Tuple[str, ...] = ()        # packed [gate; up]
    final_norm: Tuple[str, ...] = ("model.norm",)
    lm_head: Tuple[str, ...] = ("lm_head",)
    sink: Tuple[str, ...] = ()           # per-head softmax sinks
    ln1b: Tuple[str, ...] = ()           # norms on the sublayers' outputs where the inputs are normed as well
    ln2b: Tuple[str, ...] = ()
    conv1: Tuple[str, ...] = ()          # input convolutions
    conv2: Tuple[str, ...] = ()
    act: Tuple[str, ...] = ()            # learned numbers of the activation
    shift: Tuple[str, ...] = ()          # token shift
    depth_average: Tuple[str, ...] = ()  # weights of the depth average
    out_gate: Tuple[str, ...] = ()       # output gate of an attention
    lambdas: Tuple[str, ...] = ()        # the four vectors of a differential attention's lambda: q and k of map 1, of map 2
    alpha_suffix: str = ".alpha"         # slope of a Dynamic Tanh, behind the norm's name
    mixers: Optional[dict] = None        # {mixer: {parameter: names, several = stacked or concatenated}}, see mixers.mixer_shapes
    sides: Optional[Tuple[str, str, str]] = None   # prefix of a mixer's names; what replaces it for the first and the second
    #                                                of two mixers side by side
    weight_suffix: str = ".weight"
    bias_suffix: str = ".bias"
    transposed: bool = False             # GPT-2 Conv1D stores [in, out]
    router: Tuple[str, ...] = ("block_sparse_moe.gate",)
    correction: Tuple[str, ...] = ()
    shared_sg: Tuple[str, ...] = ()      # gate of the always-on expert
    expert: Tuple[str, ...] = ("block_sparse_moe.experts.{e}.",)
    e_gate: Tuple[str, ...] = ("w1",)
    e_up: Tuple[str, ...] = ("w3",)
    e_down: Tuple[str, ...] = ("w2",)
    shared_gate: Tuple[str, ...] = ("mlp.shared_experts.gate_proj",)
    shared_up: Tuple[str, ...] = ("mlp.shared_experts.up_proj",)
    shared_down: Tuple[str, ...] = ("mlp.shared_experts.down_proj",)
