"""Torch-tensor front end of the sm_100a kernel library.

Every function launches on the current CUDA stream of the tensors' device and returns torch
tensors; none of them synchronises.  Arguments are checked on the host (dtype, contiguity,
alignment) so that a bad call raises in Python instead of faulting on the device.  The kernels
record device-side problems (timeouts of bounded waits, out-of-range block-table entries) in a
per-device error word that :func:`check_device_errors` reads.
"""
from __future__ import annotations

import ctypes as C
import math
from typing import Optional, Sequence

import torch

from . import _native as N
from . import _native as N_

_err_words: dict[int, torch.Tensor] = {}


def _stream(t: torch.Tensor) -> int:
    return torch.cuda.current_stream(t.device).cuda_stream


def err_word(device) -> torch.Tensor:
    dev = torch.device(device)
    idx = dev.index if dev.index is not None else torch.cuda.current_device()
    w = _err_words.get(idx)
    if w is None:
        w = torch.zeros(2, dtype=torch.int32, device=f"cuda:{idx}")
        _err_words[idx] = w
    return w


def check_device_errors(device=None, reset: bool = True) -> None:
    """Synchronises and raises if any kernel recorded an error since the last check."""
    devs = [torch.device(device)] if device is not None else [torch.device(f"cuda:{i}") for i in _err_words]
    for d in devs:
        w = err_word(d)
        code, detail = w.tolist()
        if code != 0:
            if reset:
                w.zero_()
                gemm_streamk_reset(d)
            names = {1: "mbarrier wait timed out", 2: "flag wait timed out (peer or producer missing)",
                     3: "index out of range", 4: "bad argument"}
            raise RuntimeError(f"device error {code} ({names.get(code, '?')}), detail {detail} on {d}")


def gemm_streamk_reset(device=None) -> None:
    """Lowers the flags of the GEMM's stream-K workspace (after a step that reported a timed-out wait)."""
    with torch.cuda.device(torch.device(device) if device is not None else torch.cuda.current_device()):
        N_.cuda_lib().ub_gemm_streamk_reset(C.c_void_p(torch.cuda.current_stream().cuda_stream))


def _p(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


def _bf16c(t: torch.Tensor, name: str) -> None:
    if t.dtype != torch.bfloat16:
        raise TypeError(f"{name} must be bfloat16, got {t.dtype}")
    if not t.is_cuda:
        raise ValueError(f"{name} must be a CUDA tensor")


def _elem(name: str, t: torch.Tensor, *others: Optional[torch.Tensor]) -> bool:
    """Checks that ``t`` and the given others are CUDA tensors of one element type, bf16 or fp32; True for fp32."""
    if t.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"{name} must be bfloat16 or float32, got {t.dtype}")
    for o in (t, *others):
        if o is None:
            continue
        if o.dtype != t.dtype:
            raise TypeError(f"{name}: operands of different types ({t.dtype}, {o.dtype})")
        if not o.is_cuda:
            raise ValueError(f"{name}: operands must be CUDA tensors")
    return t.dtype == torch.float32


# ---------------------------------------------------------------------------------------------
# GEMM
# ---------------------------------------------------------------------------------------------
def gemm_tn(x: torch.Tensor, w: torch.Tensor, *, bias: Optional[torch.Tensor] = None,
            residual: Optional[torch.Tensor] = None, act: Optional[str] = None, out: Optional[torch.Tensor] = None,
            out_dtype: torch.dtype = torch.bfloat16, out_scale: float = 1.0, tile_tokens: int = 0, splits: int = 0,
            dual_rows: int = 0, rs: Optional[dict] = None, ag: Optional[dict] = None,
            grouped: Optional[dict] = None, cta_pair: int = 0, pair_splits: int = 0,
            act_params: Optional[tuple] = None) -> torch.Tensor:
    """``out[M, N] = act(x[M, K] @ w[N, K]^T * out_scale + bias) + residual`` on tcgen05 tensor cores.

    ``dual_rows = I`` switches to the gated form: ``w`` is ``[2*I, K]`` with gate rows first and the
    result is ``act(x @ w[:I]^T) * (x @ w[I:]^T)`` of shape ``[M, I]``.
    With fp32 operands everything runs in 32-bit arithmetic and the result is fp32.
    ``act_params``: the two coefficients of ``act="xielu"``.
    ``rs`` / ``ag`` carry the peer pointers for the fused reduce-scatter / all-gather variants (see
    :mod:`unillm_b200.dist.fused`).
    """
    f32 = _elem("gemm_tn", x, w, bias, residual)      # fp32 operands: 32-bit arithmetic (ub_gemm_f32)
    if x.dim() != 2 or w.dim() != 2:
        raise ValueError("gemm_tn takes 2-D operands")
    if f32:
        if rs is not None or ag is not None or (out is not None and out.dtype != torch.float32):
            raise ValueError("gemm_tn in fp32: no fused collectives, fp32 output")
        out_dtype = torch.float32
    if x.stride(1) != 1 or w.stride(1) != 1:
        raise ValueError("operands must be K-contiguous")
    M, K = x.shape
    if w.shape[1] != K:
        raise ValueError(f"K mismatch: x {tuple(x.shape)} vs w {tuple(w.shape)}")
    dual = dual_rows > 0
    Nn = dual_rows if dual else w.shape[0]
    if dual and w.shape[0] < 2 * dual_rows:
        raise ValueError("dual GEMM needs w with 2*I rows")
    if out is None:
        out = torch.empty((M, Nn), dtype=out_dtype, device=x.device)
    if out.stride(-1) != 1:
        raise ValueError("out must be row-major")
    a = N.UbGemmArgs()
    a.x, a.w, a.out = x.data_ptr(), w.data_ptr(), out.data_ptr()
    a.bias = _p(bias)
    a.residual = _p(residual)
    a.err = err_word(x.device).data_ptr()
    a.M, a.N, a.K = M, Nn, K
    a.ldx, a.ldw, a.ldo = x.stride(0), w.stride(0), out.stride(0)
    a.ldr = residual.stride(0) if residual is not None else 0
    a.act = N.ACT[act]
    if act_params is not None:
        a.act_a, a.act_b = act_params
    a.dual = 1 if dual else 0
    a.up_row_off = dual_rows
    a.w_rows_total = w.shape[0]
    a.out_f32 = 1 if out.dtype == torch.float32 else 0
    a.out_scale = out_scale
    a.tile_tokens = tile_tokens
    a.splits = splits
    a.cta_pair = cta_pair
    a.pair_splits = pair_splits
    if rs is not None:
        a.rs_world, a.rs_rank, a.rs_rows_per_rank = rs["world"], rs["rank"], rs["rows_per_rank"]
        for i in range(rs["world"]):
            a.rs_peer_out[i] = rs["peer_out"][i]
            a.rs_peer_flag[i] = rs["peer_flag"][i]
        a.rs_local_count = rs["local_count"]
    if ag is not None:
        a.ag_world, a.ag_rows_per_rank = ag["world"], ag["rows_per_rank"]
        a.ag_flags, a.ag_signals_per_use = ag["flags"], ag["signals_per_use"]
    if grouped is not None:
        a.grp_tiles, a.grp_max_tiles, a.grp_w_rows = grouped["tiles"], grouped["max_tiles"], grouped["w_rows"]
        a.tile_tokens = grouped["tile_tokens"]
    if f32:
        N.check(N.cuda_lib().ub_gemm_f32(C.byref(a), _stream(x)), "ub_gemm_f32")
    else:
        N.check(N.cuda_lib().ub_gemm_tn(C.byref(a), _stream(x)), "ub_gemm_tn")
    return out


def gemm_num_ctas(M: int, N: int, K: int, dual: bool = False, tile_tokens: int = 0, splits: int = 0, cta_pair: int = 0) -> int:
    """CTAs that ``gemm_tn`` launches for this problem (each signals every peer once in reduce-scatter mode)."""
    a = N_.UbGemmArgs()
    a.M, a.N, a.K, a.dual, a.tile_tokens, a.splits, a.cta_pair = M, N, K, int(dual), tile_tokens, splits, cta_pair
    return N_.cuda_lib().ub_gemm_num_ctas(C.byref(a))


def wait_flags(flags_ptr: int, n: int, value: int, device) -> None:
    """Enqueue a one-block kernel that waits (bounded) until n consecutive u32 counters reach ``value``."""
    lib = N_.cuda_lib()
    lib.ub_wait_flags.restype = C.c_int
    lib.ub_wait_flags.argtypes = [N_.vp, N_.i32, N_.u32, N_.vp, N_.vp]
    N_.check(lib.ub_wait_flags(flags_ptr, n, value, err_word(device).data_ptr(),
                               torch.cuda.current_stream(device).cuda_stream), "ub_wait_flags")


def linear(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, **kw) -> torch.Tensor:
    """``x[..., K] @ w[N, K]^T`` for any leading shape."""
    lead = x.shape[:-1]
    y = gemm_tn(x.reshape(-1, x.shape[-1]), w, bias=bias, **kw)
    return y.reshape(*lead, y.shape[-1])


# ---------------------------------------------------------------------------------------------
# Norm
# ---------------------------------------------------------------------------------------------
def norm(x: torch.Tensor, weight: Optional[torch.Tensor], *, bias: Optional[torch.Tensor] = None,
         residual: Optional[torch.Tensor] = None, eps: float = 1e-5, kind: str = "rms",
         weight_offset_one: bool = False, want_residual_out: bool = False,
         out: Optional[torch.Tensor] = None, residual_out: Optional[torch.Tensor] = None,
         rs: Optional[dict] = None, ag: Optional[dict] = None, T: Optional[int] = None,
         reset: Optional[tuple] = None, no_out: bool = False, x_ptr: Optional[int] = None):
    """RMSNorm / LayerNorm over the last dim, with optional fused ``x + residual``.

    Returns ``y`` or ``(y, h)`` when the residual stream ``h = x + residual`` is requested.
    """
    _bf16c(x, "x")
    H = x.shape[-1]
    if T is None:
        T = x.numel() // H
    if not x.is_contiguous():
        x = x.contiguous()
    if out is None and not no_out:
        out = torch.empty((T, H), dtype=torch.bfloat16, device=x.device)
    if want_residual_out and residual_out is None:
        residual_out = torch.empty((T, H), dtype=torch.bfloat16, device=x.device)
    a = N.UbNormArgs()
    a.x, a.residual, a.weight, a.bias = (x.data_ptr() if x_ptr is None else x_ptr), _p(residual), _p(weight), _p(bias)
    a.out, a.residual_out = _p(out), _p(residual_out)
    a.err = err_word(x.device).data_ptr()
    a.T, a.H, a.eps = T, H, eps
    a.kind = 0 if kind == "rms" else 1
    a.weight_offset_one = 1 if weight_offset_one else 0
    if rs is not None:
        a.rs_world, a.rs_flag, a.rs_signals_per_use = rs["world"], rs["flag"], rs["signals_per_use"]
        if rs.get("multimem_x"):
            a.x, a.rs_multimem = rs["multimem_x"], 1       # multicast address of this rank's rows of the partial buffer
    if reset is not None:
        a.reset_flags, a.reset_count = reset
    if ag is not None:
        a.ag_world, a.ag_rank = ag["world"], ag["rank"]
        for i in range(ag["world"]):
            a.ag_peer_out[i] = ag["peer_out"][i]
            a.ag_peer_flag[i] = ag["peer_flag"][i]
        a.ag_local_count = ag["local_count"]
        a.ag_mc_out = ag.get("mc_out") or None
    N.check(N.cuda_lib().ub_norm(C.byref(a), _stream(x)), "ub_norm")
    if residual_out is not None:
        return out, residual_out
    return out


# ---------------------------------------------------------------------------------------------
# Norms around a 32-bit residual stream
# ---------------------------------------------------------------------------------------------
def _resid_args(what: str, x: torch.Tensor, weight, bias, out, H: int, eps: float, kind: str, offset_one: bool = False):
    f32 = _elem(what, weight, bias, out)
    if x.dtype != torch.float32 or x.dim() != 2 or not x.is_contiguous() or out.shape[1:] != x.shape[1:]:
        raise ValueError(f"{what}: the residual stream is a contiguous fp32 [T, width] tensor, out has its rows' size")
    if not out.is_contiguous() or weight.numel() != x.shape[1] or (bias is not None and bias.numel() != x.shape[1]):
        raise ValueError(f"{what}: weights must cover the (padded) row")
    a = N.UbResidualNormArgs()
    a.x, a.out, a.weight, a.bias = x.data_ptr(), out.data_ptr(), weight.data_ptr(), _p(bias)
    a.err = err_word(x.device).data_ptr()
    a.T, a.H, a.Hp, a.x_rows = out.shape[0], H, x.shape[1], x.shape[0]
    a.kind, a.f32, a.eps = (0 if kind == "rms" else 1), int(f32), eps
    a.w_off = 1.0 if offset_one else 0.0
    return a


def residual_norm(x: torch.Tensor, y: Optional[torch.Tensor], weight: torch.Tensor, bias: Optional[torch.Tensor] = None, *,
                  eps: float, kind: str = "rms", width: Optional[int] = None, out: Optional[torch.Tensor] = None,
                  experts: Optional[torch.Tensor] = None, routing: Optional["MoeRouting"] = None,
                  offset_one: bool = False) -> torch.Tensor:
    """``x += norm(y)`` on the fp32 residual stream ``x`` (in place); returns the new rows in the type of ``weight``.

    ``experts`` / ``routing``: the rows to be normalised are ``y + sum_k w[t, k] * experts[row_slot[t, k]]`` (``y`` may then
    be None).  ``width``: real row size when rows are zero-padded to a multiple of 8.  ``offset_one``: norm weights are
    stored around zero."""
    if out is None:
        out = torch.empty(x.shape, dtype=weight.dtype, device=x.device)
    a = _resid_args("residual_norm", x, weight, bias, out, width or x.shape[1], eps, kind, offset_one)
    for t in (y, experts):
        if t is not None and (t.dtype != weight.dtype or t.shape[1] != x.shape[1] or not t.is_contiguous()):
            raise ValueError("residual_norm: sublayer rows must be contiguous, of the weights' type and the stream's width")
    if y is not None and y.shape[0] != x.shape[0]:
        raise ValueError("residual_norm: one sublayer row per token")
    a.y = _p(y)
    if experts is not None:
        if routing.T != x.shape[0]:
            raise ValueError("residual_norm: the routing is of another step")
        a.yx, a.row_slot, a.topk_w = experts.data_ptr(), routing.row_slot.data_ptr(), routing.topk_w.data_ptr()
        a.K, a.slots = routing.K, experts.shape[0]
    N.check(N.cuda_lib().ub_residual_norm(C.byref(a), _stream(x)), "ub_residual_norm")
    return out


def row_norm(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None, *, eps: float, kind: str = "rms",
             rows: Optional[torch.Tensor] = None, width: Optional[int] = None, offset_one: bool = False) -> torch.Tensor:
    """``norm(x[rows])`` of an fp32 residual stream (all rows when ``rows`` is None) in the type of ``weight``."""
    if rows is not None and rows.dtype != torch.int32:
        raise TypeError("rows must be int32")
    n = x.shape[0] if rows is None else rows.numel()
    out = torch.empty(n, x.shape[1], dtype=weight.dtype, device=x.device)
    a = _resid_args("row_norm", x, weight, bias, out, width or x.shape[1], eps, kind, offset_one)
    a.rows = _p(rows)
    N.check(N.cuda_lib().ub_row_norm(C.byref(a), _stream(x)), "ub_row_norm")
    return out


def embed_residual(ids: torch.Tensor, table: torch.Tensor, scale: float = 1.0):
    """First value of an fp32 residual stream: ``(x fp32, the same rows in the table's type)``."""
    f32 = _elem("embed_residual", table)
    if ids.dtype != torch.int32 or not table.is_contiguous():
        raise ValueError("embed_residual: int32 ids, contiguous table")
    T, (V, Hp) = ids.numel(), table.shape
    x = torch.empty(T, Hp, dtype=torch.float32, device=table.device)
    out = x if f32 else torch.empty(T, Hp, dtype=table.dtype, device=table.device)
    lib = N.cuda_lib()
    lib.ub_embed_residual.restype = C.c_int
    lib.ub_embed_residual.argtypes = [N.vp, N.vp, N.vp, N.vp, N.i32, N.i32, N.i32, N.f32, N.i32, N.vp, N.vp]
    N.check(lib.ub_embed_residual(ids.data_ptr(), table.data_ptr(), x.data_ptr(), out.data_ptr(), T, Hp, V, scale, int(f32),
                                  err_word(table.device).data_ptr(), _stream(table)), "ub_embed_residual")
    return x, out


# ---------------------------------------------------------------------------------------------
# Layers with carried state: input of a sublayer, wkv recurrence
# ---------------------------------------------------------------------------------------------
class Portions:
    """Rows [row0, row0 + rows) of a step as portions of sequences: ``q_start`` (int32 [n + 1], from 0) or one row per
    sequence; ``state_in`` / ``state_out`` int32 [n] rows of the state tensors (negative: none)."""

    __slots__ = ("row0", "rows", "n", "max_q", "q_start", "state_in", "state_out")

    def __init__(self, row0: int, rows: int, n: int, max_q: int, q_start, state_in, state_out):
        for t, k in ((q_start, n + 1), (state_in, n), (state_out, n)):
            if t is not None and (t.dtype != torch.int32 or t.numel() != k or not t.is_cuda):
                raise ValueError("portions: int32 CUDA tensors, one entry per sequence")
        if q_start is None and (rows != n or max_q != 1):
            raise ValueError("portions: without q_start every sequence has one row")
        self.row0, self.rows, self.n, self.max_q = row0, rows, n, max_q
        self.q_start, self.state_in, self.state_out = q_start, state_in, state_out


def _state_rows(what: str, t: Optional[torch.Tensor], tail: tuple) -> None:
    if t is not None and (t.dtype != torch.float32 or not t.is_contiguous() or tuple(t.shape[1:]) != tail):
        raise ValueError(f"{what}: state must be contiguous fp32 [rows, {', '.join(map(str, tail))}]")


def sublayer_in(x: torch.Tensor, portions: Sequence[Portions], weight: torch.Tensor, *, eps: float, y: Optional[torch.Tensor] = None,
                y_weight: Optional[torch.Tensor] = None, conv: Optional[torch.Tensor] = None,
                conv_state: Optional[torch.Tensor] = None, mu: Optional[torch.Tensor] = None,
                shift_state: Optional[torch.Tensor] = None, width: Optional[int] = None, offset_one: bool = True, tile: int = 0,
                experts: Optional[torch.Tensor] = None, routing: Optional["MoeRouting"] = None, rows: Optional[torch.Tensor] = None):
    """What the next sublayer reads: ``x' = x + norm(y)``, ``h = norm(x')`` plus its causal convolution over time with the taps
    ``conv`` ([taps, width], the last one meets the token itself), and with ``mu`` ([5, width]) the five token-shift
    mixes ``h + (previous h - h) * mu``.  Returns ``(x', out)``; out is [rows, width], or [5, rows, width] with ``mu``, in
    the type of ``weight``.  The state tensors hold what the sequences of ``portions`` carry on.

    Without ``conv`` and ``mu`` rows stand alone: ``y`` may be a mixture (``experts`` in the order of ``routing``, ``y`` the rows
    of its always-on expert or None), and ``rows`` (int32) picks the rows to compute -- only ``out`` of those is returned then,
    and ``x`` stays as it is; otherwise ``x`` is changed in place."""
    f32 = _elem("sublayer_in", weight, y, y_weight, conv, mu, experts)
    if conv is None and mu is None:
        return _sublayer_alone(x, weight, eps, y, y_weight, width, offset_one, experts, routing, rows, f32)
    if experts is not None or rows is not None:
        raise ValueError("sublayer_in: mixtures and picked rows go without convolution and mixes")
    T, Hp = x.shape
    if x.dtype != torch.float32 or not x.is_contiguous() or weight.numel() != Hp:
        raise ValueError("sublayer_in: contiguous fp32 stream, weights of its width")
    if y is not None and (y.shape != x.shape or not y.is_contiguous() or y_weight is None or y_weight.numel() != Hp):
        raise ValueError("sublayer_in: y has the stream's shape and a norm weight")
    taps = 0 if conv is None else conv.shape[0]
    n_mix = 0 if mu is None else mu.shape[0]
    for t in (conv, mu):
        if t is not None and (t.shape[1] != Hp or not t.is_contiguous()):
            raise ValueError("sublayer_in: conv and mu are contiguous [n, width]")
    if n_mix not in (0, 5):
        raise ValueError("sublayer_in: five token-shift mixes or none")
    _state_rows("sublayer_in conv", conv_state, (max(taps - 1, 0), Hp))
    _state_rows("sublayer_in shift", shift_state, (Hp,))
    states = [t for t in (conv_state, shift_state) if t is not None]
    out = torch.empty((n_mix, T, Hp) if n_mix else (T, Hp), dtype=weight.dtype, device=x.device)
    x_out = x if y is None else torch.empty_like(x)
    for p in portions:
        if p.row0 + p.rows > T:
            raise ValueError("sublayer_in: portions outside the step")
        a = N.UbSublayerInArgs()
        a.x, a.y, a.wy, a.x_out, a.wn = x.data_ptr(), _p(y), _p(y_weight), x_out.data_ptr(), weight.data_ptr()
        a.conv, a.conv_state, a.mu, a.shift_state, a.out = _p(conv), _p(conv_state), _p(mu), _p(shift_state), out.data_ptr()
        if states:
            a.state_in, a.state_out = _p(p.state_in), _p(p.state_out)
            a.state_rows = states[0].shape[0]
        a.q_start, a.err = _p(p.q_start), err_word(x.device).data_ptr()
        a.row0, a.out_mix_stride = p.row0, T * Hp
        a.H, a.Hp, a.taps, a.n_mix, a.num_seqs, a.max_q = width or Hp, Hp, taps, n_mix, p.n, p.max_q
        # rows in front of a tile are computed again: tiles as large as still leaves two CTAs per SM
        a.tile = tile or min(max(-(-p.rows // 296), 2), 32)
        a.f32, a.eps, a.w_off = int(f32), eps, 1.0 if offset_one else 0.0
        N.check(N.cuda_lib().ub_sublayer_in(C.byref(a), _stream(x)), "ub_sublayer_in")
    return x_out, out


def _sublayer_alone(x, weight, eps, y, y_weight, width, offset_one, experts, routing, rows, f32):
    T, Hp = x.shape
    if x.dtype != torch.float32 or not x.is_contiguous() or weight.numel() != Hp:
        raise ValueError("sublayer_in: contiguous fp32 stream, weights of its width")
    if y is not None and (y.shape != x.shape or not y.is_contiguous()):
        raise ValueError("sublayer_in: y has the stream's shape")
    if (y is not None or experts is not None) and (y_weight is None or y_weight.numel() != Hp):
        raise ValueError("sublayer_in: a norm weight for y")
    if rows is not None and rows.dtype != torch.int32:
        raise TypeError("sublayer_in: rows must be int32")
    a = N.UbSublayerInArgs()
    n = T if rows is None else rows.numel()
    out = torch.empty(n, Hp, dtype=weight.dtype, device=x.device)
    if n == 0:
        return out if rows is not None else (x, out)
    a.x, a.y, a.wy, a.wn, a.out, a.rows = x.data_ptr(), _p(y), _p(y_weight), weight.data_ptr(), out.data_ptr(), _p(rows)
    a.x_out = x.data_ptr() if rows is None else None
    if experts is not None:
        if routing.T != T or experts.shape[1] != Hp or not experts.is_contiguous():
            raise ValueError("sublayer_in: the routing is of another step, or expert rows of another width")
        a.yx, a.row_slot, a.topk_w = experts.data_ptr(), routing.row_slot.data_ptr(), routing.topk_w.data_ptr()
        a.K, a.slots, a.y_gate = routing.K, experts.shape[0], _p(routing.shared_gate if y is not None else None)
    a.err = err_word(x.device).data_ptr()
    a.H, a.Hp, a.n_rows, a.x_rows, a.f32, a.eps, a.w_off = width or Hp, Hp, n, T, int(f32), eps, 1.0 if offset_one else 0.0
    N.check(N.cuda_lib().ub_sublayer_in(C.byref(a), _stream(x)), "ub_sublayer_in")
    return out if rows is not None else (x, out)


def delta_mixer(proj: torch.Tensor, col: int, conv: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor, norm_w: torch.Tensor,
                conv_state: Optional[torch.Tensor], state: torch.Tensor, portions: Sequence[Portions], *, kv_heads: int, eps: float,
                dk_real: int = 0, dv_real: int = 0, out: Optional[torch.Tensor] = None, lanes: int = 0,
                decay: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None, gate_act: str = "silu") -> torch.Tensor:
    """Gated delta rule with its convolutions, head norm and gate (``gate_act``: "silu" or "sigmoid").  ``proj`` [T, ld]: from
    column ``col`` on, rows of [Q | K | V | gate | b | a] with ``kv_heads`` * Dk, the same, H * Dv, H * Dv, H and H columns.
    ``conv`` [taps, Q + K + V], ``state`` fp32 [rows, H, Dk, Dv], ``conv_state`` fp32 [rows, taps - 1, Q + K + V] -> [T, H * Dv]
    (``out`` may be columns of a wider tensor).  ``dk_real`` / ``dv_real``: head sizes before padding.  ``lanes``: see
    ``UbDeltaArgs``.

    ``decay`` (fp32 [T, H * Dk], before its non-linearities, ``dt_bias`` then [H * Dk]): one decay per key channel; with it and
    ``gate`` [T, H * Dv] the rows of ``proj`` are [Q | K | V | b]."""
    f32 = _elem("delta_mixer", proj, conv, out, gate)
    T, ld = proj.shape
    _, H, dk, dv = state.shape
    taps, Cn = conv.shape
    qk = kv_heads * dk
    chan = decay is not None
    if chan != (gate is not None):
        raise ValueError("delta_mixer: decays per channel go with gate rows of their own")
    need = Cn + (H if chan else H * dv + 2 * H)
    if proj.stride(1) != 1 or not conv.is_contiguous() or Cn != 2 * qk + H * dv or col + need > ld:
        raise ValueError("delta_mixer: rows of [Q | K | V | gate | b | a], taps over [Q | K | V]")
    if chan and (decay.dtype != torch.float32 or decay.shape != (T, H * dk) or gate.shape != (T, H * dv) or decay.stride(1) != 1 or gate.stride(1) != 1):
        raise ValueError("delta_mixer: fp32 decays [T, H * Dk] and gates [T, H * Dv]")
    for t, n in ((a_log, H), (dt_bias, H * dk if chan else H), (norm_w, dv)):
        if t.dtype != torch.float32 or t.numel() != n:
            raise ValueError("delta_mixer: fp32 a_log [H], dt_bias [H] (or [H * Dk]) and norm weight [Dv]")
    _state_rows("delta_mixer", state, (H, dk, dv))
    if taps > 1:
        _state_rows("delta_mixer convolutions", conv_state, (taps - 1, Cn))
        if conv_state.shape[0] != state.shape[0]:
            raise ValueError("delta_mixer: as many rows of either state")
    if out is None:
        out = torch.empty(T, H * dv, dtype=proj.dtype, device=proj.device)
    if out.shape != (T, H * dv) or out.stride(1) != 1:
        raise ValueError("delta_mixer: out is [T, H * Dv]")
    lib, e = N.cuda_lib(), proj.element_size()
    at = lambda c: proj.data_ptr() + (col + c) * e
    for p in portions:
        if p.row0 + p.rows > T:
            raise ValueError("delta_mixer: portions outside the step")
        a = N.UbDeltaArgs()
        if chan:
            a.qkv, a.gate, a.b, a.decay = at(0), gate.data_ptr(), at(Cn), decay.data_ptr()
            a.ld_gate, a.ld_decay = gate.stride(0), decay.stride(0)
        else:
            a.qkv, a.gate, a.b, a.a = at(0), at(Cn), at(Cn + H * dv), at(Cn + H * dv + H)
        a.gate_act = {"silu": 0, "sigmoid": 1}[gate_act]
        a.conv, a.a_log, a.dt_bias, a.norm_w = conv.data_ptr(), a_log.data_ptr(), dt_bias.data_ptr(), norm_w.data_ptr()
        a.conv_state, a.state = _p(conv_state if taps > 1 else None), state.data_ptr()
        a.state_in, a.state_out, a.q_start = _p(p.state_in), _p(p.state_out), _p(p.q_start)
        a.out, a.err = out.data_ptr(), err_word(proj.device).data_ptr()
        a.row0, a.ld, a.ld_out = p.row0, proj.stride(0), out.stride(0)
        a.H, a.G, a.dk, a.dv, a.dk_real, a.dv_real, a.taps = H, kv_heads, dk, dv, dk_real or dk, dv_real or dv, taps
        a.num_seqs, a.max_q, a.rows, a.state_rows, a.f32, a.lanes, a.eps = p.n, p.max_q, p.rows, state.shape[0], int(f32), lanes, eps
        if p.q_start is not None:
            ws = torch.empty(lib.ub_delta_workspace_floats(p.rows, p.n, H, kv_heads, dk, dv, int(chan)), dtype=torch.float32, device=proj.device)
            a.ws = ws.data_ptr()
        N.check(lib.ub_delta_mixer(C.byref(a), _stream(proj)), "ub_delta_mixer")
    return out


def stream_in(portions: Sequence[Portions], weight: torch.Tensor, bias: torch.Tensor, alpha: float, *, x: Optional[torch.Tensor] = None,
              ids: Optional[torch.Tensor] = None, table: Optional[torch.Tensor] = None, y: Optional[torch.Tensor] = None, scale: float = 1.0,
              streams: Optional[torch.Tensor] = None, mix: Optional[torch.Tensor] = None, x_res: Optional[torch.Tensor] = None,
              x_out: Optional[torch.Tensor] = None, shift: Optional[torch.Tensor] = None, shift_state: Optional[torch.Tensor] = None,
              rows: Optional[torch.Tensor] = None, tile: int = 0) -> torch.Tensor:
    """What a sublayer behind a Dynamic Tanh reads: ``x' = x + scale * y``, ``s = sum_j mix[j] * streams[j] + mix[-1] * x'`` (without
    ``mix``: x'), ``h = tanh(alpha * s) * weight + bias``, and with ``shift`` every row mixed with the row of the token before it.

    ``x``: fp32 [T, width], or ``ids`` (int32 [T]) and ``table`` for the embedding itself.  ``streams``: fp32 [n, T, width].
    ``x_res`` / ``x_out`` receive x' / s.  ``rows`` (int32, without ``shift``) picks the rows to compute.  Returns h in the type of
    ``weight``."""
    f32 = _elem("stream_in", weight, bias, y, shift, table)
    Hp = weight.numel()
    T = x.shape[0] if ids is None else ids.numel()
    if (x is None) == (ids is None) or (ids is not None and (ids.dtype != torch.int32 or table is None or table.shape[1] != Hp or not table.is_contiguous())):
        raise ValueError("stream_in: a stream, or ids and their table")
    for t in (x, x_res, x_out):
        if t is not None and (t.dtype != torch.float32 or t.shape != (T, Hp) or not t.is_contiguous()):
            raise ValueError("stream_in: streams are contiguous fp32 [T, width]")
    if bias.numel() != Hp or (y is not None and (y.shape != (T, Hp) or not y.is_contiguous())) or (shift is not None and shift.numel() != Hp):
        raise ValueError("stream_in: weights and sublayer rows of the stream's width")
    a = N.UbStreamInArgs()
    if mix is not None:
        n = mix.numel() - 1
        if mix.dtype != torch.float32 or (n and (streams is None or streams.dtype != torch.float32 or streams.shape[0] < n
                                                 or streams.shape[1:] != (T, Hp) or streams[0].stride() != (Hp, 1))):
            raise ValueError("stream_in: fp32 weights of n streams [n, T, width] and of x'")
        a.mix, a.n_hist = mix.data_ptr(), n
        if n:
            a.hist, a.hist_stride = streams.data_ptr(), streams.stride(0)
    a.x, a.ids, a.table, a.y, a.scale = _p(x), _p(ids), _p(table), _p(y), scale
    a.vocab = table.shape[0] if table is not None else 0
    a.x_res, a.x_out, a.w, a.b, a.alpha = _p(x_res), _p(x_out), weight.data_ptr(), bias.data_ptr(), alpha
    a.err, a.Hp, a.f32 = err_word(weight.device).data_ptr(), Hp, int(f32)
    lib = N.cuda_lib()
    cols = -(-Hp // 1024)
    if shift is None:
        n = T if rows is None else rows.numel()
        if rows is not None and rows.dtype != torch.int32:
            raise TypeError("stream_in: rows must be int32")
        out = torch.empty(n, Hp, dtype=weight.dtype, device=weight.device)
        a.out, a.rows, a.n_rows, a.x_rows = out.data_ptr(), _p(rows), n, T
        a.tile = tile or max(min(n * cols // 1184, 4), -(-n // 65535), 1)
        N.check(lib.ub_stream_in(C.byref(a), _stream(weight)), "ub_stream_in")
        return out
    if rows is not None:
        raise ValueError("stream_in: picked rows go without a shift")
    _state_rows("stream_in shift", shift_state, (Hp,))
    out = torch.empty(T, Hp, dtype=weight.dtype, device=weight.device)
    a.out, a.shift, a.shift_state = out.data_ptr(), shift.data_ptr(), _p(shift_state)
    for p in portions:
        if p.row0 + p.rows > T:
            raise ValueError("stream_in: portions outside the step")
        if shift_state is not None:
            a.state_in, a.state_out, a.state_rows = _p(p.state_in), _p(p.state_out), shift_state.shape[0]
        a.q_start, a.row0, a.num_seqs, a.max_q = _p(p.q_start), p.row0, p.n, p.max_q
        # the row in front of a tile is computed again: tiles as large as still leaves some CTAs per SM
        a.tile = tile or max(min(p.rows * cols // 592, 16), -(-p.max_q // 65535), 1)
        N.check(lib.ub_stream_in(C.byref(a), _stream(weight)), "ub_stream_in")
    return out


WKV_CHUNK = 64


def wkv_mixer(rkvg: torch.Tensor, ww: torch.Tensor, u: torch.Tensor, norm_w: torch.Tensor, state: torch.Tensor,
              portions: Sequence[Portions], *, eps: float, norm_dim: int = 0, chunk: Optional[int] = None) -> torch.Tensor:
    """RWKV-6 style recurrence with head norm and SiLU gate: ``rkvg`` [4, T, H * D], ``ww`` fp32 [T, H * D] (decay =
    exp(-exp(ww))), ``u`` fp32 [H, D], ``norm_w`` fp32 [H * D], ``state`` fp32 [rows, H, D, D] -> [T, H * D].  ``chunk``:
    tokens per parallel chunk of long portions (0 = one CTA walks a portion, None = chosen here)."""
    f32 = _elem("wkv_mixer", rkvg)
    _, T, ld = rkvg.shape
    H, D = u.shape
    if not rkvg.is_contiguous() or ld != H * D or ww.dtype != torch.float32 or ww.shape != (T, ld) or not ww.is_contiguous():
        raise ValueError("wkv_mixer: rkvg [4, T, H * D] and fp32 ww [T, H * D], contiguous")
    if u.dtype != torch.float32 or norm_w.dtype != torch.float32 or norm_w.numel() != ld:
        raise ValueError("wkv_mixer: fp32 u [H, D] and norm weight [H * D]")
    _state_rows("wkv_mixer", state, (H, D, D))
    out = torch.empty(T, ld, dtype=rkvg.dtype, device=rkvg.device)
    lib = N.cuda_lib()
    for p in portions:
        if p.row0 + p.rows > T:
            raise ValueError("wkv_mixer: portions outside the step")
        a = N.UbWkvArgs()
        e = rkvg.element_size() * T * ld
        a.r, a.k, a.v, a.g = (rkvg.data_ptr() + i * e for i in range(4))
        a.ww, a.u, a.norm_w, a.state, a.out = ww.data_ptr(), u.data_ptr(), norm_w.data_ptr(), state.data_ptr(), out.data_ptr()
        a.state_in, a.state_out, a.q_start, a.err = _p(p.state_in), _p(p.state_out), _p(p.q_start), err_word(rkvg.device).data_ptr()
        a.row0, a.ld, a.H, a.D, a.norm_dim, a.num_seqs = p.row0, ld, H, D, norm_dim or D, p.n
        a.state_rows, a.f32, a.eps = state.shape[0], int(f32), eps
        c = chunk
        if c is None:       # chunks pay once a portion is long and the sequences alone do not fill the device
            c = WKV_CHUNK if p.max_q > 2 * WKV_CHUNK and p.n * H < 4 * 148 else 0
        if p.q_start is None:
            c = 0
        if c:
            a.chunk, a.rows, a.max_chunks = c, p.rows, p.rows // c + p.n
            ws = torch.empty(lib.ub_wkv_workspace_floats(p.rows, ld, H, D, a.max_chunks), dtype=torch.float32, device=rkvg.device)
            a.ws = ws.data_ptr()
        N.check(lib.ub_wkv_mixer(C.byref(a), _stream(rkvg)), "ub_wkv_mixer")
    return out


_GROUP_TILES: dict = {}


def gemm_stacked(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``out[e] = x[e] @ w[e]^T`` for a stack of equal products: x [E, T, K] (contiguous), w [E, N, K] -> [E, T, N].  Up to 16
    rows on the weight-streaming kernel, beyond on the grouped GEMM with a tile table that is fixed by the sizes; thousands of
    rows fill the device one product at a time, in the CTA-pair kernel that the grouped form does not have."""
    f32 = _elem("gemm_stacked", x, w)
    E, T, Kd = x.shape
    n = w.shape[1]
    if not x.is_contiguous() or not w.is_contiguous() or w.shape[0] != E or w.shape[2] != Kd:
        raise ValueError("gemm_stacked: contiguous x [E, T, K] and w [E, N, K]")
    out = torch.empty(E, T, n, dtype=x.dtype, device=x.device)
    if T <= 16 and not f32:
        a = N.UbGemmArgs()
        a.x, a.w, a.out, a.err = x.data_ptr(), w.data_ptr(), out.data_ptr(), err_word(x.device).data_ptr()
        a.M, a.N, a.K, a.ldx, a.ldw, a.ldo, a.w_rows_total = T, n, Kd, Kd, Kd, n, n
        a.batch, a.x_batch, a.w_batch, a.out_batch = E, T * Kd, n * Kd, T * n
        N.check(N.cuda_lib().ub_gemm_tn(C.byref(a), _stream(x)), "ub_gemm_tn(stacked)")
        return out
    if T >= 4096 and not f32:
        for e in range(E):
            gemm_tn(x[e], w[e], out=out[e])
        return out
    tn = moe_tile_tokens(E * T, 1, E)
    key = (E, T, tn, x.device)
    tiles = _GROUP_TILES.get(key)
    if tiles is None:
        rows = [[e, e * T + t, (e + 1) * T, 0] for e in range(E) for t in range(0, T, tn)]
        tiles = _GROUP_TILES[key] = torch.tensor(rows, dtype=torch.int32).to(x.device)
    _gemm_grouped_plain(x.view(E * T, Kd), w.view(E * n, Kd), n, None, out.view(E * T, n),
                        {"tiles": tiles.data_ptr(), "max_tiles": tiles.shape[0], "w_rows": n, "tile_tokens": tn}, f32)
    return out


# ---------------------------------------------------------------------------------------------
# Multi-head latent attention
# ---------------------------------------------------------------------------------------------
def _latent_args(T: int, positions, inv_freq, rot: int, f32: bool, gain: float, device):
    if positions.dtype != torch.int32 or inv_freq.dtype != torch.float32 or positions.numel() != T:
        raise TypeError("latent attention: int32 positions, fp32 frequencies")
    a = N.UbLatentArgs()
    a.positions, a.inv_freq, a.err = positions.data_ptr(), inv_freq.data_ptr(), err_word(device).data_ptr()
    a.T, a.rot, a.rot_dims, a.f32, a.gain = T, rot, 2 * inv_freq.numel(), int(f32), gain
    return a


def latent_rows(down: torch.Tensor, positions: torch.Tensor, slot_mapping: torch.Tensor, cache: torch.Tensor, q_norm_w: torch.Tensor,
                kv_norm_w: torch.Tensor, inv_freq: torch.Tensor, *, eps: float, gain: float = 1.0, q_real: int = 0,
                kv_real: int = 0) -> torch.Tensor:
    """``down`` [T, q_rank + kv_rank + rot] -> normed query latents [T, q_rank]; the normed kv latent and the rotated key part
    go to the rows ``slot_mapping`` of ``cache`` [num_blocks, 1, block_size, kv_rank + rot].  ``q_real`` / ``kv_real``:
    elements that the norms average over when segments are padded."""
    f32 = _elem("latent_rows", down, cache, q_norm_w, kv_norm_w)
    T, qr, kvr = down.shape[0], q_norm_w.numel(), kv_norm_w.numel()
    rot = down.shape[1] - qr - kvr
    if cache.shape[-1] != kvr + rot or cache.shape[1] != 1 or not cache.is_contiguous() or not down.is_contiguous():
        raise ValueError("latent_rows: cache rows are [kv latent | rotated part]")
    if slot_mapping.dtype != torch.int32 or slot_mapping.numel() != T:
        raise TypeError("latent_rows: int32 slots, one per token")
    out = torch.empty(T, qr, dtype=down.dtype, device=down.device)
    a = _latent_args(T, positions, inv_freq, rot, f32, gain, down.device)
    a.down, a.q_latent, a.cache, a.q_norm_w, a.kv_norm_w = down.data_ptr(), out.data_ptr(), cache.data_ptr(), q_norm_w.data_ptr(), kv_norm_w.data_ptr()
    a.slot_mapping, a.num_slots = slot_mapping.data_ptr(), cache.shape[0] * cache.shape[2]
    a.q_rank, a.kv_rank, a.q_real, a.kv_real, a.eps = qr, kvr, q_real or qr, kv_real or kvr, eps
    N.check(N.cuda_lib().ub_latent_rows(C.byref(a), _stream(down)), "ub_latent_rows")
    return out


def latent_rotate(q: torch.Tensor, positions: torch.Tensor, inv_freq: torch.Tensor, rot: int, out: Optional[torch.Tensor] = None,
                  gain: float = 1.0) -> torch.Tensor:
    """Turns the last ``rot`` elements of every head of ``q`` [T, heads, size] (rows may be strided) and puts them last in the
    heads of ``out`` (default: in place)."""
    out = q if out is None else out
    f32 = _elem("latent_rotate", q, out)
    T, H = q.shape[:2]
    if q.stride(2) != 1 or out.stride(2) != 1 or out.shape[:2] != q.shape[:2]:
        raise ValueError("latent_rotate: heads must be contiguous")
    a = _latent_args(T, positions, inv_freq, rot, f32, gain, q.device)
    a.H, a.q, a.q_out = H, q.data_ptr(), out.data_ptr()
    a.q_stride, a.q_head, a.q_off = q.stride(0), q.stride(1), q.shape[2] - rot
    a.qo_stride, a.qo_head, a.qo_off = out.stride(0), out.stride(1), out.shape[2] - rot
    N.check(N.cuda_lib().ub_latent_rotate(C.byref(a), _stream(q)), "ub_latent_rotate")
    return out


def gemm_heads(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``out[t, h] = x[t, h] @ w[h]^T``: x [T, H, K] and out [T, H, N] with any token and head strides, w [H, N, K]."""
    f32 = _elem("gemm_heads", x, w, out)
    T, H, Kd = x.shape
    if w.shape != (H, out.shape[2], Kd) or out.shape[:2] != (T, H) or x.stride(2) != 1 or out.stride(2) != 1 or not w.is_contiguous():
        raise ValueError("gemm_heads: x [T, H, K], w [H, N, K], out [T, H, N]")
    a = N.UbHeadGemmArgs()
    a.x, a.w, a.out = x.data_ptr(), w.data_ptr(), out.data_ptr()
    a.x_stride, a.x_head, a.out_stride, a.out_head = x.stride(0), x.stride(1), out.stride(0), out.stride(1)
    a.M, a.N, a.K, a.H, a.f32 = T, w.shape[1], Kd, H, int(f32)
    N.check(N.cuda_lib().ub_gemm_heads(C.byref(a), _stream(x)), "ub_gemm_heads")
    return out


def latent_splits(seqs: int, heads: int, ctx: int, row: int, v_dim: int) -> int:
    """Key ranges per sequence of a decode step: rounds of CTAs over the SMs at their share of the bandwidth, against what the
    partial results cost to write and merge."""
    ctas = seqs * -(-heads // (16 if heads <= 16 else 32))
    resident = 148 * (2 if row <= 328 and heads <= 16 else 1)
    best, cost = 1, None
    for s in (1, 2, 4, 8, 16, 32):
        if s > 1 and ctx // s < 64:
            break
        us = -(-ctas * s // resident) * (ctx / s * row * 2 / 45e3 * (resident // 148) + 3.0)
        us += 0.0 if s == 1 else 3.0 + seqs * heads * s * v_dim * 8 / 4e6
        if cost is None or us < cost:
            best, cost = s, us
    return best


def attn_latent(q: torch.Tensor, cache: torch.Tensor, v_dim: int, block_tables: torch.Tensor, seq_lens: torch.Tensor, *, scale: float,
                sinks: Optional[torch.Tensor] = None, q_start: Optional[torch.Tensor] = None, max_q_len: int = 1,
                out: Optional[torch.Tensor] = None, splits: int = 0, scratch: Optional[torch.Tensor] = None,
                max_seq_len: Optional[int] = None) -> torch.Tensor:
    """Attention of all heads over one cached row per token: q [T, H, D], cache [num_blocks, 1, block_size, D]; keys are the
    rows, values their first ``v_dim`` elements -> [T, H, v_dim].  With ``q_start`` prompt portions, else one query per
    sequence; causal."""
    f32 = _elem("attn_latent", q, cache, out)
    T, H, D = q.shape
    if cache.shape[1] != 1 or cache.shape[3] != D or not cache.is_contiguous() or q.stride(1) != D or q.stride(2) != 1:
        raise ValueError("attn_latent: cache rows and query heads of one size")
    if out is None:
        out = torch.empty(T, H, v_dim, dtype=q.dtype, device=q.device)
    a = _attn_args(q, cache, cache[..., :v_dim], out, None, block_tables, seq_lens, H, 1, D, scale, sinks)
    a.kv_shared, a.causal = 1, 1
    if q_start is not None or f32:
        splits = 1
    if splits <= 0:
        ctx = max_seq_len if max_seq_len is not None else block_tables.shape[1] * cache.shape[2]
        splits = latent_splits(T, H, ctx, D, v_dim)
    if splits > 1:
        need = T * H * splits * (v_dim + 2)
        if scratch is None or scratch.numel() < need:
            scratch = torch.empty(need, dtype=torch.float32, device=q.device)
        a.scratch = scratch.data_ptr()
    a.splits = splits
    if q_start is not None:
        a.q_start, a.total_q, a.max_q_len = q_start.data_ptr(), T, max_q_len
    lib = N.cuda_lib()
    N.check((lib.ub_attn_f32 if f32 else lib.ub_attn_latent)(C.byref(a), _stream(q)), "ub_attn_latent")
    return out


def expanded_supported(dim: int, rot: int, vdim: int) -> bool:
    """Whether ``attn_expanded`` takes these (padded) head sizes."""
    return dim % 16 == 0 and 16 <= dim <= 128 and vdim % 16 == 0 and 16 <= vdim <= 128 and rot % 8 == 0 and 8 <= rot <= 64


def latent_gather(cache: torch.Tensor, block_tables: torch.Tensor, seq_lens: torch.Tensor, page_start: torch.Tensor,
                  rows: int) -> torch.Tensor:
    """Cache rows of sequences, one after the other: sequence i from row ``16 * page_start[i]`` on, zeros behind its end and
    behind the last one -> [rows, row size] (``rows`` a multiple of 16)."""
    _bf16c(cache, "cache")
    if page_start.dtype != torch.int32 or page_start.numel() != seq_lens.numel() + 1 or cache.shape[1] != 1 or cache.shape[2] != 16:
        raise ValueError("latent_gather: int32 page_start [n + 1], pages of 16 rows")
    out = torch.empty(rows, cache.shape[3], dtype=cache.dtype, device=cache.device)
    a = N.UbExpandArgs()
    a.cache, a.lat, a.block_tables, a.seq_lens = cache.data_ptr(), out.data_ptr(), block_tables.data_ptr(), seq_lens.data_ptr()
    a.page_start, a.err, a.rows, a.row, a.num_seqs = page_start.data_ptr(), err_word(cache.device).data_ptr(), rows, cache.shape[3], seq_lens.numel()
    a.block_size, a.num_blocks, a.max_blocks_per_seq = 16, cache.shape[0], block_tables.shape[1]
    N.check(N.cuda_lib().ub_latent_gather(C.byref(a), _stream(cache)), "ub_latent_gather")
    return out


def attn_expanded(q: torch.Tensor, kv: torch.Tensor, lat: torch.Tensor, v_dim: int, seq_lens: torch.Tensor, q_start: torch.Tensor,
                  page_start: torch.Tensor, max_q_len: int, *, scale: float, sinks: Optional[torch.Tensor] = None,
                  out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal prompt attention over expanded latents on tcgen05: q [T, H, dim + rot] (rotated), kv [R, H * (dim + v_dim)], lat
    [R, kv_rank + rot] as ``latent_gather`` gives them -> [T, H, v_dim]."""
    for t, n in ((q, "q"), (kv, "kv"), (lat, "lat")):
        _bf16c(t, n)
    T, H, size = q.shape
    dim = kv.shape[1] // H - v_dim
    if kv.shape[0] != lat.shape[0] or not kv.is_contiguous() or not lat.is_contiguous() or q.stride(1) != size or q.stride(2) != 1:
        raise ValueError("attn_expanded: contiguous kv and lat rows of the same number, contiguous heads")
    if sinks is not None and (sinks.dtype != torch.float32 or sinks.numel() != H):
        raise ValueError("sinks: fp32, one per query head")
    if out is None:
        out = torch.empty(T, H, v_dim, dtype=q.dtype, device=q.device)
    a = N.UbExpandArgs()
    a.q, a.kv, a.lat, a.out, a.sinks = q.data_ptr(), kv.data_ptr(), lat.data_ptr(), out.data_ptr(), _p(sinks)
    a.seq_lens, a.q_start, a.page_start, a.err = seq_lens.data_ptr(), q_start.data_ptr(), page_start.data_ptr(), err_word(q.device).data_ptr()
    a.q_stride, a.o_stride, a.T, a.H, a.dim, a.rot, a.vdim = q.stride(0), out.stride(0), T, H, dim, size - dim, v_dim
    a.row, a.kv_rank, a.rows, a.num_seqs, a.max_q, a.scale = lat.shape[1], lat.shape[1] - a.rot, lat.shape[0], seq_lens.numel(), max_q_len, scale
    N.check(N.cuda_lib().ub_attn_expanded(C.byref(a), _stream(q)), "ub_attn_expanded")
    return out


# ---------------------------------------------------------------------------------------------
# RoPE + KV append
# ---------------------------------------------------------------------------------------------
def rope_kv_append(qkv: torch.Tensor, positions: torch.Tensor, slot_mapping: Optional[torch.Tensor],
                   k_cache: Optional[torch.Tensor], v_cache: Optional[torch.Tensor], *, num_q_heads: int,
                   num_kv_heads: int, head_dim: int, rotary_dim: Optional[int] = None, theta: float = 10000.0,
                   pos_scale: float = 1.0, interleaved: bool = False, q_norm_w: Optional[torch.Tensor] = None,
                   k_norm_w: Optional[torch.Tensor] = None, norm_eps: float = 1e-6,
                   llama3_scaling: Optional[Sequence[float]] = None, v_head_dim: Optional[int] = None,
                   norm_dim: int = 0, inv_freq: Optional[torch.Tensor] = None, k_cache_only: bool = False,
                   row_norm: bool = False, gain: float = 1.0, v_inv_freq: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Rotates q and k inside ``qkv`` [T, (Hq+Hkv)*D + Hkv*Dv] in place and appends k, v to the paged cache.

    ``num_kv_heads = 0``: rows hold queries only (a layer that reads another layer's keys).  ``inv_freq`` (fp32
    [rotary_dim / 2]) replaces the frequencies that ``theta`` and the scaling give; ``norm_dim`` is the number of elements
    the head norm averages over when heads are zero-padded.  ``k_cache_only``: the rotated k is needed in the cache only.
    ``row_norm``: one norm over all queries of a token and one over all its keys (weights of that size).  ``qkv`` may be the
    first columns of wider rows.  ``gain``: factor on cosine and sine (with ``inv_freq``).  ``v_inv_freq`` (fp32 [n]): values are
    cached turned by their position, element i with element i + n."""
    f32 = _elem("rope_kv_append", qkv, k_cache, v_cache, q_norm_w, k_norm_w)
    if gain != 1.0 and inv_freq is None:
        raise ValueError("rope_kv_append: a gain goes with a frequency table")
    if qkv.stride(1) != 1:
        raise ValueError("qkv: rows must be contiguous")
    T = qkv.shape[0]
    if positions.dtype != torch.int32 or (slot_mapping is not None and slot_mapping.dtype != torch.int32):
        raise TypeError("positions / slot_mapping must be int32")
    a = N.UbRopeArgs()
    a.qkv, a.positions, a.slot_mapping = qkv.data_ptr(), positions.data_ptr(), _p(slot_mapping)
    a.k_cache, a.v_cache = _p(k_cache), _p(v_cache)
    a.q_norm_w, a.k_norm_w = _p(q_norm_w), _p(k_norm_w)
    a.err = err_word(qkv.device).data_ptr()
    a.T, a.Hq, a.Hkv, a.D = T, num_q_heads, num_kv_heads, head_dim
    a.rotary_dim = head_dim if rotary_dim is None else rotary_dim
    if k_cache is not None:
        a.block_size = k_cache.shape[2]
        a.num_slots = k_cache.shape[0] * k_cache.shape[2]
    else:
        a.block_size, a.num_slots = 16, 0
        a.slot_mapping = None
    a.theta, a.pos_scale, a.norm_eps = theta, pos_scale, norm_eps
    a.interleaved = 1 if interleaved else 0
    a.Dv, a.norm_dim, a.f32 = v_head_dim or head_dim, norm_dim, int(f32)
    a.k_cache_only, a.row_norm, a.ld = int(k_cache_only), int(row_norm), qkv.stride(0)
    if row_norm and (q_norm_w is None or q_norm_w.numel() != num_q_heads * head_dim or
                     (num_kv_heads and (k_norm_w is None or k_norm_w.numel() != num_kv_heads * head_dim))):
        raise ValueError("rope_kv_append: row norms take weights over all heads")
    if qkv.shape[1] != (num_q_heads + num_kv_heads) * head_dim + num_kv_heads * a.Dv:
        raise ValueError(f"rope_kv_append: rows of {qkv.shape[1]} elements do not hold these heads")
    if k_cache is not None and (k_cache.shape[1], k_cache.shape[3], v_cache.shape[3]) != (num_kv_heads, head_dim, a.Dv):
        raise ValueError("rope_kv_append: cache shapes do not match the heads")
    if inv_freq is not None:
        if inv_freq.dtype != torch.float32 or inv_freq.numel() != a.rotary_dim // 2:
            raise ValueError("inv_freq: fp32, one entry per rotated pair")
        a.inv_freq, a.gain = inv_freq.data_ptr(), gain
    if v_inv_freq is not None:
        if v_inv_freq.dtype != torch.float32 or 2 * v_inv_freq.numel() > a.Dv:
            raise ValueError("v_inv_freq: fp32, one entry per turned pair")
        a.v_inv_freq, a.v_rot = v_inv_freq.data_ptr(), 2 * v_inv_freq.numel()
    if llama3_scaling is not None:
        a.l3_factor, a.l3_low_freq_factor, a.l3_high_freq_factor, a.l3_orig_ctx = llama3_scaling
    N.check(N.cuda_lib().ub_rope_kv_append(C.byref(a), _stream(qkv)), "ub_rope_kv_append")
    return qkv


def map_rows(qkv: torch.Tensor, slot_mapping: Optional[torch.Tensor], k_cache: Optional[torch.Tensor], v_cache: Optional[torch.Tensor], *,
             num_heads: int, maps: int, dim: int) -> torch.Tensor:
    """Queries of a differential attention for the attention kernels, keys and values into the cache.  ``qkv`` [T, ..]: rows of
    [Q: heads * maps * dim | K: kv heads * maps * dim | V: kv heads * Dv] (``slot_mapping`` None: Q alone is read); ``k_cache``
    [.., kv heads, block, maps * dim] -> [T, heads * maps, maps * dim], each query zero where the other maps' keys lie."""
    f32 = _elem("map_rows", qkv, k_cache, v_cache)
    if qkv.stride(1) != 1 or dim % 8:
        raise ValueError("map_rows: contiguous rows, sizes in multiples of 8")
    out = torch.empty(qkv.shape[0], num_heads * maps, maps * dim, dtype=qkv.dtype, device=qkv.device)
    a = N.UbMapRowsArgs()
    a.src, a.q_out, a.err = qkv.data_ptr(), out.data_ptr(), err_word(qkv.device).data_ptr()
    a.T, a.H, a.maps, a.dim, a.ld, a.f32 = qkv.shape[0], num_heads, maps, dim, qkv.stride(0), int(f32)
    need = num_heads * maps * dim
    if slot_mapping is not None:
        if slot_mapping.dtype != torch.int32 or k_cache.shape[:3] != v_cache.shape[:3] or k_cache.shape[3] != maps * dim:
            raise ValueError("map_rows: caches do not match the heads")
        a.G, a.block_size, a.dv = k_cache.shape[1], k_cache.shape[2], v_cache.shape[3]
        a.slot_mapping, a.k_cache, a.v_cache = slot_mapping.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr()
        a.num_slots = k_cache.shape[0] * k_cache.shape[2]
        need += a.G * (maps * dim + a.dv)
    if qkv.shape[1] < need:
        raise ValueError(f"map_rows: rows of {qkv.shape[1]} elements do not hold these heads")
    N.check(N.cuda_lib().ub_map_rows(C.byref(a), _stream(qkv)), "ub_map_rows")
    return out


def attn_finish(att: torch.Tensor, v_dim: int, *, gate: Optional[torch.Tensor] = None, gate_kind: str = "", maps: int = 1, lam: float = 0.0,
                factor: float = 1.0, eps: float = 0.0, positions: Optional[torch.Tensor] = None, inv_freq: Optional[torch.Tensor] = None,
                dv_real: int = 0) -> torch.Tensor:
    """Between an attention's outputs ``att`` [T, heads * maps * v_dim] and its output projection: maps subtracted
    (``(a1 - lam * a2) / rms * factor``), outputs turned back by their position (``inv_freq`` fp32 [dv_real / 2]), times the sigmoid
    of ``gate`` (``gate_kind`` "head": [T, >= heads], "element": [T, heads * v_dim]) -> [T, heads * v_dim]."""
    f32 = _elem("attn_finish", att, gate)
    T, H = att.shape[0], att.shape[1] // (v_dim * maps)
    if att.stride(1) != 1 or H * v_dim * maps != att.shape[1]:
        raise ValueError("attn_finish: rows of whole heads")
    out = torch.empty(T, H * v_dim, dtype=att.dtype, device=att.device)
    a = N.UbAttnFinishArgs()
    a.att, a.out, a.ld_att, a.ld_out = att.data_ptr(), out.data_ptr(), att.stride(0), out.stride(0)
    a.gate_kind = {"": 0, "head": 1, "element": 2}[gate_kind]
    if a.gate_kind:
        if gate.shape[0] != T or gate.stride(1) != 1 or gate.shape[1] < (H if gate_kind == "head" else H * v_dim):
            raise ValueError("attn_finish: one gate row per token")
        a.gate, a.ld_gate = gate.data_ptr(), gate.stride(0)
    a.T, a.H, a.dv, a.dv_real, a.maps, a.f32 = T, H, v_dim, dv_real or v_dim, maps, int(f32)
    a.lambda_, a.factor, a.eps = lam, factor, eps
    if inv_freq is not None:
        if inv_freq.dtype != torch.float32 or positions.dtype != torch.int32 or inv_freq.numel() != a.dv_real // 2 or positions.numel() != T:
            raise ValueError("attn_finish: fp32 frequencies per pair, int32 positions")
        a.inv_freq, a.positions = inv_freq.data_ptr(), positions.data_ptr()
    N.check(N.cuda_lib().ub_attn_finish(C.byref(a), _stream(att)), "ub_attn_finish")
    return out


# ---------------------------------------------------------------------------------------------
# Attention
# ---------------------------------------------------------------------------------------------
def _attn_args(q, k_cache, v_cache, out, lse, block_tables, seq_lens, Hq, Hkv, D, scale, sinks=None, softcap=0.0, chunk=0):
    a = N.UbAttnArgs()
    a.q, a.k_cache, a.v_cache, a.out, a.lse = q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), _p(lse)
    a.block_tables, a.seq_lens = block_tables.data_ptr(), seq_lens.data_ptr()
    a.err = err_word(q.device).data_ptr()
    a.num_seqs, a.Hq, a.Hkv, a.D = seq_lens.shape[0], Hq, Hkv, D
    a.block_size, a.max_blocks_per_seq, a.num_blocks = k_cache.shape[2], block_tables.shape[1], k_cache.shape[0]
    a.q_stride, a.o_stride = q.stride(0), out.stride(0)
    a.scale = scale if scale is not None else 1.0 / math.sqrt(D)
    a.Dv, a.softcap, a.chunk = v_cache.shape[3], softcap, chunk
    if k_cache.shape[3] != D or out.shape[-1] != a.Dv:
        raise ValueError("attention: head sizes of q, caches and out do not match")
    if sinks is not None:
        if sinks.dtype != torch.float32 or sinks.numel() != Hq:
            raise ValueError("sinks: fp32, one per query head")
        a.sinks = sinks.data_ptr()
    return a


def attn_decode(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_tables: torch.Tensor,
                seq_lens: torch.Tensor, *, scale: Optional[float] = None, window: int = 0, kv_start: int = 0,
                alibi_slopes: Optional[torch.Tensor] = None, splits: int = 0, scratch: Optional[torch.Tensor] = None,
                out: Optional[torch.Tensor] = None, return_lse: bool = False, lse: Optional[torch.Tensor] = None,
                max_seq_len: Optional[int] = None, merge: Optional[tuple] = None, kernel: Optional[str] = None,
                sinks: Optional[torch.Tensor] = None, softcap: float = 0.0, chunk: int = 0):
    """One query token per sequence.  q: [B, Hq, D] (last two dims contiguous); caches [nb, Hkv, bs, D] (the value cache may
    have a head size of its own).  ``sinks``: fp32 [Hq], one logit per head that joins the softmax denominator.
    ``softcap`` > 0: scores become softcap * tanh(score / softcap).  ``chunk`` > 0: a query sees keys of its own chunk of that many
    positions only.  fp32 operands run in 32-bit arithmetic.

    ``kernel="warp"`` calls the warp-per-item kernel directly (page size 16, head size 64 / 128, ``splits == 1``, no
    window, no ALiBi) instead of going through the dispatcher's choice."""
    f32 = _elem("attn_decode", q, k_cache, v_cache, out)
    B, Hq, D = q.shape
    Hkv, Dv = k_cache.shape[1], v_cache.shape[3]
    if out is None:
        out = torch.empty((B, Hq, Dv), dtype=q.dtype, device=q.device)
    if return_lse and lse is None:
        lse = torch.empty((B, Hq), dtype=torch.float32, device=q.device)
    if f32:
        splits = 1
    if splits <= 0:
        ctx = max_seq_len if max_seq_len is not None else block_tables.shape[1] * k_cache.shape[2]
        if window > 0:
            ctx = min(ctx, window)
        if chunk > 0:
            ctx = min(ctx, chunk)
        ctas = B * Hkv
        splits = 1
        while ctas * splits < 2 * 148 and ctx // (splits * 2) >= 256 and splits < 16:
            splits *= 2
    a = _attn_args(q, k_cache, v_cache, out, lse, block_tables, seq_lens, Hq, Hkv, D, scale, sinks, softcap, chunk)
    if splits > 1:
        need = B * Hq * splits * (Dv + 2)
        if scratch is None or scratch.numel() < need:
            scratch = torch.empty(need, dtype=torch.float32, device=q.device)
        a.scratch = scratch.data_ptr()
    a.window, a.splits, a.kv_start = window, splits, kv_start
    a.alibi_slopes = _p(alibi_slopes)
    if merge is not None:        # (o [B, Hq, D] bf16 contiguous, lse [B, Hq] fp32): partial over a disjoint key set
        a.merge_o, a.merge_lse = merge[0].data_ptr(), merge[1].data_ptr()
    if f32:
        N.check(N.cuda_lib().ub_attn_f32(C.byref(a), _stream(q)), "ub_attn_f32")
    elif kernel == "warp":
        lib = N.cuda_lib()
        if not lib.ub_attn_decode_warp_supported(C.byref(a)):
            raise ValueError("attn_decode(kernel='warp'): page size 16, head size 64 / 128, one split, no window / ALiBi")
        N.check(lib.ub_attn_decode_warp(C.byref(a), _stream(q)), "ub_attn_decode_warp")
    else:
        N.check(N.cuda_lib().ub_attn_decode(C.byref(a), _stream(q)), "ub_attn_decode")
    return (out, lse) if return_lse else out


def attn_prefill(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_tables: torch.Tensor,
                 seq_lens: torch.Tensor, q_start: torch.Tensor, max_q_len: int, *, scale: Optional[float] = None,
                 causal: bool = True, window: int = 0, kv_start: int = 0,
                 alibi_slopes: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
                 return_lse: bool = False, lse: Optional[torch.Tensor] = None, merge: Optional[tuple] = None,
                 kv_splits: int = 1, scratch: Optional[torch.Tensor] = None, sinks: Optional[torch.Tensor] = None,
                 softcap: float = 0.0, chunk: int = 0):
    """Ragged prefill: q [T, Hq, D]; sequence i owns query rows q_start[i]:q_start[i+1] and sees
    seq_lens[i] keys, its last query at kv position seq_lens[i]-1.  ``softcap``, ``chunk``: see :func:`attn_decode`.

    ``kv_splits > 1`` (tensor-core kernel only, no ``merge``) divides every CTA's key tiles over that many CTAs and
    folds the partial results with a second small kernel: for launches with few query tiles and many keys, such as
    the shared-prefix pass of a tensor-parallel rank that holds one KV head.  ``scratch`` (fp32, at least
    :func:`attn_prefill_split_scratch_floats` elements) holds the partials."""
    f32 = _elem("attn_prefill", q, k_cache, v_cache, out)
    T, Hq, D = q.shape
    Hkv = k_cache.shape[1]
    if out is None:
        out = torch.empty((T, Hq, v_cache.shape[3]), dtype=q.dtype, device=q.device)
    if return_lse and lse is None:
        lse = torch.empty((T, Hq), dtype=torch.float32, device=q.device)
    a = _attn_args(q, k_cache, v_cache, out, lse, block_tables, seq_lens, Hq, Hkv, D, scale, sinks, softcap, chunk)
    a.q_start = q_start.data_ptr()
    a.causal, a.window, a.kv_start = (1 if causal else 0), window, kv_start
    a.total_q, a.max_q_len = T, max_q_len
    a.alibi_slopes = _p(alibi_slopes)
    if merge is not None:
        a.merge_o, a.merge_lse = merge[0].data_ptr(), merge[1].data_ptr()
    if kv_splits > 1:
        need = attn_prefill_split_scratch_floats(T, Hq, D, kv_splits)
        if scratch is None or scratch.numel() < need:
            scratch = torch.empty(need, dtype=torch.float32, device=q.device)
        if scratch.dtype != torch.float32:
            raise TypeError("scratch must be float32")
        a.splits, a.scratch = kv_splits, scratch.data_ptr()
    if f32:
        N.check(N.cuda_lib().ub_attn_f32(C.byref(a), _stream(q)), "ub_attn_f32")
    else:
        N.check(N.cuda_lib().ub_attn_prefill(C.byref(a), _stream(q)), "ub_attn_prefill")
    return (out, lse) if return_lse else out


def attn_prefill_split_scratch_floats(T: int, Hq: int, D: int, kv_splits: int) -> int:
    """fp32 elements of workspace that ``attn_prefill(kv_splits=...)`` needs: the log-sum-exps, then the bf16 rows."""
    lse = (kv_splits * T * Hq + 3) // 4 * 4
    return lse + (kv_splits * T * Hq * D + 1) // 2


def dense_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, *, causal: bool = False,
                    scale: Optional[float] = None) -> torch.Tensor:
    """Attention over dense tensors on the paged prefill kernels: ``q`` [B, Hq, Sq, D], ``k`` / ``v`` [B, Hkv, Sk, D]
    (bf16 CUDA, D = 64 or 128, Hq a multiple of Hkv) -> [B, Hq, Sq, D].  Keys and values are laid out as pages of 16
    positions with an identity block table, so bidirectional encoders (BERT, ViT, Whisper, CLIP), cross-attention and
    cached decoders share the kernels of the serving engine; with ``causal`` query i sees keys ``<= Sk - Sq + i``."""
    _bf16c(q, "q"), _bf16c(k, "k"), _bf16c(v, "v")
    B, Hq, Sq, D = q.shape
    Hkv, Sk = k.shape[1], k.shape[2]
    if D not in (64, 128) or Hq % Hkv:
        raise ValueError("dense_attention: head size 64 or 128, query heads a multiple of KV heads")
    nb = (Sk + 15) // 16
    pad = nb * 16 - Sk

    def pages(t):
        if pad:
            t = torch.nn.functional.pad(t, (0, 0, 0, pad))
        return t.reshape(B, Hkv, nb, 16, D).permute(0, 2, 1, 3, 4).reshape(B * nb, Hkv, 16, D).contiguous()

    kp, vp = pages(k), pages(v)
    bt = torch.arange(B * nb, dtype=torch.int32, device=q.device).view(B, nb)
    lens = torch.full((B,), Sk, dtype=torch.int32, device=q.device)
    qs = torch.arange(B + 1, dtype=torch.int32, device=q.device) * Sq
    qt = q.permute(0, 2, 1, 3).reshape(B * Sq, Hq, D).contiguous()
    out = attn_prefill(qt, kp, vp, bt, lens, qs, Sq, scale=scale, causal=causal)
    return out.view(B, Sq, Hq, D).permute(0, 2, 1, 3)


def softmax_rows(x: torch.Tensor) -> torch.Tensor:
    """Softmax over the last dimension of a bf16 CUDA tensor."""
    _bf16c(x, "x")
    x = x.contiguous()
    out = torch.empty_like(x)
    n = x.shape[-1]
    lib = N.cuda_lib()
    lib.ub_softmax_rows.restype = C.c_int
    lib.ub_softmax_rows.argtypes = [N.vp, N.vp, N.i64, N.i32, N.vp]
    N.check(lib.ub_softmax_rows(x.data_ptr(), out.data_ptr(), x.numel() // n, n, _stream(x)), "ub_softmax_rows")
    return out


def attn_prefill_last_path() -> str:
    """Which kernel the last ``attn_prefill`` call ran: ``"tcgen05"`` or ``"mma.sync"``."""
    lib = N.cuda_lib()
    lib.ub_attn_prefill_last_path.restype = C.c_int
    return {1: "tcgen05", 2: "mma.sync"}.get(lib.ub_attn_prefill_last_path(), "none")


def attn_merge(o_a: torch.Tensor, lse_a: torch.Tensor, o_b: torch.Tensor, lse_b: torch.Tensor,
               out: Optional[torch.Tensor] = None, lse_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Combine two attention partials over disjoint key sets.  o_*: [T, Hq, D] contiguous, lse_*: [T, Hq]."""
    if out is None:
        out = torch.empty_like(o_a)
    lib = N.cuda_lib()
    lib.ub_attn_merge.restype = C.c_int
    lib.ub_attn_merge.argtypes = [N.vp, N.vp, N.vp, N.vp, N.vp, N.vp, N.i64, N.i32, N.vp]
    rows = o_a.shape[0] * o_a.shape[1]
    N.check(lib.ub_attn_merge(o_a.data_ptr(), lse_a.data_ptr(), o_b.data_ptr(), lse_b.data_ptr(), out.data_ptr(),
                              _p(lse_out), rows, o_a.shape[-1], _stream(o_a)), "ub_attn_merge")
    return out


# ---------------------------------------------------------------------------------------------
# Sampling
# ---------------------------------------------------------------------------------------------
def sample(logits: torch.Tensor, *, temperature: Optional[torch.Tensor] = None, top_p: Optional[torch.Tensor] = None,
           top_k: Optional[torch.Tensor] = None, rep_penalty: Optional[torch.Tensor] = None,
           prev_ids: Optional[torch.Tensor] = None, seed: int = 0, step: int = 0, vocab_offset: int = 0,
           out_ids: Optional[torch.Tensor] = None, out_vals: Optional[torch.Tensor] = None,
           return_vals: bool = False, candidates: int = 0, id_map: Optional[torch.Tensor] = None,
           stats: bool = False, target: Optional[torch.Tensor] = None):
    """Greedy when ``temperature`` is None (or <= 0 for a row); otherwise temperature / top-k / top-p.

    Vocabulary-parallel draws run in two stages.  ``candidates = k`` (on every shard, with ``vocab_offset``): returns
    ``(vals [B, k] fp32, ids [B, k] int32)``, the row's best entries after penalty and temperature, instead of drawing.
    ``id_map`` (identical on every rank): ``logits`` are the gathered fp32 candidates ``[B, world * k]`` and ``id_map``
    their global ids; the usual top-k / top-p / draw runs over them and returns global ids.

    Whole-vocabulary (temperature only) draws over shards: ``stats=True`` returns ``[B, 2]`` fp32 (the shard's largest
    scaled logit, the sum of ``exp(logit - max)``) instead of drawing; ``target`` ([B] fp32, in those units, negative =
    another shard draws) makes the shard that owns the draw pick the token, the others return -1."""
    if logits.dim() != 2 or logits.stride(1) != 1:
        raise ValueError("logits must be [B, V] with contiguous rows")
    if logits.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError("logits must be bf16 or fp32")
    B, V = logits.shape
    if out_ids is None:
        out_ids = torch.empty(B, dtype=torch.int32, device=logits.device)
    if return_vals and out_vals is None:
        out_vals = torch.empty(B, dtype=torch.float32, device=logits.device)
    a = N.UbSampleArgs()
    a.logits, a.ld, a.logits_f32 = logits.data_ptr(), logits.stride(0), int(logits.dtype == torch.float32)
    a.out_ids, a.out_vals = out_ids.data_ptr(), _p(out_vals)
    a.temperature, a.top_p, a.top_k, a.rep_penalty = _p(temperature), _p(top_p), _p(top_k), _p(rep_penalty)
    if prev_ids is not None:
        a.prev_ids, a.prev_ld = prev_ids.data_ptr(), prev_ids.shape[1]
    a.seed, a.step, a.B, a.V, a.vocab_offset = seed & (2**64 - 1), step, B, V, vocab_offset
    a.err = err_word(logits.device).data_ptr()
    cv = ci = None
    if candidates:
        cv = torch.empty(B, candidates, dtype=torch.float32, device=logits.device)
        ci = torch.empty(B, candidates, dtype=torch.int32, device=logits.device)
        a.cand_vals, a.cand_ids, a.cand_k = cv.data_ptr(), ci.data_ptr(), candidates
    if id_map is not None:
        if id_map.dtype != torch.int32 or id_map.shape != logits.shape or not id_map.is_contiguous() or \
                logits.dtype != torch.float32 or not logits.is_contiguous():
            raise ValueError("id_map: int32, contiguous, same shape as the contiguous fp32 candidate values")
        a.id_map = id_map.data_ptr()
    st = None
    if stats:
        st = torch.empty(B, 2, dtype=torch.float32, device=logits.device)
        a.stats_out = st.data_ptr()
    if target is not None:
        a.target_in = target.data_ptr()
    N.check(N.cuda_lib().ub_sample(C.byref(a), _stream(logits)), "ub_sample")
    if stats:
        return st
    if candidates:
        return cv, ci
    return (out_ids, out_vals) if return_vals else out_ids


def vocab_shard_targets(maxes: torch.Tensor, masses: torch.Tensor, uniform: torch.Tensor):
    """Where a draw from the whole vocabulary falls when the vocabulary is cut into shards.  ``maxes`` / ``masses``
    ([B, W] fp32: every shard's largest scaled logit and its sum of ``exp(logit - max)``, as ``sample(stats=True)`` reports
    them) and the row's uniform number give ``(owner [B], target [B])``: the shard whose running mass passes
    ``uniform * total`` (shards in vocabulary order, like the single-kernel inverse CDF) and the target inside that shard
    in the shard's own units."""
    gmax = maxes.max(dim=1, keepdim=True).values
    mass = masses * torch.exp(maxes - gmax)
    cum = mass.cumsum(dim=1)
    tgt = uniform * cum[:, -1]
    owner = (cum > tgt[:, None]).float().argmax(dim=1)
    owner = torch.where(cum[:, -1] > tgt, owner, torch.full_like(owner, maxes.shape[1] - 1))
    before = (cum - mass).gather(1, owner[:, None])[:, 0]
    local = (tgt - before) * torch.exp(gmax[:, 0] - maxes.gather(1, owner[:, None])[:, 0])
    return owner, local.clamp_min(0.0)


def argmax_merge(vals: torch.Tensor, ids: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """vals/ids [world, B] per-shard greedy winners -> global winners [B]."""
    world, B = vals.shape
    if out is None:
        out = torch.empty(B, dtype=torch.int32, device=vals.device)
    lib = N.cuda_lib()
    lib.ub_argmax_merge.restype = C.c_int
    lib.ub_argmax_merge.argtypes = [N.vp, N.vp, N.i32, N.i32, N.vp, N.vp]
    N.check(lib.ub_argmax_merge(vals.data_ptr(), ids.data_ptr(), world, B, out.data_ptr(), _stream(vals)),
            "ub_argmax_merge")
    return out


# ---------------------------------------------------------------------------------------------
# Element-wise
# ---------------------------------------------------------------------------------------------
def embed_gather(ids: torch.Tensor, table: torch.Tensor, scale: float = 1.0,
                 out: Optional[torch.Tensor] = None) -> torch.Tensor:
    _bf16c(table, "table")
    if ids.dtype != torch.int32:
        ids = ids.to(torch.int32)
    ids = ids.contiguous()
    T = ids.numel()
    V, H = table.shape
    if out is None:
        out = torch.empty((T, H), dtype=torch.bfloat16, device=table.device)
    lib = N.cuda_lib()
    lib.ub_embed_gather.restype = C.c_int
    lib.ub_embed_gather.argtypes = [N.vp, N.vp, N.vp, N.i32, N.i32, N.i32, N.f32, N.vp, N.vp]
    N.check(lib.ub_embed_gather(ids.data_ptr(), table.data_ptr(), out.data_ptr(), T, H, V, scale,
                                err_word(table.device).data_ptr(), _stream(table)), "ub_embed_gather")
    return out


def act_mul(gate_up: torch.Tensor, act: str = "silu", out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``act(gate) * up`` for gate_up [..., 2*I] (gate first)."""
    _bf16c(gate_up, "gate_up")
    gate_up = gate_up.contiguous()
    I = gate_up.shape[-1] // 2
    T = gate_up.numel() // (2 * I)
    if out is None:
        out = torch.empty((*gate_up.shape[:-1], I), dtype=torch.bfloat16, device=gate_up.device)
    lib = N.cuda_lib()
    lib.ub_act_mul.restype = C.c_int
    lib.ub_act_mul.argtypes = [N.vp, N.vp, N.i64, N.i32, N.i32, N.vp]
    N.check(lib.ub_act_mul(gate_up.data_ptr(), out.data_ptr(), T, I, N.ACT[act], _stream(gate_up)), "ub_act_mul")
    return out


def eltwise(x: torch.Tensor, act: Optional[str], alpha: float = 1.0, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    _bf16c(x, "x")
    x = x.contiguous()
    if out is None:
        out = torch.empty_like(x)
    lib = N.cuda_lib()
    lib.ub_eltwise.restype = C.c_int
    lib.ub_eltwise.argtypes = [N.vp, N.vp, N.i64, N.i32, N.f32, N.vp]
    N.check(lib.ub_eltwise(x.data_ptr(), out.data_ptr(), x.numel(), N.ACT[act], alpha, _stream(x)), "ub_eltwise")
    return out


def add(a: torch.Tensor, b: torch.Tensor, sa: float = 1.0, sb: float = 1.0,
        out: Optional[torch.Tensor] = None) -> torch.Tensor:
    _bf16c(a, "a"), _bf16c(b, "b")
    a, b = a.contiguous(), b.contiguous()
    if a.shape != b.shape:
        raise ValueError("add: shapes differ")
    if out is None:
        out = torch.empty_like(a)
    lib = N.cuda_lib()
    lib.ub_add.restype = C.c_int
    lib.ub_add.argtypes = [N.vp, N.vp, N.vp, N.i64, N.f32, N.f32, N.vp]
    N.check(lib.ub_add(a.data_ptr(), b.data_ptr(), out.data_ptr(), a.numel(), sa, sb, _stream(a)), "ub_add")
    return out


def l2_normalize(x: torch.Tensor, eps: float = 1e-12) -> torch.Tensor:
    _bf16c(x, "x")
    x = x.contiguous()
    out = torch.empty_like(x)
    H = x.shape[-1]
    lib = N.cuda_lib()
    lib.ub_l2_normalize.restype = C.c_int
    lib.ub_l2_normalize.argtypes = [N.vp, N.vp, N.i32, N.i32, N.f32, N.vp]
    N.check(lib.ub_l2_normalize(x.data_ptr(), out.data_ptr(), x.numel() // H, H, eps, _stream(x)), "ub_l2_normalize")
    return out


# ------------------------------------------------------------------------------------------------
# Mixture of experts
# ------------------------------------------------------------------------------------------------
class MoeRouting:
    """Device-side routing state of one MoE layer call (all int32 / fp32 tensors, sized from T, K, E)."""

    __slots__ = ("T", "K", "E", "tile_tokens", "max_tiles", "topk_ids", "topk_w", "counts", "offsets", "sorted_rows",
                 "row_slot", "tiles", "shared_gate")

    def __init__(self, T: int, K: int, E: int, tile_tokens: int, device, shared_gate: bool = False):
        self.T, self.K, self.E, self.tile_tokens = T, K, E, tile_tokens
        self.max_tiles = (T * K + tile_tokens - 1) // tile_tokens + E
        i32 = dict(dtype=torch.int32, device=device)
        self.topk_ids = torch.empty(T, K, **i32)
        self.topk_w = torch.empty(T, K, dtype=torch.float32, device=device)
        self.counts = torch.empty(E, **i32)
        self.offsets = torch.empty(E + 1, **i32)
        self.sorted_rows = torch.empty(T * K, **i32)
        self.row_slot = torch.empty(T * K, **i32)
        self.tiles = torch.empty(self.max_tiles, 4, **i32)
        self.shared_gate = torch.empty(T, dtype=torch.float32, device=device) if shared_gate else None


def moe_tile_tokens(T: int, K: int, E: int) -> int:
    """Token tile for the grouped GEMM: the power of two covering the mean rows per expert, 16..128."""
    avg = max(1, (T * K + E - 1) // E)
    tn = 16
    while tn < avg and tn < 128:
        tn <<= 1
    return tn


def moe_route(x: Optional[torch.Tensor], router_w: Optional[torch.Tensor], top_k: int, *, norm_topk: bool = True,
              logits: Optional[torch.Tensor] = None, weight_scale: float = 1.0, tile_tokens: int = 0,
              round_logits_bf16: bool = True, routing: Optional[MoeRouting] = None, expert_lo: int = 0,
              num_local_experts: int = 0, router_b: Optional[torch.Tensor] = None, correction: Optional[torch.Tensor] = None,
              groups: int = 1, keep_groups: int = 1, shared_w: Optional[torch.Tensor] = None, shared_gate: bool = False,
              num_experts: Optional[int] = None) -> MoeRouting:
    """Router GEMV (+ bias) + top-k + softmax weights + expert sort + grouped-GEMM tile table, two launches.  ``x`` may be
    bf16 or an fp32 residual stream, whatever the type of the router.

    ``expert_lo`` / ``num_local_experts`` restrict the sort to the experts of this rank (expert parallelism): pairs
    routed to other ranks get ``row_slot = -1`` and take no part in the grouped GEMMs.

    ``correction`` ([E]) and / or ``groups``: experts are chosen by softmax + correction within the ``keep_groups`` best groups of
    neighbours, and weighted by their softmax values.  ``shared_w`` ([H]): ``routing.shared_gate[t] = sigmoid(x[t] . shared_w)``;
    with given ``logits`` and ``shared_gate`` the gates are those of the column after the experts'.  ``num_experts``: columns
    of ``logits`` that are experts (the first ones; default all)."""
    if router_w is not None:
        _elem("moe_route x", x), _elem("moe_route router", router_w, router_b, correction, shared_w)
        T, H = x.shape
        if router_w.shape[1] != H or not x.is_contiguous() or not router_w.is_contiguous():
            raise ValueError("moe_route: x [T, H] and router [E, H] must be contiguous")
        E = router_w.shape[0]
        dev = x.device
    else:
        T, cols = logits.shape
        E = cols - int(shared_gate) if num_experts is None else num_experts
        H = 0
        dev = logits.device
        if not logits.is_contiguous() or cols < E + int(shared_gate) or shared_w is not None:
            raise ValueError("moe_route: contiguous logits [T, experts (+ gate)]")
    tn = tile_tokens or moe_tile_tokens(T, top_k, E)
    gated = shared_w is not None or shared_gate
    r = routing if routing is not None else MoeRouting(T, top_k, E, tn, dev, gated)
    for t, n in ((correction, E), (shared_w, H)):
        if t is not None and (t.numel() != n or not t.is_contiguous()):
            raise ValueError("moe_route: correction [E] and shared_w [H]")
    a = N.UbMoeRouteArgs()
    a.logits, a.x, a.router_w = _p(logits), _p(x) if router_w is not None else None, _p(router_w)
    a.topk_ids, a.topk_w = r.topk_ids.data_ptr(), r.topk_w.data_ptr()
    a.expert_counts, a.expert_offsets = r.counts.data_ptr(), r.offsets.data_ptr()
    a.sorted_rows, a.row_slot, a.tiles = r.sorted_rows.data_ptr(), r.row_slot.data_ptr(), r.tiles.data_ptr()
    a.err = err_word(dev).data_ptr()
    a.logits_f32 = 1 if (logits is not None and logits.dtype == torch.float32) else 0
    a.T, a.E, a.K, a.H = T, E, top_k, H
    a.norm_topk = 1 if norm_topk else 0
    a.round_logits_bf16 = 1 if round_logits_bf16 else 0
    a.weight_scale = weight_scale
    if router_w is not None:
        a.router_b, a.x_f32, a.router_f32 = _p(router_b), int(x.dtype == torch.float32), int(router_w.dtype == torch.float32)
    a.tile_tokens, a.max_tiles = r.tile_tokens, r.max_tiles
    a.expert_lo, a.num_local_experts = expert_lo, num_local_experts
    a.correction, a.groups, a.keep_groups = _p(correction), groups, keep_groups
    if correction is not None:
        a.router_f32 = int(correction.dtype == torch.float32)
    a.shared_w, a.shared_gate = _p(shared_w), _p(r.shared_gate if gated else None)
    a.ld_logits = 0 if router_w is not None else logits.shape[1]
    N.check(N.cuda_lib().ub_moe_route(C.byref(a), torch.cuda.current_stream(dev).cuda_stream), "ub_moe_route")
    return r


def moe_gather(x: torch.Tensor, r: MoeRouting, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out[slot] = x[sorted_rows[slot] // K]``: activations in expert order."""
    f32 = _elem("moe_gather", x, out)
    T, H = x.shape
    if out is None:
        out = torch.empty(T * r.K, H, dtype=x.dtype, device=x.device)
    lib = N.cuda_lib()
    gather = lib.ub_moe_gather_f32 if f32 else lib.ub_moe_gather
    gather.restype = C.c_int
    gather.argtypes = [N.vp, N.vp, N.vp, N.i32, N.i32, N.i32, N.vp]
    N.check(gather(x.data_ptr(), r.sorted_rows.data_ptr(), out.data_ptr(), T * r.K, r.K, H, _stream(x)),
            "ub_moe_gather")
    return out


def gather_rows(x: torch.Tensor, rows: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out[i] = x[rows[i]]`` for int32 ``rows`` (negative entries leave ``out[i]`` untouched)."""
    _bf16c(x, "x")
    H = x.shape[1]
    n = rows.numel()
    if out is None:
        out = torch.empty(n, H, dtype=torch.bfloat16, device=x.device)
    lib = N.cuda_lib()
    lib.ub_moe_gather.restype = C.c_int
    lib.ub_moe_gather.argtypes = [N.vp, N.vp, N.vp, N.i32, N.i32, N.i32, N.vp]
    N.check(lib.ub_moe_gather(x.data_ptr(), rows.data_ptr(), out.data_ptr(), n, 1, H, _stream(x)), "ub_moe_gather")
    return out


def moe_combine(y: torch.Tensor, r: MoeRouting, residual: Optional[torch.Tensor] = None,
                out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``out[t] = residual[t] + sum_k w[t,k] * y[row_slot[t,k]]``."""
    _bf16c(y, "y")
    H = y.shape[1]
    if out is None:
        out = torch.empty(r.T, H, dtype=torch.bfloat16, device=y.device)
    lib = N.cuda_lib()
    lib.ub_moe_combine.restype = C.c_int
    lib.ub_moe_combine.argtypes = [N.vp, N.vp, N.vp, N.vp, N.vp, N.i32, N.i32, N.i32, N.vp]
    N.check(lib.ub_moe_combine(y.data_ptr(), r.row_slot.data_ptr(), r.topk_w.data_ptr(), _p(residual), out.data_ptr(),
                               r.T, r.K, H, _stream(y)), "ub_moe_combine")
    return out


def moe_combine_num_ctas(T: int, H: int) -> int:
    lib = N.cuda_lib()
    lib.ub_moe_combine_num_ctas.restype = C.c_int
    lib.ub_moe_combine_num_ctas.argtypes = [N.i32, N.i32]
    return lib.ub_moe_combine_num_ctas(T, H)


def moe_combine_rs(y: torch.Tensor, r: MoeRouting, rs: dict) -> None:
    """Combine fused with the reduce-scatter: partial rows go into the owners' receive slots (``rs`` as for
    ``gemm_tn``: world, rank, rows_per_rank, peer_out, peer_flag, local_count); the last CTA signals each peer once."""
    _bf16c(y, "y")
    H = y.shape[1]
    W = rs["world"]
    outs = (C.c_void_p * W)(*[(int(p) or None) for p in rs["peer_out"][:W]])
    flags = (C.c_void_p * W)(*[int(p) for p in rs["peer_flag"][:W]])
    lib = N.cuda_lib()
    lib.ub_moe_combine_rs.restype = C.c_int
    lib.ub_moe_combine_rs.argtypes = [N.vp, N.vp, N.vp, N.i32, N.i32, N.i32, N.i32, N.i32, N.i32, N.vp, N.vp, N.vp, N.vp, N.vp]
    N.check(lib.ub_moe_combine_rs(y.data_ptr(), r.row_slot.data_ptr(), r.topk_w.data_ptr(), r.T, r.K, H, W, rs["rank"],
                                  rs["rows_per_rank"], C.cast(outs, C.c_void_p), C.cast(flags, C.c_void_p),
                                  rs["local_count"], rs.get("local_out") or None, _stream(y)),
            "ub_moe_combine_rs")


class MoeDispatch:
    """Device-side state of one sparse expert-parallel MoE call on one rank: the routing of this rank's own ``R`` rows
    (``route``), the send scratch, and what the receive side builds (row order, return addresses, tile table).  The
    attributes ``tiles`` / ``max_tiles`` / ``tile_tokens`` make it usable where ``grouped_gemm`` expects a routing."""

    def __init__(self, R: int, K: int, E: int, world: int, device):
        self.R, self.K, self.E, self.world = R, K, E, world
        self.experts_local = E // world
        self.cap = R * K
        self.slots = world * self.cap                         # = T * K: every pair of the step could land here
        self.tile_tokens = moe_tile_tokens(R * world, K, E)
        self.max_tiles = (self.slots + self.tile_tokens - 1) // self.tile_tokens + self.experts_local
        i32 = dict(dtype=torch.int32, device=device)
        self.route = MoeRouting(R, K, E, self.tile_tokens, device)
        self.send_slot = torch.empty(R * K, **i32)
        self.send_counts = torch.empty(E, **i32)
        self.sorted_rows = torch.empty(self.slots, **i32)
        self.slot_meta = torch.empty(self.slots, 4, **i32)
        self.counts = torch.empty(self.experts_local, **i32)
        self.offsets = torch.empty(self.experts_local + 1, **i32)
        self.tiles = torch.empty(self.max_tiles, 4, **i32)


def moe_dispatch(x: torch.Tensor, d: MoeDispatch, comm: dict) -> None:
    """F5 send side: rows of ``x`` ([R, H], this rank's tokens, routed in ``d.route``) go to the ranks of their
    experts.  ``comm``: world, rank, peer_rows / peer_meta / peer_counts / peer_flag (one address per rank) and
    local_count, as ``FusedComm.moe_dispatch_args`` builds them."""
    _bf16c(x, "x")
    a = N.UbMoeDispatchArgs()
    a.x, a.topk_ids, a.topk_w = x.data_ptr(), d.route.topk_ids.data_ptr(), d.route.topk_w.data_ptr()
    a.send_slot, a.send_counts = d.send_slot.data_ptr(), d.send_counts.data_ptr()
    for r in range(comm["world"]):
        a.peer_rows[r], a.peer_meta[r] = comm["peer_rows"][r], comm["peer_meta"][r]
        a.peer_counts[r], a.peer_flag[r] = comm["peer_counts"][r], comm["peer_flag"][r]
    a.local_count = comm["local_count"]
    a.err = err_word(x.device).data_ptr()
    a.R, a.K, a.H, a.E = d.R, d.K, x.shape[1], d.E
    a.world, a.rank, a.experts_local, a.cap = comm["world"], comm["rank"], d.experts_local, d.cap
    lib = N.cuda_lib()
    lib.ub_moe_dispatch.restype = C.c_int
    N.check(lib.ub_moe_dispatch(C.byref(a), _stream(x)), "ub_moe_dispatch")


def moe_recv_build(d: MoeDispatch, comm: dict, device) -> None:
    """F5 receive side: waits (bounded, on the device) for every source's arrival, then orders the received rows by
    expert: ``d.sorted_rows`` (receive row per slot), ``d.slot_meta`` (return address), ``d.tiles``."""
    a = N.UbMoeRecvArgs()
    a.counts, a.meta, a.flag, a.round = comm["counts"], comm["meta"], comm["flag"], comm["round"]
    a.sorted_rows, a.slot_meta = d.sorted_rows.data_ptr(), d.slot_meta.data_ptr()
    a.expert_counts, a.expert_offsets, a.tiles = d.counts.data_ptr(), d.offsets.data_ptr(), d.tiles.data_ptr()
    a.err = err_word(device).data_ptr()
    a.world, a.experts_local, a.cap = d.world, d.experts_local, d.cap
    a.tile_tokens, a.max_tiles = d.tile_tokens, d.max_tiles
    lib = N.cuda_lib()
    lib.ub_moe_recv_build.restype = C.c_int
    N.check(lib.ub_moe_recv_build(C.byref(a), torch.cuda.current_stream(device).cuda_stream), "ub_moe_recv_build")


def moe_combine_push(y: torch.Tensor, d: MoeDispatch, comm: dict) -> None:
    """F6: ``y[slot] * weight`` goes into slot ``[k][row]`` of the token owner's combine area; one arrival per rank."""
    _bf16c(y, "y")
    a = N.UbMoeReturnArgs()
    a.y, a.slot_meta, a.expert_offsets = y.data_ptr(), d.slot_meta.data_ptr(), d.offsets.data_ptr()
    for r in range(comm["world"]):
        a.peer_comb[r], a.peer_flag[r] = comm["peer_comb"][r], comm["peer_flag"][r]
    a.local_count = comm["local_count"]
    a.err = err_word(y.device).data_ptr()
    a.R, a.K, a.H, a.world, a.experts_local = d.R, d.K, y.shape[1], comm["world"], d.experts_local
    lib = N.cuda_lib()
    lib.ub_moe_combine_push.restype = C.c_int
    N.check(lib.ub_moe_combine_push(C.byref(a), d.slots, _stream(y)), "ub_moe_combine_push")


def grouped_gemm(x_sorted: torch.Tensor, w: torch.Tensor, r: MoeRouting, *, dual_rows: int = 0, act: Optional[str] = None,
                 out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Expert-grouped GEMM: rows of ``x_sorted`` that belong to expert e multiply ``w[e]`` (``[E, rows, K]``).

    ``dual_rows = I``: ``w[e]`` is ``[2I, K]`` (gate rows then up rows) and the result is ``act(gate) * up``.
    """
    if w.dim() != 3 or not w.is_contiguous():
        raise ValueError("grouped_gemm takes contiguous weights [E, rows, K]")
    E, rows, Kd = w.shape
    g = {"tiles": r.tiles.data_ptr(), "max_tiles": r.max_tiles, "w_rows": rows, "tile_tokens": r.tile_tokens}
    n_out = dual_rows if dual_rows else rows
    f32 = _elem("grouped_gemm", x_sorted, w, out)
    if out is None:
        out = torch.empty(x_sorted.shape[0], n_out, dtype=x_sorted.dtype, device=x_sorted.device)
    w2 = w.view(E * rows, Kd)
    if dual_rows:
        return gemm_tn(x_sorted, w2, dual_rows=dual_rows, act=act, out=out, grouped=g)
    # non-dual: N is the per-expert row count while w2 has E*rows rows
    return _gemm_grouped_plain(x_sorted, w2, rows, act, out, g, f32)


def _gemm_grouped_plain(x, w2, rows, act, out, g, f32=False):
    a = N.UbGemmArgs()
    a.x, a.w, a.out = x.data_ptr(), w2.data_ptr(), out.data_ptr()
    a.err = err_word(x.device).data_ptr()
    a.M, a.N, a.K = x.shape[0], rows, x.shape[1]
    a.ldx, a.ldw, a.ldo = x.stride(0), w2.stride(0), out.stride(0)
    a.act = N.ACT[act]
    a.w_rows_total = w2.shape[0]
    a.out_scale = 1.0
    a.grp_tiles, a.grp_max_tiles, a.grp_w_rows, a.tile_tokens = g["tiles"], g["max_tiles"], g["w_rows"], g["tile_tokens"]
    lib = N.cuda_lib()
    N.check((lib.ub_gemm_f32 if f32 else lib.ub_gemm_tn)(C.byref(a), _stream(x)), "ub_gemm_tn(grouped)")
    return out
