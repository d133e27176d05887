"""Tasadra on the GPU: each mechanism's kernel alone and the serving engine on them, against the plain statement."""
import dataclasses
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import tasadra_cases as C
import tasadra_plain as P
from test_gpu_bakasun import DTYPES, _close, _i32, _pad, _paged, _plant, _portions, _r8, _rand, _steps

pytestmark = pytest.mark.gpu

LENS = [75, 5, 1, 64, 33, 16]
CUTS = [[75], [2], [1], [33, 1, 2, 14], [1, 17, 1], [16]]


# ------------------------------------------------------------------------------------------------
# sublayer input: residual, depth average, Dynamic Tanh, token shift
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,n,tile", [(8, 0, 0), (50, 3, 1), (136, 1, 7), (1000, 6, 16), (1032, 2, 3), (9000, 0, 2)])
def test_stream_in_with_shift(dtype, H, n, tile):
    """Portions of several sequences, from a state row into another, against whole ones: tiles of any size, one token beside
    longer portions, rows of the stream that are averaged over depth."""
    from unillm_b200.ops import cuda_ops as K

    Hp, scale, alpha = _r8(H), 0.6, 0.7
    w, b, mu = 1 + _rand(H, seed=1, scale=0.3), _rand(H, seed=2, scale=0.3), _rand(H, seed=3, scale=0.7)
    mix = _rand(n + 1, seed=4, dtype=torch.float32)
    dev = lambda t: _pad(t, Hp).to("cuda", dtype).contiguous()
    f32 = lambda t: _pad(t, Hp).cuda().contiguous()
    xs = [{"x": _rand(m, H, seed=10 + s, dtype=torch.float32), "y": _rand(m, H, seed=30 + s), "X": _rand(n, m, H, seed=50 + s, dtype=torch.float32)}
          for s, m in enumerate(LENS)]
    state = torch.full((2 * len(LENS), Hp), 77.0, device="cuda")               # never to be read before it is written
    half, got, res, run = [0] * len(LENS), [[] for _ in LENS], [[] for _ in LENS], [[] for _ in LENS]
    for step in _steps(LENS, CUTS):
        order, parts = _portions(step, half)
        rows = sum(e - a for _, a, e in order)
        cat = lambda k, dim=0: torch.cat([xs[s][k].narrow(dim, a, e - a) for s, a, e in order], dim)
        x_res, x_out = (torch.full((rows, Hp), 5.0, device="cuda") for _ in range(2))
        kw = dict(streams=f32(cat("X", 1)) if n else None, mix=mix.cuda())
        out = K.stream_in(parts, dev(w), dev(b), alpha, x=f32(cat("x")), y=dev(cat("y")), scale=scale, x_res=x_res, x_out=x_out, shift=dev(mu),
                          shift_state=state, tile=tile, **kw)
        assert out[:, H:].abs().sum() == 0 and x_out[:, H:].abs().sum() == 0
        r = 0
        for s, a, e in order:
            for keep, t in ((got, out), (res, x_res), (run, x_out)):
                keep[s].append(t[r:r + e - a, :H].cpu())
            r += e - a
    for s, t in enumerate(xs):
        x = t["x"].double() + scale * t["y"].double()
        mean = P.depth_average([*t["X"].double(), x], mix.double())
        h = P.dyt(mean, {"n": w.double(), "n.b": b.double(), "n.alpha": alpha}, "n")
        _close(torch.cat(res[s]), x, torch.float32)
        _close(torch.cat(run[s]), mean, torch.float32)
        _close(torch.cat(got[s]), P.token_shift(h, mu.double()), dtype)
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,T", [(8, 1), (50, 7), (1032, 20), (4096, 700)])
def test_stream_in_of_rows_that_stand_alone(dtype, H, T):
    """The embedding's rows, a stream changed in place, and picked rows, which leave the stream as it is."""
    from unillm_b200.ops import cuda_ops as K

    Hp, alpha = _r8(H), 1.3
    w, b, table = 1 + _rand(H, seed=1, scale=0.3), _rand(H, seed=2, scale=0.3), _rand(31, H, seed=3)
    ids = torch.randint(0, 31, (T,), generator=torch.Generator().manual_seed(4)).to(torch.int32)
    dev = lambda t: _pad(t, Hp).to("cuda", dtype).contiguous()
    norm = lambda x: P.dyt(x, {"n": w.double(), "n.b": b.double(), "n.alpha": alpha}, "n")
    x = torch.empty(T, Hp, device="cuda")
    out = K.stream_in((), dev(w), dev(b), alpha, ids=ids.cuda(), table=dev(table), x_res=x)
    assert torch.equal(x[:, :H].cpu(), table[ids.long()].float())
    _close(out[:, :H], norm(table[ids.long()].double()), dtype)
    y = _rand(T, H, seed=5)
    want = table[ids.long()].double() - 0.25 * y.double()
    pick, before = torch.tensor([T - 1, 0, T // 2]), x.clone()
    mix, old = torch.tensor([0.5, -1.5]), _rand(1, T, H, seed=6, dtype=torch.float32)
    few = K.stream_in((), dev(w), dev(b), alpha, x=x, y=dev(y), scale=-0.25, rows=_i32(pick), streams=_pad(old, Hp).cuda(), mix=mix.cuda())
    assert torch.equal(x, before)
    _close(few[:, :H], norm(0.5 * old[0].double() - 1.5 * want)[pick], dtype)
    out = K.stream_in((), dev(w), dev(b), alpha, x=x, y=dev(y), scale=-0.25, x_out=x)
    _close(x[:, :H], want, torch.float32)
    _close(out[:, :H], norm(want), dtype)
    K.check_device_errors()


# ------------------------------------------------------------------------------------------------
# rows for the attention kernels
# ------------------------------------------------------------------------------------------------
POS, SLOTS = [0, 1, 15, 16, 17, 300, 299, 1000, 3], [40, 0, 111, -1, 16, 15, 3, 77, 50]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,d,dv,dims", [(3, 1, 10, 14, 6), (4, 2, 24, 40, 16), (2, 2, 20, 18, 20), (18, 3, 72, 136, 36), (5, 5, 128, 64, 96),
                                              (8, 1, 256, 8, 254), (2, 1, 64, 64, 64), (1, 1, 16, 256, 16)])
def test_turned_values_and_yarn(dtype, hq, hkv, d, dv, dims):
    """Head norms, YaRN frequencies with their gain on the rotated part alone, values cached turned by their position."""
    from unillm_b200.ops import cuda_ops as K
    from unillm_b200.precompute import rope_gain, rope_inv_freq

    T, bs, nb, dp, vp = 9, 16, 7, _r8(d), _r8(dv)
    q, k, v = _rand(T, hq, d, seed=1, scale=2.0), _rand(T, hkv, d, seed=2), _rand(T, hkv, dv, seed=3)
    qw, kw = 1 + _rand(d, seed=4, scale=0.4), 1 + _rand(d, seed=5, scale=0.4)
    pos, slots = torch.tensor(POS, dtype=torch.int32), torch.tensor(SLOTS, dtype=torch.int32)
    dev = lambda t: t.to("cuda", dtype).contiguous()
    rows = torch.cat([_pad(q, dp).flatten(1), _pad(k, dp).flatten(1), _pad(v, vp).flatten(1)], 1)
    wide = dev(torch.cat([rows, torch.full((T, 24), 7.0)], 1))
    kc, vc = dev(torch.full((nb, hkv, bs, dp), 5.0)), dev(torch.full((nb, hkv, bs, vp), 5.0))
    yarn = (6.0, 60.0, 4.0, 0.5)
    K.rope_kv_append(wide[:, :rows.shape[1]], pos.cuda(), slots.cuda(), kc, vc, num_q_heads=hq, num_kv_heads=hkv, head_dim=dp, v_head_dim=vp,
                     rotary_dim=dims, inv_freq=rope_inv_freq(dims, 700.0, yarn=yarn).cuda(), gain=rope_gain(yarn), norm_dim=d, norm_eps=1e-3,
                     q_norm_w=dev(_pad(qw, dp)), k_norm_w=dev(_pad(kw, dp)), k_cache_only=True, v_inv_freq=rope_inv_freq(dv, 700.0).cuda())
    rot = {"base": 700.0, "dims": dims, "scaling": dict(zip(("factor", "original", "fast", "slow"), yarn))}
    want = lambda x, w: P.turn(P.rms(x.double(), 1e-3) * w.double(), pos, *P.yarn_frequencies(rot))
    tol = dict(f32_tol=3e-4)                         # angles of hundreds of radians in 32 bits
    _close(wide[:, :hq * dp].unflatten(1, (hq, dp))[..., :d], want(q, qw), dtype, **tol)
    assert (wide[:, rows.shape[1]:] == 7.0).all()
    keep = slots >= 0
    at = slots[keep].long()
    kk, vv = (c.transpose(1, 2).flatten(0, 1)[at.cuda()] for c in (kc, vc))
    _close(kk[..., :d], want(k, kw)[keep], dtype, **tol)
    _close(vv[..., :dv], P.turn(v.double(), pos, P.value_frequencies(700.0, dv))[keep], dtype, **tol)
    assert kk[..., d:].abs().sum() == 0 and vv[..., dv:].abs().sum() == 0
    assert int((vc.transpose(1, 2).flatten(0, 1) == 5.0).all(-1).all(-1).sum()) == nb * bs - int(keep.sum())       # no other slot was touched
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dim,dv", [(1, 1, 8, 8), (4, 2, 16, 40), (10, 1, 72, 128), (6, 3, 64, 128), (2, 2, 128, 256)])
def test_rows_of_two_maps(dtype, H, G, dim, dv):
    from unillm_b200.ops import cuda_ops as K

    T, bs, nb = 9, 16, 7
    q, k, v = _rand(T, H, 2, dim, seed=1), _rand(T, G, 2, dim, seed=2), _rand(T, G, dv, seed=3)
    dev = lambda t: t.to("cuda", dtype).contiguous()
    wide = dev(torch.cat([q.flatten(1), k.flatten(1), v.flatten(1), torch.full((T, 16), 7.0, dtype=torch.bfloat16)], 1))
    kc, vc = dev(torch.full((nb, G, bs, 2 * dim), 5.0)), dev(torch.full((nb, G, bs, dv), 5.0))
    slots = torch.tensor(SLOTS, dtype=torch.int32)
    n = wide.shape[1] - 16
    want = torch.zeros(T, H, 2, 2, dim, dtype=torch.bfloat16)
    want[:, :, 0, 0], want[:, :, 1, 1] = q[:, :, 0], q[:, :, 1]
    for own in (False, True):
        out = K.map_rows(wide[:, :n], slots.cuda() if own else None, kc if own else None, vc if own else None, num_heads=H, maps=2, dim=dim)
        assert torch.equal(out.cpu(), want.reshape(T, 2 * H, 2 * dim).to(dtype))
    keep = slots >= 0
    kk, vv = (c.transpose(1, 2).flatten(0, 1)[slots[keep].long().cuda()].cpu() for c in (kc, vc))
    assert torch.equal(kk, k.flatten(2)[keep].to(dtype)) and torch.equal(vv, v[keep].to(dtype))
    assert int((kc.transpose(1, 2).flatten(0, 1) == 5.0).all(-1).all(-1).sum()) == nb * bs - int(keep.sum())
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dv", [(1, 8), (3, 14), (5, 40), (18, 136), (4, 64), (2, 256), (9, 96), (7, 22)])
@pytest.mark.parametrize("kind", ["", "head", "element"])
def test_attention_outputs(dtype, H, dv, kind):
    """Outputs turned back and gated; two maps subtracted, normed and gated."""
    from unillm_b200.ops import cuda_ops as K
    from unillm_b200.precompute import rope_inv_freq

    T, vp = 9, _r8(dv)
    pos = torch.tensor(POS, dtype=torch.int32)
    a, g = _rand(T, 2 * H, dv, seed=1), _rand(T, H, dv, seed=2, scale=2.0)
    dev = lambda t: t.to("cuda", dtype).contiguous()
    gate = {"": None, "head": dev(torch.cat([_rand(T, 8, seed=7), _pad(g[:, :, 0], _r8(H))], 1))[:, 8:], "element": dev(_pad(g, vp).flatten(1))}[kind]
    s = 1.0 if not kind else P.sigmoid(g.double())[..., :1] if kind == "head" else P.sigmoid(g.double())
    got = K.attn_finish(dev(_pad(a[:, :H], vp).flatten(1)), vp, gate=gate, gate_kind=kind, positions=pos.cuda(), inv_freq=rope_inv_freq(dv, 700.0).cuda(),
                        dv_real=dv).unflatten(1, (H, vp))
    _close(got[..., :dv], P.turn(a[:, :H].double(), -pos, P.value_frequencies(700.0, dv)) * s, dtype, f32_tol=3e-4)
    assert got[..., dv:].abs().sum() == 0
    got = K.attn_finish(dev(_pad(a, vp).flatten(1)), vp, gate=gate, gate_kind=kind, maps=2, lam=0.6, factor=0.3, eps=1e-4, dv_real=dv).unflatten(1, (H, vp))
    pair = a.double().unflatten(1, (H, 2))
    _close(got[..., :dv], P.difference(pair[:, :, 0], pair[:, :, 1], 0.6, 0.7, 1e-4) * s, dtype)
    assert got[..., dv:].abs().sum() == 0
    K.check_device_errors()


# ------------------------------------------------------------------------------------------------
# attention in chunks, capped scores
# ------------------------------------------------------------------------------------------------
SHAPES = [(6, 3, 48, 88), (3, 1, 16, 24), (18, 1, 72, 136), (4, 4, 128, 128), (16, 2, 128, 128), (2, 1, 200, 256), (8, 2, 64, 64), (32, 1, 128, 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,d,dv", SHAPES)
@pytest.mark.parametrize("chunk,cap", [(42, 10.0), (16, None), (64, 25.0), (1, 8.0), (0, 6.0), (100, None), (128, 200.0)])
def test_attention_in_chunks(dtype, hq, hkv, d, dv, chunk, cap):
    """Prompts, portions and single tokens, on whichever kernel takes the sizes; keys that stand out just inside and just outside
    of a chunk, at page and tile borders, at the start and at the query itself; many scores far above the cap and far below it."""
    from unillm_b200.ops import cuda_ops as K

    lens, qlens, scale = [310, 5, 83, 17, 129], [310, 2, 40, 1, 1], 0.6 * d ** -0.5
    k, v, bt, fill = _paged(lens, hkv, d, dv, seed=d + chunk)
    q = [_rand(n, hq, d, seed=70 + i) for i, n in enumerate(lens)]
    c = chunk or 10 ** 6
    for s, pos in ((0, 309), (0, 256), (0, 200), (0, 127), (0, 99), (0, 64), (2, 82), (2, 60), (3, 16), (4, 128)):
        for key in (pos // c * c, pos // c * c - 1):
            if 0 <= key:
                _plant(q[s], k[s], pos, key, scale)
    for s, pos, key in ((0, 140, 127), (0, 120, 112), (0, 290, 255), (0, 70, 0), (2, 77, 63), (2, 50, 50), (1, 4, 0), (4, 127, 111)):
        _plant(q[s], k[s], pos, key, scale)
    want = [P.attend(a.double(), b.double(), x.double(), scale, chunk or None, cap) for a, b, x in zip(q, k, v)]
    kc, vc = fill(dtype)
    kw, tol = dict(scale=scale, chunk=chunk, softcap=cap or 0.0), dict(bf16_tol=3e-2)
    rows = lambda ts: torch.cat([torch.cat([x.flatten(1) for x in ts]), torch.zeros(sum(len(x) for x in ts), 24, dtype=torch.bfloat16)], 1).to(
        "cuda", dtype)[:, :hq * d].unflatten(1, (hq, d))                        # queries inside wider rows
    new = rows([a[n - m:] for a, n, m in zip(q, lens, qlens)])
    out = torch.full((new.shape[0], hq * dv + 8), 3.0, device="cuda", dtype=dtype)
    K.attn_prefill(new, kc, vc, bt.cuda(), _i32(lens), _i32([0, *torch.tensor(qlens).cumsum(0).tolist()]), max(qlens),
                   out=out[:, :hq * dv].unflatten(1, (hq, dv)), **kw)
    _close(out[:, :hq * dv].unflatten(1, (hq, dv)), torch.cat([x[n - m:] for x, n, m in zip(want, lens, qlens)]), dtype, **tol)
    assert (out[:, hq * dv:] == 3.0).all()
    if dtype == torch.bfloat16 and d == dv == 128:
        assert K.attn_prefill_last_path() == "tcgen05"
    for splits in (1, 3):
        got = K.attn_decode(rows([a[-1:] for a in q]), kc, vc, bt.cuda(), _i32(lens), splits=splits, **kw)
        _close(got, torch.cat([x[-1:] for x in want]), dtype, **tol)
    K.check_device_errors()


@pytest.mark.parametrize("chunk,cap,seqs", [(100, None, 150), (64, 12.0, 300), (0, 9.0, 300), (1, None, 260)])
@pytest.mark.parametrize("hq,hkv,d", [(8, 2, 128), (4, 2, 64)])
def test_decoding_of_many_sequences(chunk, cap, seqs, hq, hkv, d):
    """Batches large enough for the kernel with one pipeline per warp; lengths that end anywhere in a page and a chunk."""
    from unillm_b200.ops import cuda_ops as K

    lens, scale = [1 + (37 * s) % 210 for s in range(seqs)], 0.8 * d ** -0.5
    k, v, bt, fill = _paged(lens, hkv, d, d, seed=3)
    q = [_rand(1, hq, d, seed=900 + s) for s in range(seqs)]
    c = chunk or 10 ** 6
    for s, n in enumerate(lens):
        for key in ((n - 1) // c * c, (n - 1) // c * c - 1, n - 1):
            if key >= 0:
                h = (n + key) % hkv
                x = q[s][0, h * (hq // hkv)].float()
                k[s][key, h] = (x * (11.0 / (scale * x.pow(2).sum()))).to(torch.bfloat16)
    kc, vc = fill(torch.bfloat16)
    want = []
    for s, n in enumerate(lens):
        lo = (n - 1) // c * c
        p = torch.softmax(P.softcap(torch.einsum("hd,khd->hk", q[s][0].double(), k[s][lo:].double().repeat_interleave(hq // hkv, 1)) * scale, cap), -1)
        want.append(torch.einsum("hk,khd->hd", p, v[s][lo:].double().repeat_interleave(hq // hkv, 1)))
    got = K.attn_decode(torch.cat(q).cuda(), kc, vc, bt.cuda(), _i32(lens), scale=scale, chunk=chunk, softcap=cap or 0.0, splits=1)
    _close(got, torch.stack(want), torch.bfloat16, bf16_tol=3e-2)
    K.check_device_errors()


# ------------------------------------------------------------------------------------------------
# delta rule with decays per channel
# ------------------------------------------------------------------------------------------------
DELTA = [(1, 1, 8, 8, 4, 0), (3, 3, 13, 21, 1, 0), (4, 2, 20, 72, 2, 0), (4, 1, 32, 40, 3, 0), (6, 3, 64, 64, 4, 8), (2, 1, 64, 80, 5, 16),
         (3, 1, 40, 128, 4, 8), (2, 2, 128, 128, 4, 8), (4, 2, 128, 96, 4, 16), (2, 1, 100, 16, 9, 32), (2, 1, 136, 200, 4, 16), (1, 1, 256, 256, 16, 32),
         (2, 2, 192, 64, 2, 0), (1, 1, 8, 256, 3, 0), (2, 1, 256, 8, 3, 0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,taps,lanes", DELTA)
def test_delta_rule_by_channel(dtype, H, G, dk, dv, taps, lanes):
    """Convolutions, unit norms, decays per channel from none to all, recurrence, head norm and gate: portions of several
    sequences against the plain recurrence on whole ones, from a state row into another."""
    from unillm_b200.ops import cuda_ops as K

    kp, vp, C_ = _r8(dk), _r8(dv), 2 * G * _r8(dk) + H * _r8(dv)
    width = {"q": (G, dk, kp), "k": (G, dk, kp), "v": (H, dv, vp)}
    conv = {c: _rand(n, w, taps, seed=i, scale=0.6) for i, (c, (n, w, _)) in enumerate(width.items())}
    a_log, dt = _rand(H, seed=5, dtype=torch.float32) - 0.5, _rand(H, dk, seed=6, dtype=torch.float32, scale=2.0) - 1.0
    nw = 1 + _rand(dv, seed=7, dtype=torch.float32, scale=0.3)
    xs = [{c: _rand(n, h, w, seed=20 * s + i) for i, (c, (h, w, _)) in enumerate(width.items())} for s, n in enumerate(LENS)]
    for s, (x, n) in enumerate(zip(xs, LENS)):
        x["b"], x["a"] = _rand(n, H, seed=500 + s, scale=1.5), _rand(n, H, dk, seed=600 + s, dtype=torch.float32, scale=2.5)
        x["g"] = _rand(n, H, dv, seed=700 + s)
        x["a"][n // 2, :, ::2] = 40.0                           # a token at which half of the channels forget everything
        x["a"][n // 3, :, 1::2] = -30.0                         # ... and one at which the others forget nothing
        x["k"][0] *= 6                                          # and a first token that stands out
    col, ld = 16, _r8(16 + C_ + H)
    cat = torch.cat([_pad(conv[c], width[c][2], 1).flatten(0, 1) for c in "qkv"])
    taps_dev = cat.t().to("cuda", dtype).contiguous()
    state = torch.full((2 * len(LENS), H, kp, vp), 77.0, device="cuda")          # never to be read before it is written
    conv_state = torch.full((2 * len(LENS), taps - 1, C_), 77.0, device="cuda")
    half, got = [0] * len(LENS), [[] for _ in LENS]
    for step in _steps(LENS, CUTS):
        order, parts = _portions(step, half)
        rows = sum(b - a for _, a, b in order)
        proj = torch.full((rows, ld), 9.0, device="cuda", dtype=dtype)
        at = col
        for c, (_, _, p) in width.items():
            t = torch.cat([_pad(xs[s][c][a:b], p).flatten(1) for s, a, b in order])
            proj[:, at:at + t.shape[1]] = t.to("cuda", dtype)
            at += t.shape[1]
        proj[:, at:at + H] = torch.cat([xs[s]["b"][a:b] for s, a, b in order]).to("cuda", dtype)
        decay = torch.cat([_pad(xs[s]["a"][a:b], kp).flatten(1) for s, a, b in order]).cuda()
        gate = torch.cat([torch.cat([_pad(xs[s]["g"][a:b], vp).flatten(1) for s, a, b in order]), torch.zeros(rows, 8)], 1).to("cuda", dtype)
        wide = torch.full((rows, 8 + H * vp), 5.0, device="cuda", dtype=dtype)
        K.delta_mixer(proj, col, taps_dev, a_log.cuda(), _pad(dt, kp).flatten().cuda(), _pad(nw, vp).cuda(), conv_state, state, parts, kv_heads=G,
                      eps=1e-4, dk_real=dk, dv_real=dv, out=wide[:, 8:], lanes=lanes, decay=decay, gate=gate[:, :H * vp], gate_act="sigmoid")
        assert (wide[:, :8] == 5.0).all()
        out = wide[:, 8:].reshape(rows, H, vp).cpu()
        assert out[..., dv:].abs().sum() == 0
        r = 0
        for s, a, b in order:
            got[s].append(out[r:r + b - a, :, :dv])
            r += b - a
    for s, x in enumerate(xs):
        y = {c: P.silu(P.short_conv(x[c].double().flatten(1), conv[c].double().flatten(0, 1))).reshape(x[c].shape) for c in "qkv"}
        rep = lambda t: P.unit(t).repeat_interleave(H // G, dim=1)
        g = torch.exp(-torch.exp(a_log.double())[:, None] * P.softplus(x["a"].double() + dt.double()))
        o = P.delta_recurrence(rep(y["q"]) * dk ** -0.5, rep(y["k"]), y["v"], g, P.sigmoid(x["b"].double()))
        want = P.rms(o, 1e-4) * nw.double() * P.sigmoid(x["g"].double())
        _close(torch.cat(got[s]), want, dtype, f32_tol=1e-4)
    K.check_device_errors()


def test_delta_rule_by_channel_over_a_long_prompt():
    """A thousand tokens in one portion, in uneven portions, and in steps of one token leave the same state and outputs; every
    choice of lanes per column gives the same."""
    from unillm_b200.ops import cuda_ops as K

    H, G, dk, dv, taps, T = 2, 1, 64, 48, 4, 1000
    Cn = 2 * G * dk + H * dv
    proj, conv, nw = _rand(T, Cn + 8, seed=1).cuda().float(), _rand(taps, Cn, seed=2, scale=0.5).cuda().float(), torch.ones(dv, device="cuda")
    a_log, dt = torch.full((H,), -2.0, device="cuda"), torch.linspace(-6.0, 1.0, H * dk).cuda()      # from hundreds of tokens to a few
    decay, gate = _rand(T, H * dk, seed=3).cuda().float(), _rand(T, H * dv, seed=4).cuda().float()

    def run(cuts, lanes):
        state, cs = torch.zeros(2, H, dk, dv, device="cuda"), torch.zeros(2, taps - 1, Cn, device="cuda")
        out, half = [], 0
        for a, b in C.portions(T, cuts):
            si, so = _i32([half if a else -1]), _i32([half ^ 1])
            p = K.Portions(0, 1, 1, 1, None, si, so) if b - a == 1 else K.Portions(0, b - a, 1, b - a, _i32([0, b - a]), si, so)
            out.append(K.delta_mixer(proj[a:b].contiguous(), 0, conv, a_log, dt, nw, cs, state, [p], kv_heads=G, eps=1e-6, lanes=lanes,
                                     decay=decay[a:b], gate=gate[a:b], gate_act="sigmoid"))
            half ^= 1
        return torch.cat(out), state[half]

    ref, end = run([1], 0)
    for cuts, lanes in (([T], 8), ([T], 16), ([500, 3, 1, 40, 17], 8), ([2], 16)):
        got, st = run(cuts, lanes)
        _close(got, ref.cpu(), torch.float32, f32_tol=1e-3)
        _close(st, end.cpu(), torch.float32, f32_tol=1e-4)
    K.check_device_errors()


# ------------------------------------------------------------------------------------------------
# the serving engine
# ------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=sorted(C.CASES))
def case(request):
    cfg = C.CASES[request.param]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 200, 1)
    return request.param, cfg, w, C.load_model(cfg, w), toks, P.forward(cfg, w, toks)


def _engine(m, dtype, blocks=16, **kw):
    from unillm_b200.engine.factory import build_engine

    o = dict(max_num_seqs=4, max_num_batched_tokens=256, max_model_len=256, use_cuda_graphs=False, enable_prefix_caching=False)
    o.update(kw)
    return build_engine(m, device="cuda", dtype=dtype, num_blocks=blocks, **o)


def _check_rows(got, want, dtype):
    err = C.row_error(got, want)
    assert err.max() < (1e-4 if dtype == torch.float32 else 0.08), (err.max(), err.median())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[200], [1], [2], [3, 1, 2], [16], [17, 2, 31], [64, 1], [150] + [1] * 50])
def test_portions_and_decoding(case, dtype, sizes):
    """Whole prompts, portions down to two tokens, token by token, and a long decoded tail give the same logits."""
    _, _, _, m, toks, ref = case
    eng = _engine(m, dtype)
    got = C.score(eng, toks, C.portions(len(toks), sizes))
    eng.runner.raise_on_device_error()
    _check_rows(got, ref, dtype)
    _check_rows(got, C.score(eng, toks, [(0, len(toks))]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_with_blocks_and_slots_used_again(case, dtype):
    _, cfg, w, m, _, _ = case
    seqs = {k: C.tokens(cfg, n, 10 + k) for k, n in C.BATCH.items()}
    eng = _engine(m, dtype, blocks=11, max_num_seqs=3)
    got = C.score_batch(eng, seqs, C.BATCH_SIZES)
    eng.runner.raise_on_device_error()
    assert eng.pool.num_free() == 11 and eng.slots.num_free() == 3
    alone = _engine(m, dtype)
    for k in seqs:
        _check_rows(got[k], P.forward(cfg, w, seqs[k]), dtype)
        _check_rows(got[k], C.score(alone, seqs[k], [(0, len(seqs[k]))]), dtype)


def test_layers_one_by_one(case):
    """The residual stream behind every layer: models cut off behind layer i whose head reads the stream through a nearly linear
    final norm."""
    _, cfg, w, _, toks, _ = case
    n, H = 40, cfg["width"]
    _, after = P.forward(cfg, w, toks[:n], keep_layers=True)
    for i in range(len(cfg["layers"])):
        cut = dict(cfg, vocab=cfg["vocab"], layers=cfg["layers"][:i + 1])
        w2 = dict(w)
        tiny = 2.0 ** -12
        w2["final.norm.alpha"], w2["final.norm"], w2["final.norm.b"] = torch.tensor(tiny), torch.full((H,), 1.0 / tiny), torch.zeros(H)
        w2["head"] = torch.eye(H)[torch.arange(cfg["vocab"]) % H]
        got = C.score(_engine(C.load_model(cut, w2), torch.float32), toks[:n], [(0, 25), (25, n)])
        m = min(H, cfg["vocab"])
        want = after[i][:, :m]
        assert (got[:, :m] - want).abs().max() < 2e-4 * want.abs().max(), i


@pytest.mark.parametrize("graphs,ahead", [(False, False), (True, False), (True, True)])
def test_greedy_generation(case, graphs, ahead):
    """Requests through the scheduler (chunked prompts, a pool too small for all, CUDA graphs, the host one step ahead), in 32
    bits token for token; in bf16 graphs and plain launches agree."""
    from unillm_b200.sampling import SamplingParams

    name, _, _, m, _, _ = case
    prompts, want = C.expected_generation(name)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    kw = dict(blocks=9, max_num_batched_tokens=24, use_cuda_graphs=graphs, async_scheduling=ahead, enable_prefix_caching=True)
    eng = _engine(m, torch.float32, **kw)
    assert eng.generate(prompts, sp) == want
    eng.runner.raise_on_device_error()
    half = _engine(m, torch.bfloat16, **kw).generate(prompts, sp)
    plain = _engine(m, torch.bfloat16, **{**kw, "use_cuda_graphs": False, "async_scheduling": False}).generate(prompts, sp)
    same = sum(a == b for x, y in zip(half, plain) for a, b in zip(x, y))
    assert same >= 0.7 * 36


def test_pipeline_serves_on_the_kernels(case):
    from unillm_b200.config import GenerationConfig
    from unillm_b200.pipeline import InferencePipelineBuilder

    name, _, _, m, _, _ = case
    prompts, want = C.expected_generation(name)
    pipe = InferencePipelineBuilder().model(m).device("cuda").engine_options(max_num_seqs=2, max_model_len=256, num_blocks=32,
                                                                             dtype=torch.float32).build()
    got = pipe.generate_tokens(prompts[0], GenerationConfig.greedy(6, eos_token_id=-1))
    assert pipe.engine_kind == "gpu-kernels" and got == want[0]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(tmp_path, dtype):
    cfg = C.CASES["mixed"]
    w, toks = C.make_weights(cfg), C.tokens(cfg, 80, 1)
    ref = P.forward(cfg, w, toks)
    d = C.write_model(tmp_path / "m", cfg, w)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:70], "want": [3, 69]}, {"id": "y", "tokens": toks[:9], "want": [8]}],
              "end": ["y"]},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[70:71], "want": []}, {"id": "z", "tokens": toks[:2], "want": [1]}], "end": []},
             {"step": 2, "entries": [{"id": "z", "tokens": toks[2:33], "want": [30]}, {"id": "x", "tokens": toks[71:72], "want": [0]}],
              "end": ["x", "z"]}]
    exe = os.path.join(os.path.dirname(__file__), "..", "bin", "trace_run")
    r = subprocess.run([sys.executable, exe, "--model", d, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "160"],
                       input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    for step, rows in ((0, [3, 69, 8]), (1, [1]), (2, [32, 71])):
        got = torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32).reshape(len(rows), -1)
        assert C.row_error(got.double(), ref[rows]).max() < (1e-4 if dtype == "float32" else 0.08)


@pytest.mark.parametrize("change", ["no average", "no shift", "gated", "plain attention"])
def test_other_uses_of_the_parts(change):
    """Designs that take some of the mechanisms only: the GPU engine against the host engine."""
    from unillm_b200.engine.factory import build_cpu_engine

    cfg = C.CASES["mixed"]
    m = C.load_model(cfg, C.make_weights(cfg))
    s = m.spec
    if change == "no average":
        m.spec = dataclasses.replace(s, depth_average=False)
    elif change == "no shift":
        m.spec = dataclasses.replace(s, token_shift=False)
    elif change == "gated":
        m.spec = dataclasses.replace(s, mlp="gated", act="silu", mlp_bias=False)
    else:
        plain = [dataclasses.replace(ls, value_rope=False, out_gate="", chunk=21) if ls.maps == 1 and ls.mixer == "attention" else ls for ls in s.layers]
        m.spec = dataclasses.replace(s, layers=tuple(plain))
    m.spec = dataclasses.replace(m.spec, initializer_range=0.15)
    m._init_params("random", seed=3)
    toks = C.tokens(cfg, 90, 2)
    want = C.score(build_cpu_engine(m, num_blocks=16), toks, [(0, 90)])
    assert math.isfinite(float(want.abs().sum()))
    for dtype in DTYPES:
        for sizes in ([90], [33, 1, 2, 17]):
            eng = _engine(m, dtype)
            _check_rows(C.score(eng, toks, C.portions(90, sizes)), want, dtype)
            eng.runner.raise_on_device_error()


def test_wide_heads_are_refused():
    from unillm_b200.engine.factory import why_not_gpu

    cfg = C.CASES["wide"]
    m = C.load_model(cfg, C.make_weights(cfg))
    assert why_not_gpu(m) is None
    layers = list(m.spec.layers)
    layers[2] = dataclasses.replace(layers[2], head_dim=136)
    m.spec = dataclasses.replace(m.spec, layers=tuple(layers))
    assert "256" in why_not_gpu(m)
