"""Bakasun on the GPU: each mechanism's kernel alone and the serving engine on them, against the plain statement."""
import json
import os
import subprocess
import sys

import pytest
import torch

import bakasun_cases as C
import bakasun_plain as P

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def _close(got, want, dtype, f32_tol=2e-5, bf16_tol=1e-2):
    """Largest difference relative to the expected value and the spread of all of them."""
    got, want = got.double().cpu(), want.double()
    spread = want.std().item() if want.numel() > 1 else 0.0
    err = ((got - want).abs() / (want.abs() + spread).clamp_min(1e-6)).max().item()
    assert err < (f32_tol if dtype == torch.float32 else bf16_tol), err


def _rand(*shape, seed=0, dtype=torch.bfloat16, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def _r8(n):
    return (n + 7) // 8 * 8


def _pad(t, n, dim=-1):
    shape = list(t.shape)
    shape[dim] = n - t.shape[dim]
    return torch.cat([t, t.new_zeros(shape)], dim)


def _i32(v):
    return torch.as_tensor(v, dtype=torch.int32).cuda()


def _steps(lens, cuts):
    """Portions of several sequences that run together: per step (sequence, first, end) of those that still have tokens."""
    todo = [C.portions(n, c) for n, c in zip(lens, cuts)]
    while any(todo):
        yield [(s, *t.pop(0)) for s, t in enumerate(todo) if t]


def _portions(step, half):
    """The step's rows as the runner packs them (single tokens first) and the order of its sequences.  State rows: 2 s and
    2 s + 1 of sequence s take turns."""
    from unillm_b200.ops import cuda_ops as K

    one, more = [e for e in step if e[2] - e[1] == 1], [e for e in step if e[2] - e[1] > 1]
    rows = lambda group: (_i32([-1 if a == 0 else 2 * s + half[s] for s, a, _ in group]), _i32([2 * s + (half[s] ^ 1) for s, _, _ in group]))
    parts = []
    if one:
        parts.append(K.Portions(0, len(one), len(one), 1, None, *rows(one)))
    if more:
        n = [b - a for _, a, b in more]
        qs = [0] + [sum(n[:i + 1]) for i in range(len(n))]
        parts.append(K.Portions(len(one), qs[-1], len(n), max(n), _i32(qs), *rows(more)))
    for s, _, _ in step:
        half[s] ^= 1
    return one + more, parts


# ------------------------------------------------------------------------------------------------
# gated delta rule
# ------------------------------------------------------------------------------------------------
LENS = [75, 5, 1, 64, 33, 16]
CUTS = [[75], [2], [1], [33, 1, 2, 14], [1, 17, 1], [16]]
DELTA = [(1, 1, 8, 8, 4, 0), (3, 3, 13, 21, 1, 0), (4, 2, 20, 72, 2, 0), (4, 1, 32, 40, 3, 0), (6, 3, 64, 64, 4, 8), (2, 1, 64, 80, 5, 16),
         (3, 1, 40, 128, 4, 8), (2, 2, 128, 128, 4, 8), (4, 2, 128, 96, 4, 16), (2, 1, 100, 16, 9, 32), (2, 1, 136, 200, 4, 16), (1, 1, 256, 256, 16, 32),
         (2, 2, 192, 64, 2, 0), (1, 1, 8, 256, 3, 0), (2, 1, 256, 8, 3, 0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,taps,lanes", DELTA)
def test_delta_rule(dtype, H, G, dk, dv, taps, lanes):
    """Convolutions, unit norms, gates, recurrence, head norm and output gate: portions of several sequences against the plain
    recurrence on whole ones, from a state row into another, single tokens beside longer portions."""
    from unillm_b200.ops import cuda_ops as K

    kp, vp, C_ = _r8(dk), _r8(dv), 2 * G * _r8(dk) + H * _r8(dv)
    conv = {c: _rand(n, w, taps, seed=i, scale=0.6) for i, (c, n, w) in enumerate((("q", G, dk), ("k", G, dk), ("v", H, dv)))}
    a_log, dt = _rand(H, seed=5, dtype=torch.float32) - 0.5, _rand(H, seed=6, dtype=torch.float32, scale=2.0) - 1.0
    nw = 1 + _rand(dv, seed=7, dtype=torch.float32, scale=0.3)
    width = {"q": (G, dk, kp), "k": (G, dk, kp), "v": (H, dv, vp), "g": (H, dv, vp)}
    xs = [{c: _rand(n, h, w, seed=20 * s + i) for i, (c, (h, w, _)) in enumerate(width.items())} for s, n in enumerate(LENS)]
    for s, (x, n) in enumerate(zip(xs, LENS)):
        x["b"], x["a"] = _rand(n, H, seed=500 + s, scale=1.5), _rand(n, H, seed=600 + s, scale=2.5)
        x["a"][n // 2] = 30.0                                   # a token that forgets almost everything
        x["k"][0] *= 6                                          # and a first token that stands out
    col, ld = 16, _r8(16 + C_ + H * vp + 2 * H)
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
        for c in "ba":
            proj[:, at:at + H] = torch.cat([xs[s][c][a:b] for s, a, b in order]).to("cuda", dtype)
            at += H
        wide = torch.full((rows, 8 + H * vp), 5.0, device="cuda", dtype=dtype)
        K.delta_mixer(proj, col, taps_dev, a_log.cuda(), dt.cuda(), _pad(nw, vp).cuda(), conv_state, state, parts, kv_heads=G, eps=1e-4,
                      dk_real=dk, dv_real=dv, out=wide[:, 8:], lanes=lanes)
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
        g = torch.exp(-torch.exp(a_log.double()) * P.softplus(x["a"].double() + dt.double()))
        o = P.delta_recurrence(rep(y["q"]) * dk ** -0.5, rep(y["k"]), y["v"], g, P.sigmoid(x["b"].double()))
        want = P.rms(o, 1e-4) * nw.double() * P.silu(x["g"].double())
        _close(torch.cat(got[s]), want, dtype, f32_tol=1e-4)
    K.check_device_errors()


def test_delta_rule_over_a_long_prompt():
    """A thousand tokens in one portion, in uneven portions, and in steps of one token leave the same state and outputs; every
    choice of lanes per column gives the same."""
    from unillm_b200.ops import cuda_ops as K

    H, G, dk, dv, taps, T = 2, 1, 64, 48, 4, 1000
    ld = 2 * G * dk + 2 * H * dv + 8
    proj = _rand(T, ld, seed=1).cuda().float()
    conv, nw = _rand(taps, 2 * G * dk + H * dv, seed=2, scale=0.5).cuda().float(), torch.ones(dv, device="cuda")
    a_log, dt = torch.full((H,), -2.0, device="cuda"), torch.full((H,), -3.0, device="cuda")      # a memory of hundreds of tokens

    def run(cuts, lanes):
        state, cs = torch.zeros(2, H, dk, dv, device="cuda"), torch.zeros(2, taps - 1, 2 * G * dk + H * dv, device="cuda")
        out, half = [], 0
        for a, b in C.portions(T, cuts):
            si, so = _i32([half if a else -1]), _i32([half ^ 1])
            p = K.Portions(0, 1, 1, 1, None, si, so) if b - a == 1 else K.Portions(0, b - a, 1, b - a, _i32([0, b - a]), si, so)
            out.append(K.delta_mixer(proj[a:b].contiguous(), 0, conv, a_log, dt, nw, cs, state, [p], kv_heads=G, eps=1e-6, lanes=lanes))
            half ^= 1
        return torch.cat(out), state[half]

    ref, end = run([1], 0)
    for cuts, lanes in (([T], 8), ([T], 16), ([500, 3, 1, 40, 17], 8), ([2], 16)):
        got, st = run(cuts, lanes)
        _close(got, ref.cpu(), torch.float32, f32_tol=1e-3)
        _close(st, end.cpu(), torch.float32, f32_tol=1e-4)
    K.check_device_errors()


# ------------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,d,dv,dims", [(3, 1, 10, 14, 6), (4, 2, 24, 40, 16), (2, 2, 20, 9, 20), (18, 3, 72, 136, 36), (5, 5, 128, 64, 44),
                                              (8, 1, 256, 8, 254), (1, 1, 8, 8, 2), (2, 1, 64, 64, 64)])
@pytest.mark.parametrize("row_norm", [True, False])
def test_row_norm_and_rotation(dtype, hq, hkv, d, dv, dims, row_norm):
    """One norm over all queries and one over all keys, rotations of any even size with slowed-down frequencies, rows that are the
    front of wider ones."""
    from unillm_b200.ops import cuda_ops as K
    from unillm_b200.precompute import rope_inv_freq

    T, bs, nb, dp, vp = 9, 16, 7, _r8(d), _r8(dv)
    q, k, v = _rand(T, hq, d, seed=1, scale=2.0), _rand(T, hkv, d, seed=2), _rand(T, hkv, dv, seed=3)
    qw, kw = 1 + _rand(hq * d, seed=4, scale=0.4), 1 + _rand(hkv * d, seed=5, scale=0.4)
    pos = torch.tensor([0, 1, 15, 16, 17, 300, 299, 1000, 3], dtype=torch.int32)
    slots = torch.tensor([40, 0, 111, -1, 16, 15, 3, 77, 50], dtype=torch.int32)
    dev = lambda t: t.to("cuda", dtype).contiguous()
    rows = torch.cat([_pad(q, dp).flatten(1), _pad(k, dp).flatten(1), _pad(v, vp).flatten(1)], 1)
    wide = dev(torch.cat([rows, torch.full((T, 24), 7.0)], 1))
    kc, vc = dev(torch.full((nb, hkv, bs, dp), 5.0)), dev(torch.full((nb, hkv, bs, vp), 5.0))
    norm_w = lambda w, n: dev(_pad(w.reshape(n, d), dp).flatten()) if row_norm else None
    K.rope_kv_append(wide[:, :rows.shape[1]], pos.cuda(), slots.cuda(), kc, vc, num_q_heads=hq, num_kv_heads=hkv, head_dim=dp, v_head_dim=vp,
                     rotary_dim=dims, inv_freq=rope_inv_freq(dims, 700.0, linear=2.5).cuda(), norm_dim=d, norm_eps=1e-3,
                     q_norm_w=norm_w(qw, hq), k_norm_w=norm_w(kw, hkv), row_norm=row_norm, k_cache_only=True)
    rot = {"base": 700.0, "dims": dims, "scaling": {"factor": 2.5}}
    def want(x, w):
        y = x.double().flatten(1)
        if row_norm:
            y = P.rms(y, 1e-3) * w.double()
        return P.rotate(y.reshape(x.shape), pos, rot)
    tol = dict(f32_tol=3e-4)                         # angles of hundreds of radians in 32 bits
    got_q = wide[:, :hq * dp].unflatten(1, (hq, dp))
    _close(got_q[..., :d], want(q, qw), dtype, **tol)
    assert got_q[..., d:].abs().sum() == 0 and (wide[:, rows.shape[1]:] == 7.0).all()
    keep = slots >= 0
    at = slots[keep].long()
    kk, vv = (c.transpose(1, 2).flatten(0, 1)[at.cuda()] for c in (kc, vc))
    _close(kk[..., :d], want(k, kw)[keep], dtype, **tol)
    assert torch.equal(vv[..., :dv].cpu(), v[keep].to(dtype)) and kk[..., d:].abs().sum() == 0 and vv[..., dv:].abs().sum() == 0
    assert int((kc.transpose(1, 2).flatten(0, 1) == 5.0).all(-1).all(-1).sum()) == nb * bs - int(keep.sum())       # no other slot was touched
    K.check_device_errors()


SHAPES = [(6, 3, 48, 88), (3, 1, 16, 24), (18, 1, 72, 136), (40, 2, 40, 16), (4, 4, 128, 128), (2, 1, 200, 256), (5, 1, 8, 8)]


def _paged(lens, hkv, d, dv, seed, bs=16):
    """Random keys and values of several sequences in shuffled pages; unused slots hold large numbers."""
    g = torch.Generator().manual_seed(seed)
    nb = sum((n + bs - 1) // bs for n in lens) + 3
    perm, bt = torch.randperm(nb, generator=g).tolist(), torch.full((len(lens), (max(lens) + bs - 1) // bs), -1, dtype=torch.int32)
    k = [torch.randn(n, hkv, d, generator=g).to(torch.bfloat16) for n in lens]
    v = [torch.randn(n, hkv, dv, generator=g).to(torch.bfloat16) for n in lens]
    for s, n in enumerate(lens):
        for p in range(0, n, bs):
            bt[s, p // bs] = perm.pop()
    def fill(dtype):
        kc, vc = torch.full((nb, hkv, bs, d), 30.0), torch.full((nb, hkv, bs, dv), 30.0)
        for s, n in enumerate(lens):
            for p in range(n):
                kc[bt[s, p // bs], :, p % bs], vc[bt[s, p // bs], :, p % bs] = k[s][p].float(), v[s][p].float()
        return kc.to("cuda", dtype), vc.to("cuda", dtype)
    return k, v, bt, fill


def _plant(q, k, pos, key, scale, score=13.0):
    """Makes the score of ``key`` stand out for the first query head of its group at ``pos``."""
    h = (pos + key) % k.shape[1]
    n = q[pos, h * (q.shape[1] // k.shape[1])].float()
    k[key, h] = (n * (score / (scale * n.pow(2).sum()))).to(torch.bfloat16)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,d,dv", SHAPES)
@pytest.mark.parametrize("window,cap", [(42, 10.0), (17, None), (64, 25.0), (1, 8.0), (0, 6.0), (100, None)])
def test_capped_windowed_attention(dtype, hq, hkv, d, dv, window, cap):
    """Prompts, portions and single tokens; keys that stand out just inside and just outside of the window, at page and tile
    borders, at the start and at the query itself; the constant term of the denominator."""
    from unillm_b200.ops import cuda_ops as K

    lens, qlens, scale = [150, 5, 83, 17, 129], [150, 2, 40, 1, 1], 0.6 * d ** -0.5
    k, v, bt, fill = _paged(lens, hkv, d, dv, seed=d + window)
    q = [_rand(n, hq, d, seed=70 + i) for i, n in enumerate(lens)]
    w = window or 10 ** 6
    for s, pos in ((0, 149), (0, 128), (0, 100), (0, 64), (2, 82), (2, 60), (3, 16), (4, 128)):
        for key in (pos - w + 1, pos - w):
            if 0 <= key:
                _plant(q[s], k[s], pos, key, scale)
    for s, pos, key in ((0, 140, 127), (0, 120, 112), (0, 70, 0), (2, 77, 63), (2, 50, 50), (1, 4, 0), (4, 128, 111)):
        _plant(q[s], k[s], pos, key, scale)
    want = [P.attend(a.double(), b.double(), c.double(), scale, window or None, cap) for a, b, c in zip(q, k, v)]
    kc, vc = fill(dtype)
    zero, kw = torch.zeros(hq, device="cuda"), dict(scale=scale, window=window, softcap=cap or 0.0)
    tol = dict(bf16_tol=3e-2)
    ld = hq * d + 24                                  # queries inside wider rows, outputs into wider rows
    def rows(ts):
        t = torch.cat([torch.cat([x.flatten(1) for x in ts]), torch.zeros(sum(len(x) for x in ts), 24, dtype=torch.bfloat16)], 1).to("cuda", dtype)
        return t[:, :hq * d].unflatten(1, (hq, d))
    new = rows([a[n - m:] for a, n, m in zip(q, lens, qlens)])
    out = torch.full((new.shape[0], hq * dv + 8), 3.0, device="cuda", dtype=dtype)
    K.attn_prefill(new, kc, vc, bt.cuda(), _i32(lens), _i32([0, *torch.tensor(qlens).cumsum(0).tolist()]), max(qlens), sinks=zero,
                   out=out[:, :hq * dv].unflatten(1, (hq, dv)), **kw)
    _close(out[:, :hq * dv].unflatten(1, (hq, dv)), torch.cat([x[n - m:] for x, n, m in zip(want, lens, qlens)]), dtype, **tol)
    assert (out[:, hq * dv:] == 3.0).all() and ld == new.stride(0)
    for splits in (1, 3):
        got = K.attn_decode(rows([a[-1:] for a in q]), kc, vc, bt.cuda(), _i32(lens), sinks=zero, splits=splits, **kw)
        _close(got, torch.cat([x[-1:] for x in want]), dtype, **tol)
    K.check_device_errors()


# ------------------------------------------------------------------------------------------------
# mixtures and norms
# ------------------------------------------------------------------------------------------------
ROUTERS = [(12, 3, 4, 1, 40), (9, 4, 3, 2, 96), (5, 1, 1, 1, 16), (40, 6, 8, 3, 200), (256, 16, 16, 4, 72), (256, 2, 256, 2, 8), (6, 6, 2, 2, 24), (96, 8, 2, 1, 1024)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 7, 1300])
@pytest.mark.parametrize("E,top,count,keep,H", ROUTERS)
@pytest.mark.parametrize("given", [False, True])
def test_router(dtype, T, E, top, count, keep, H, given):
    """Choice by corrected scores inside the best groups, weights without the correction, gate of the shared expert; from the rows
    or from logits in wider rows."""
    from unillm_b200.ops import cuda_ops as K

    x, w, sg = _rand(T, H, seed=1), _rand(E, H, seed=2, scale=1.5 * H ** -0.5), _rand(H, seed=3, scale=2 * H ** -0.5)
    corr = (_rand(E, seed=4, dtype=torch.float32, scale=1.5 / E) - 0.6 / E).to(torch.bfloat16)      # choice scores of both signs
    dev = lambda t: t.to("cuda", dtype).contiguous()
    kw = dict(correction=dev(corr), groups=count, keep_groups=keep)
    if given:
        full = torch.cat([x.double() @ w.double().T, x.double() @ sg.double()[:, None], torch.full((T, 5), 1e3)], 1).float().cuda()
        r = K.moe_route(None, None, top, logits=full, num_experts=E, shared_gate=True, **kw)
    else:
        r = K.moe_route(dev(x), dev(w), top, round_logits_bf16=False, shared_w=dev(sg), **kw)
    s = torch.softmax(x.double() @ w.double().T, -1)
    choice = s + corr.double()
    _close(r.shared_gate, P.sigmoid(x.double() @ sg.double()), torch.float32)
    ids, ws = r.topk_ids.cpu(), r.topk_w.double().cpu()
    for t in range(T) if T < 100 else range(0, T, 37):
        want = P.choose(choice[t], top, {"count": count, "keep": keep})
        if set(ids[t].tolist()) != set(want):            # allowed only where scores tie to rounding
            a, b = sorted(float(choice[t, e]) for e in set(ids[t].tolist()) - set(want)), sorted(float(choice[t, e]) for e in set(want) - set(ids[t].tolist()))
            assert max(abs(x - y) for x, y in zip(a, b)) < 1e-5, (t, a, b)
            continue
        total = sum(s[t, e] for e in want) + 1e-20
        for j, e in enumerate(ids[t].tolist()):
            assert abs(float(ws[t, j] - s[t, e] / total)) < 1e-5
    counts = torch.bincount(ids.flatten().long(), minlength=E)
    assert torch.equal(r.counts.cpu().long(), counts)
    K.check_device_errors()


def test_router_refuses_groups_that_do_not_fit():
    from unillm_b200.ops import cuda_ops as K

    x, w = _rand(2, 16).cuda(), _rand(8, 16).cuda()
    for groups, keep, top in ((3, 1, 1), (4, 5, 1), (4, 1, 3)):
        with pytest.raises(RuntimeError):
            K.moe_route(x, w, top, groups=groups, keep_groups=keep)
    with pytest.raises(ValueError):
        K.moe_route(None, None, 2, logits=_rand(2, 8).cuda(), shared_w=_rand(8).cuda())
    with pytest.raises(ValueError):
        K.moe_route(x, w, 2, correction=_rand(7).cuda())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,T,top", [(8, 1, 1), (50, 7, 3), (136, 20, 5), (1000, 3, 2), (4096, 9, 6), (9000, 2, 4), (16384, 2, 1)])
def test_norms_around_a_mixture(dtype, H, T, top):
    """Residual add of the normed weighted sum of expert rows and the gated shared expert's, then the next norm; and the same for
    picked rows alone, which leaves the stream as it is."""
    from unillm_b200.ops import cuda_ops as K

    E, Hp = 8, _r8(H)
    x, base, ex = _rand(T, H, seed=1, dtype=torch.float32, scale=2.0), _rand(T, H, seed=2), _rand(T * top, H, seed=3)
    wy, wn = _rand(H, seed=4, scale=0.3), _rand(H, seed=5, scale=0.3)
    dev = lambda t: _pad(t, Hp).to("cuda", dtype).contiguous()
    r = K.moe_route(_rand(T, 16, seed=6).cuda(), _rand(E, 16, seed=7).cuda(), top, shared_w=_rand(16, seed=8).cuda())
    slot, w, gate = r.row_slot.cpu().view(T, top).long(), r.topk_w.double().cpu(), r.shared_gate.double().cpu()[:, None]
    for with_base, with_experts in ((True, True), (False, True), (True, False), (False, False)):
        kw = dict(eps=1e-4, width=H, y=dev(base) if with_base else None, y_weight=dev(wy) if with_base or with_experts else None)
        f = torch.zeros(T, H, dtype=torch.float64)
        if with_experts:
            kw.update(experts=dev(ex), routing=r)
            f += (ex.double()[slot] * w[..., None]).sum(1)
        if with_base:
            f += base.double() * (gate if with_experts else 1.0)
        want_x = x.double() + (P.norm(f, wy.double(), 1e-4) if with_base or with_experts else 0)
        stream = _pad(x, Hp).cuda()
        pick = torch.tensor([T - 1, 0, T // 2])
        got = K.sublayer_in(stream, (), dev(wn), rows=_i32(pick), **kw)
        assert torch.equal(stream.cpu(), _pad(x, Hp)) and got[:, H:].abs().sum() == 0
        _close(got[:, :H], P.norm(want_x, wn.double(), 1e-4)[pick], dtype, f32_tol=5e-5)
        xs, out = K.sublayer_in(stream, (), dev(wn), **kw)
        _close(xs[:, :H], want_x, torch.float32)
        _close(out[:, :H], P.norm(want_x, wn.double(), 1e-4), dtype, f32_tol=5e-5)
        assert xs[:, H:].abs().sum() == 0 and out[:, H:].abs().sum() == 0
    K.check_device_errors()


def test_router_of_many_rows_is_a_matrix_product():
    """From a thousand rows on, logits and gates come from the tensor cores; the choice is that of the router kernel."""
    from unillm_b200.engine import moe_runner
    from unillm_b200.engine.runner import GpuModelRunner, RunnerWeights

    cfg = C.CASES["mixed"]
    m = C.load_model(cfg, C.make_weights(cfg))
    runner = GpuModelRunner(m.spec, RunnerWeights(m.spec, m.p, "cuda"), num_blocks=8, max_num_seqs=4, max_num_batched_tokens=2048,
                            max_model_len=256, use_cuda_graphs=False)
    h = _rand(1100, cfg["width"], seed=3).cuda()
    base, y, r = moe_runner.moe_branch(runner, 1, h, h)
    few = [moe_runner.moe_branch(runner, 1, h[i:i + 550].contiguous(), h[i:i + 550].contiguous()) for i in (0, 550)]
    ids = torch.cat([x[2].topk_ids for x in few])
    same = (r.topk_ids == ids).all(1)
    assert same.float().mean() > 0.99
    for got, want in ((r.topk_w, torch.cat([x[2].topk_w for x in few])), (r.shared_gate, torch.cat([x[2].shared_gate for x in few]))):
        assert (got - want)[same].abs().max() < 1e-4
    assert _close(base, torch.cat([x[0] for x in few]).cpu(), torch.bfloat16, bf16_tol=3e-2) is None


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
    """In bf16 a router's close call may go the other way, which moves single rows by more than rounding does."""
    err = C.row_error(got, want)
    if dtype == torch.float32:
        assert err.max() < 5e-4 and err.median() < 3e-5, (err.max(), err.median())
    else:
        assert err.median() < 0.12 and err.quantile(0.9) < 0.5, (err.median(), err.quantile(0.9), err.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[200], [1], [2], [3, 1, 2], [16], [17, 2, 31], [64, 1], [150] + [1] * 50])
def test_portions_and_decoding(case, dtype, sizes):
    """Whole prompts, portions down to two tokens, token by token, and a long decoded tail give the same logits."""
    _, _, _, m, toks, ref = case
    eng = _engine(m, dtype)
    got = C.score(eng, toks, C.portions(len(toks), sizes))
    eng.runner.raise_on_device_error()
    _check_rows(got, ref, dtype)
    whole = C.score(eng, toks, [(0, len(toks))])
    _check_rows(got, whole, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_with_blocks_and_slots_used_again(case, dtype):
    _, cfg, w, m, _, _ = case
    seqs = {k: C.tokens(cfg, n, 10 + k) for k, n in C.BATCH.items()}
    eng = _engine(m, dtype, blocks=11, max_num_seqs=3)
    got = C.score_batch(eng, seqs, C.BATCH_SIZES)
    eng.runner.raise_on_device_error()
    assert eng.pool.num_free() == 11 and (eng.slots is None or eng.slots.num_free() == 3)
    alone = _engine(m, dtype)
    for k in seqs:
        if dtype == torch.bfloat16 and len(seqs[k]) < 30:
            continue                                 # a handful of rows, whose median says little
        _check_rows(got[k], P.forward(cfg, w, seqs[k]), dtype)
        _check_rows(got[k], C.score(alone, seqs[k], [(0, len(seqs[k]))]), dtype)


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
        assert C.row_error(got.double(), ref[rows]).median() < (5e-4 if dtype == "float32" else 0.3)


def test_layers_with_the_delta_rule_alone():
    """The mechanism as a layer's only mixer (another design's use of it): the GPU engine against the host engine."""
    import dataclasses

    from unillm_b200.engine.factory import build_cpu_engine

    cfg = C.CASES["mixed"]
    m = C.load_model(cfg, C.make_weights(cfg))
    rule = dataclasses.replace(m.spec.layer(1).beside, mlp="dense", intermediate_size=40)
    m.spec = dataclasses.replace(m.spec, layers=(rule, dataclasses.replace(rule, mlp=None), m.spec.layer(3)), num_layers=3, initializer_range=0.15)
    m._init_params("random", seed=3)
    m.p["layers.0.dt_bias"] = m.p["layers.0.dt_bias"] - 3.0
    toks = C.tokens(cfg, 90, 2)
    want = C.score(build_cpu_engine(m, num_blocks=16), toks, [(0, 90)])
    for dtype in DTYPES:
        for sizes in ([90], [33, 1, 2, 17], [1]):
            eng = _engine(m, dtype)
            _check_rows(C.score(eng, toks, C.portions(90, sizes)), want, dtype)
            eng.runner.raise_on_device_error()
