"""Nipulorn on the GPU: each mechanism's kernel alone and the serving engine on them, against the plain statement."""
import json
import os
import subprocess
import sys

import pytest
import torch

import nipulorn_cases as C
import nipulorn_plain as P

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
    def rows(group):
        si = [-1 if a == 0 else 2 * s + half[s] for s, a, _ in group]
        so = [2 * s + (half[s] ^ 1) for s, _, _ in group]
        return _i32(si), _i32(so)
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
# mechanisms
# ------------------------------------------------------------------------------------------------
LENS = [37, 5, 1, 64, 18]
CUTS = [[37], [2], [1], [33, 1, 2, 1, 27], [1, 17]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,taps,mix,tile", [(8, 2, 5, 0), (50, 4, 5, 0), (136, 7, 0, 1), (200, 1, 5, 3), (1000, 3, 0, 0), (2048, 4, 5, 16),
                                             (4096, 5, 0, 2), (9000, 2, 5, 0), (4096, 4, 5, 0), (2048, 1, 0, 0), (264, 24, 5, 4)])
def test_sublayer_input(dtype, H, taps, mix, tile):
    """Residual add of the normed sublayer rows, the next norm, its convolution and the token-shift mixes, in portions."""
    from unillm_b200.ops import cuda_ops as K

    Hp = _r8(H)
    x = [_rand(n, H, seed=10 + i, dtype=torch.float32, scale=2.0) for i, n in enumerate(LENS)]
    y = [_rand(n, H, seed=30 + i) for i, n in enumerate(LENS)]
    wy, wn = _rand(H, seed=1, scale=0.3), _rand(H, seed=2, scale=0.3)
    conv, mu = _rand(H, taps, seed=3, scale=0.4), _rand(mix, H, seed=4) if mix else None
    dev = lambda t: _pad(t, Hp).to("cuda", dtype).contiguous()
    f32 = lambda t: _pad(t.float(), Hp).cuda().contiguous()
    conv_state = torch.full((2 * len(LENS), taps - 1, Hp), 77.0, device="cuda")       # never to be read before it is written
    shift = torch.full((2 * len(LENS), Hp), 77.0, device="cuda") if mix else None
    for with_y in (True, False):
        half = [0] * len(LENS)
        got_x, got = [[] for _ in LENS], [[] for _ in LENS]
        for step in _steps(LENS, CUTS):
            order, parts = _portions(step, half)
            cat = lambda ts: torch.cat([ts[s][a:b] for s, a, b in order])
            xs, out = K.sublayer_in(f32(cat(x)), parts, dev(wn), eps=1e-4, y=dev(cat(y)) if with_y else None,
                                    y_weight=dev(wy) if with_y else None, conv=dev(conv.t()), conv_state=conv_state,
                                    mu=None if mu is None else dev(mu), shift_state=shift, width=H, tile=tile)
            assert xs[:, H:].abs().sum() == 0 and out[..., H:].abs().sum() == 0
            r = 0
            for s, a, b in order:
                got_x[s].append(xs[r:r + b - a, :H].cpu()), got[s].append(out[..., r:r + b - a, :H].cpu())
                r += b - a
        for s in range(len(LENS)):
            want_x = x[s].double() + (P.norm(y[s].double(), wy.double(), 1e-4) if with_y else 0)
            h = P.input_conv(P.norm(want_x, wn.double(), 1e-4), conv.double())
            want = torch.stack([P.token_mix(h, m.double()) for m in mu]) if mix else h
            _close(torch.cat(got_x[s]), want_x, torch.float32, f32_tol=1e-5)
            _close(torch.cat(got[s], -2), want, dtype)
    K.check_device_errors()


def _wkv_inputs(H, D, lens, seed=0):
    g = torch.Generator().manual_seed(seed)
    out = []
    for n in lens:
        r, k, v, gate = ((torch.randn(n, H, D, generator=g)).to(torch.bfloat16) for _ in range(4))
        ww = torch.rand(n, H, D, generator=g) * 9 - 7           # decays from almost one to almost zero
        ww[n // 2] = 4.0                                        # a token that forgets everything
        k[0] *= 8                                               # a key at the start that a long memory keeps
        out.append((r, k, v, gate, ww))
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D", [(1, 8), (3, 13), (2, 20), (4, 32), (3, 40), (5, 64), (2, 72), (2, 128)])
@pytest.mark.parametrize("chunk", [0, 16, 64])
def test_wkv_recurrence(dtype, H, D, chunk):
    """Portions of several sequences against the recurrence on whole ones: from a state row into another, walked by one CTA or
    in parallel chunks, with head norm and gate."""
    from unillm_b200.ops import cuda_ops as K

    lens, cuts, Dp = [150, 5, 1, 70, 64], [[150], [2], [1], [33, 1, 2, 34], [64]], _r8(D)
    u, nw = _rand(H, D, seed=5), 1 + _rand(H * D, seed=6, scale=0.3)
    xs = _wkv_inputs(H, D, lens)
    dev = lambda t: _pad(t, Dp).flatten(-2)
    state = torch.full((2 * len(lens), H, Dp, Dp), 77.0, device="cuda")
    half, got = [0] * len(lens), [[] for _ in lens]
    for step in _steps(lens, cuts):
        order, parts = _portions(step, half)
        rkvg = torch.stack([torch.cat([dev(xs[s][j][a:b]) for s, a, b in order]) for j in range(4)]).to("cuda", dtype).contiguous()
        ww = torch.cat([dev(xs[s][4][a:b]) for s, a, b in order]).float().cuda().contiguous()
        out = K.wkv_mixer(rkvg, ww, _pad(u.float(), Dp).cuda(), _pad(nw.float().view(H, D), Dp).flatten().cuda(), state, parts,
                          eps=1e-4, norm_dim=D, chunk=chunk)
        out = out.view(-1, H, Dp).cpu()
        assert out[..., D:].abs().sum() == 0
        r = 0
        for s, a, b in order:
            got[s].append(out[r:r + b - a, :, :D])
            r += b - a
    for s, (r, k, v, gate, ww) in enumerate(xs):
        o = P.wkv_recurrence(r.double(), k.double(), v.double(), torch.exp(-torch.exp(ww.double())), u.double())
        want = P.rms(o, 1e-4) * nw.double().view(H, D) * P.silu(gate.double())
        _close(torch.cat(got[s]), want, dtype, f32_tol=1e-4)
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,q_rank,kv_rank,rot", [(3, 21, 18, 6), (1, 8, 8, 2), (16, 1536, 512, 64), (5, 56, 264, 40)])
@pytest.mark.parametrize("scaled", [True, False])
def test_latent_rows_and_rotation(dtype, heads, q_rank, kv_rank, rot, scaled):
    from unillm_b200.ops import cuda_ops as K
    from unillm_b200.precompute import rope_gain, rope_inv_freq

    T, bs, nb, qp, cp, rp = 9, 16, 7, _r8(q_rank), _r8(kv_rank), _r8(rot)
    spec = {"base": 700.0, "dims": rot}
    if scaled:
        spec["scaling"] = {"factor": 4.0, "original": 200, "fast": 8.0, "slow": 1.0}
    yarn = (4.0, 200.0, 8.0, 1.0) if scaled else None
    freq, gain = rope_inv_freq(rot, 700.0, None, yarn).cuda(), rope_gain(yarn)
    dq, dc, dr = _rand(T, q_rank, seed=1, scale=2.0), _rand(T, kv_rank, seed=2), _rand(T, rot, seed=3)
    qw, cw, q = _rand(q_rank, seed=4) + 1, _rand(kv_rank, seed=5) + 1, _rand(T, heads, rot, seed=6)
    pos = torch.tensor([0, 1, 15, 16, 17, 300, 299, 1000, 3], dtype=torch.int32)
    slots = torch.tensor([40, 0, 111, -1, 16, 15, 3, 77, 50], dtype=torch.int32)
    dev = lambda t: t.to("cuda", dtype).contiguous()
    cache = dev(torch.full((nb, 1, bs, cp + rp), 5.0))
    down = dev(torch.cat([_pad(dq, qp), _pad(dc, cp), _pad(dr, rp)], 1))
    cq = K.latent_rows(down, pos.cuda(), slots.cuda(), cache, dev(_pad(qw, qp)), dev(_pad(cw, cp)), freq, eps=1e-3, gain=gain,
                       q_real=q_rank, kv_real=kv_rank)
    _close(cq[:, :q_rank], P.rms(dq.double(), 1e-3) * qw.double(), dtype)
    assert cq[:, q_rank:].abs().sum() == 0
    keep = slots >= 0
    rows = cache[:, 0].flatten(0, 1)[slots[keep].long().cuda()]
    _close(rows[:, :kv_rank], (P.rms(dc.double(), 1e-3) * cw.double())[keep], dtype)
    tol = dict(f32_tol=3e-4)                         # angles up to 1000 radians in 32 bits
    _close(rows[:, cp:cp + rot], P.rotate(dr.double(), pos, spec)[keep], dtype, **tol)
    assert rows[:, kv_rank:cp].abs().sum() == 0 and rows[:, cp + rot:].abs().sum() == 0
    assert int((cache[:, 0] == 5.0).all(-1).sum()) == nb * bs - int(keep.sum())         # no other slot was touched
    qs = dev(torch.cat([torch.full((T, heads, 24), 3.0, dtype=torch.bfloat16), _pad(q, rp)], -1))
    qa = dev(torch.full((T, heads, 40 + rp), 9.0))
    K.latent_rotate(qs, pos.cuda(), freq, rp, out=qa, gain=gain)
    _close(qa[..., 40:40 + rot], P.rotate(q.double(), pos, spec), dtype, **tol)
    assert (qa[..., :40] == 9.0).all()
    K.latent_rotate(qs, pos.cuda(), freq, rp, gain=gain)
    assert torch.equal(qs[..., 24:], qa[..., 40:]) and (qs[..., :24] == 3.0).all()
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,H,N,Kd", [(1, 1, 8, 8), (3, 5, 24, 40), (16, 3, 512, 128), (33, 2, 72, 200), (130, 16, 136, 512)])
def test_matrices_per_head(dtype, M, H, N, Kd):
    from unillm_b200.ops import cuda_ops as K

    x, w = _rand(M, H, Kd + 16, seed=1), _rand(H, N, Kd, seed=2, scale=Kd ** -0.5)
    out = torch.full((M, H, N + 8), 7.0, device="cuda", dtype=dtype)
    K.gemm_heads(x.to("cuda", dtype)[..., 16:], w.to("cuda", dtype), out[..., :N])
    _close(out[..., :N], torch.einsum("mhk,hnk->mhn", x[..., 16:].double(), w.double()), dtype)
    assert (out[..., N:] == 7.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,T,N,Kd", [(4, 1, 40, 56), (4, 16, 256, 192), (4, 17, 64, 96), (3, 300, 136, 72), (4, 1000, 512, 256), (2, 4100, 136, 64)])
def test_stacked_products(dtype, E, T, N, Kd):
    from unillm_b200.ops import cuda_ops as K

    x, w = _rand(E, T, Kd, seed=1), _rand(E, N, Kd, seed=2, scale=Kd ** -0.5)
    got = K.gemm_stacked(x.to("cuda", dtype), w.to("cuda", dtype))
    _close(got, torch.einsum("etk,enk->etn", x.double(), w.double()), dtype)
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,Kd", [(1, 40, 56), (16, 72, 96), (40, 256, 192), (700, 1024, 256), (2048, 512, 1024)])
def test_xielu_epilogue(dtype, M, N, Kd):
    from unillm_b200.models.mixers import xielu_coefficients
    from unillm_b200.ops import cuda_ops as K

    x, w, act = _rand(M, Kd, seed=1), _rand(N, Kd, seed=2, scale=2 * Kd ** -0.5), torch.tensor([0.7, -1.2])
    got = K.gemm_tn(x.to("cuda", dtype), w.to("cuda", dtype), act="xielu", act_params=xielu_coefficients(act))
    _close(got, P.xielu(x.double() @ w.double().T, *act.double()), dtype)


# ------------------------------------------------------------------------------------------------
# attention over latents
# ------------------------------------------------------------------------------------------------
SIZES = [(4, 32, 8), (5, 24, 16), (16, 128, 32), (18, 264, 40), (35, 144, 24), (3, 400, 64), (16, 512, 64), (130, 64, 16)]


def _paged(lens, R, rot, bs=16, seed=0):
    """Random latents of several sequences in shuffled pages; unused slots hold a large value."""
    g = torch.Generator().manual_seed(seed)
    nb = sum((n + bs - 1) // bs for n in lens) + 3
    perm = torch.randperm(nb, generator=g).tolist()
    cache, bt = torch.full((nb, 1, bs, R + rot), 50.0), torch.full((len(lens), (max(lens) + bs - 1) // bs), -1, dtype=torch.int32)
    rows = []
    for s, n in enumerate(lens):
        rows.append(torch.randn(n, R + rot, generator=g).to(torch.bfloat16))
        for p in range(0, n, bs):
            bt[s, p // bs] = perm.pop()
    def fill():
        for s, n in enumerate(lens):
            for p in range(n):
                cache[bt[s, p // bs], 0, p % bs] = rows[s][p].float()
        return cache
    return rows, bt, fill


def _plant(rows, q, pos, key, h, scale):
    """Makes the score of query ``q[pos, h]`` with the row ``key`` stand out by 12."""
    n = q[pos, h].float()
    rows[key] = (n * (12.0 / (scale * n.pow(2).sum()))).to(torch.bfloat16)


def _plain_latent(q, rows, R, sinks, scale):
    """The rows are keys (latent and rotated part) and values of all heads: identity key and value matrices."""
    eye = torch.eye(R, dtype=torch.float64).expand(q.shape[1], R, R)
    return P.latent_attention(q[..., :R].double(), q[..., R:].double(), rows[:, :R].double(), rows[:, R:].double(), eye, eye,
                              sinks.double(), scale)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,R,rot", SIZES)
def test_prompt_attention(dtype, H, R, rot):
    """Portions of unequal sequences; keys that stand out at the start, at page and tile borders and at the query itself."""
    from unillm_b200.ops import cuda_ops as K

    lens, qlens, scale = [83, 5, 150, 17], [83, 2, 40, 1], 0.5 * (R + rot) ** -0.5
    rows, bt, fill = _paged(lens, R, rot, seed=R)
    q = [_rand(n, H, R + rot, seed=70 + i) for i, n in enumerate(lens)]
    for s, pos, key in ((0, 80, 0), (0, 70, 63), (0, 75, 64), (0, 40, 41), (2, 149, 128), (2, 130, 127), (2, 120, 15), (2, 111, 111), (3, 16, 16)):
        _plant(rows[s], q[s], pos, key, (pos + key) % H, scale)
    sinks = _rand(H, seed=9, dtype=torch.float32, scale=2.0)
    new = torch.cat([t[n - m:] for t, n, m in zip(q, lens, qlens)]).to("cuda", dtype)
    qs = _i32([0, *torch.tensor(qlens).cumsum(0).tolist()])
    cache = fill().to("cuda", dtype)
    for sk in (sinks, None):
        want = torch.cat([_plain_latent(a[n - m:], r, R, torch.full((H,), -1e4) if sk is None else sk, scale)
                          for a, r, n, m in zip(q, rows, lens, qlens)])
        got = K.attn_latent(new, cache, R, bt.cuda(), _i32(lens), scale=scale, q_start=qs, max_q_len=max(qlens),
                            sinks=None if sk is None else sk.cuda())
        _close(got, want, dtype, bf16_tol=2e-2)
        K.check_device_errors()


@pytest.mark.parametrize("H,dim,rot,vdim,R", [(3, 64, 32, 64, 128), (2, 128, 64, 128, 512), (5, 16, 8, 16, 24), (1, 112, 40, 48, 64),
                                              (4, 48, 16, 96, 72), (2, 80, 64, 112, 136)])
def test_prompt_attention_over_expanded_latents(H, dim, rot, vdim, R):
    """Gathered cache rows, expanded to keys and values of every head; keys that stand out at the start, at page and tile borders
    and at the query itself; rows of other sequences and behind the end in the same tiles."""
    from unillm_b200.ops import cuda_ops as K

    lens, qlens, scale, T = [300, 5, 150, 17, 129], [300, 2, 40, 1, 128], 0.5 * (dim + rot) ** -0.5, 471
    rows, bt, fill = _paged(lens, R, rot, seed=R)
    q = [_rand(n, H, dim + rot, seed=70 + i) for i, n in enumerate(lens)]
    wuk, wuv = _rand(H, dim, R, seed=3, scale=R ** -0.5), _rand(H, vdim, R, seed=4, scale=R ** -0.5)
    for s, pos, key in ((0, 280, 0), (0, 256, 127), (0, 299, 128), (0, 255, 256), (0, 128, 128), (0, 190, 63), (0, 130, 64), (2, 149, 15),
                        (2, 120, 120), (3, 16, 16), (4, 128, 127), (4, 127, 128)):
        h = (pos + key) % H                              # only the rotated part of a row is free to be chosen here
        n = q[s][pos, h, dim:].float()
        rows[s][key, R:] = (n * (14.0 / (scale * n.pow(2).sum()))).to(torch.bfloat16)
    sinks = _rand(H, seed=9, dtype=torch.float32, scale=2.0)
    cache = fill().cuda().to(torch.bfloat16)
    starts = [0]
    for n in lens:
        starts.append(starts[-1] + (n + 15) // 16)
    lat = K.latent_gather(cache, bt.cuda(), _i32(lens), _i32(starts), starts[-1] * 16 + 48)
    for s, n in enumerate(lens):
        a, z = starts[s] * 16, starts[s + 1] * 16
        assert torch.equal(lat[a:a + n].cpu(), rows[s]) and lat[a + n:z].abs().sum() == 0
    assert lat[starts[-1] * 16:].abs().sum() == 0
    kv = K.gemm_tn(lat[:, :R], torch.cat([wuk, wuv], 1).flatten(0, 1).cuda())
    new = torch.cat([t[n - m:] for t, n, m in zip(q, lens, qlens)]).cuda()
    qs = _i32([0, *torch.tensor(qlens).cumsum(0).tolist()])
    for sk in (sinks, None):
        want = torch.cat([P.latent_attention(a[n - m:, :, :dim].double(), a[n - m:, :, dim:].double(), r[:, :R].double(), r[:, R:].double(),
                                             wuk.double(), wuv.double(), torch.full((H,), -1e4) if sk is None else sk.double(), scale)
                          for a, r, n, m in zip(q, rows, lens, qlens)])
        got = K.attn_expanded(new, kv, lat, vdim, _i32(lens), qs, _i32(starts), max(qlens), scale=scale, sinks=None if sk is None else sk.cuda())
        _close(got, want, torch.bfloat16, bf16_tol=2e-2)
        K.check_device_errors()
    assert got.shape == (T, H, vdim)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,R,rot", SIZES)
@pytest.mark.parametrize("splits", [1, 3, 8])
def test_decode_attention(dtype, H, R, rot, splits):
    from unillm_b200.ops import cuda_ops as K

    lens, scale = [1, 16, 17, 64, 333, 65], 0.5 * (R + rot) ** -0.5
    rows, bt, fill = _paged(lens, R, rot, seed=R + splits)
    q = [_rand(1, H, R + rot, seed=170 + i) for i, n in enumerate(lens)]
    for s, n in enumerate(lens):
        for key in (0, n - 1, 48, 200):
            if key < n and (s + key) % 2 == 0:
                _plant(rows[s], q[s], 0, key, (H - 1 + key) % H, scale)
    sinks = _rand(H, seed=9, dtype=torch.float32, scale=2.0)
    cache, new = fill().to("cuda", dtype), torch.cat(q).to("cuda", dtype)
    for sk in (sinks, None):
        want = torch.cat([_plain_latent(a, r, R, torch.full((H,), -1e4) if sk is None else sk, scale) for a, r in zip(q, rows)])
        got = K.attn_latent(new, cache, R, bt.cuda(), _i32(lens), scale=scale, splits=splits, sinks=None if sk is None else sk.cuda())
        _close(got, want, dtype, bf16_tol=2e-2)
        K.check_device_errors()


# ------------------------------------------------------------------------------------------------
# the serving engine
# ------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=sorted(C.CASES))
def case(request):
    cfg = C.CASES[request.param]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 200, 1)
    return cfg, w, C.load_model(cfg, w), toks, P.forward(cfg, w, toks)


def _engine(m, dtype, blocks=16, **kw):
    from unillm_b200.engine.factory import build_engine

    o = dict(max_num_seqs=4, max_num_batched_tokens=256, max_model_len=256, use_cuda_graphs=False, enable_prefix_caching=False)
    o.update(kw)
    return build_engine(m, device="cuda", dtype=dtype, num_blocks=blocks, **o)


def _check_rows(got, want, dtype):
    err = C.row_error(got, want)
    if dtype == torch.float32:
        assert err.max() < 5e-4 and err.median() < 3e-5, (err.max(), err.median())
    else:                                            # no dtype: a handful of rows, whose median says little
        assert (dtype is None or err.median() < 0.06) and err.max() < 0.35, (err.median(), err.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[200], [1], [2], [3, 1, 2], [16], [17, 2, 31], [64, 1], [150] + [1] * 50])
def test_portions_and_decoding(case, dtype, sizes):
    """Whole prompts, portions down to two tokens, token by token, and a long decoded tail give the same logits."""
    _, _, m, toks, ref = case
    eng = _engine(m, dtype)
    got = C.score(eng, toks, C.portions(len(toks), sizes))
    eng.runner.raise_on_device_error()
    _check_rows(got, ref, dtype)
    whole = C.score(eng, toks, [(0, len(toks))])
    err = C.row_error(got, whole)
    assert err.max() < 5e-4 if dtype == torch.float32 else err.median() < 0.06


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_with_blocks_and_slots_used_again(case, dtype):
    cfg, w, m, _, _ = case
    seqs = {k: C.tokens(cfg, n, 10 + k) for k, n in C.BATCH.items()}
    eng = _engine(m, dtype, blocks=11, max_num_seqs=3)
    got = C.score_batch(eng, seqs, C.BATCH_SIZES)
    eng.runner.raise_on_device_error()
    assert eng.pool.num_free() == 11 and (eng.slots is None or eng.slots.num_free() == 3)
    alone = _engine(m, dtype)
    for k in seqs:
        want = P.forward(cfg, w, seqs[k])
        _check_rows(got[k], want, dtype if dtype == torch.float32 or len(seqs[k]) > 40 else None)
        err = C.row_error(got[k], C.score(alone, seqs[k], [(0, len(seqs[k]))]))
        assert err.max() < (5e-4 if dtype == torch.float32 else 0.3)


def _greedy(cfg, w, prompt, n):
    out = []
    for _ in range(n):
        out.append(int(P.forward(cfg, w, prompt + out)[-1].argmax()))
    return out


@pytest.mark.parametrize("graphs,ahead", [(False, False), (True, False), (True, True)])
def test_greedy_generation(case, graphs, ahead):
    """Requests through the scheduler (chunked prompts, a pool too small for all, CUDA graphs, the host one step ahead), in 32
    bits token for token; in bf16 graphs and plain launches agree."""
    from unillm_b200.sampling import SamplingParams

    cfg, w, m, _, _ = case
    prompts = [C.tokens(cfg, n, 30 + n) for n in (19, 3, 34, 1, 50)]
    prompts.append(prompts[4][:40])
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    kw = dict(blocks=9, max_num_batched_tokens=24, use_cuda_graphs=graphs, async_scheduling=ahead, enable_prefix_caching=True)
    eng = _engine(m, torch.float32, **kw)
    assert eng.generate(prompts, sp) == [_greedy(cfg, w, p, 6) for p in prompts]
    eng.runner.raise_on_device_error()
    half = _engine(m, torch.bfloat16, **kw).generate(prompts, sp)
    plain = _engine(m, torch.bfloat16, **{**kw, "use_cuda_graphs": False, "async_scheduling": False}).generate(prompts, sp)
    same = sum(a == b for x, y in zip(half, plain) for a, b in zip(x, y))
    assert same >= 0.7 * 36


def test_pipeline_serves_on_the_kernels(case):
    from unillm_b200.config import GenerationConfig
    from unillm_b200.pipeline import InferencePipelineBuilder

    cfg, w, m, toks, _ = case
    pipe = InferencePipelineBuilder().model(m).device("cuda").engine_options(max_num_seqs=2, max_model_len=256, num_blocks=32,
                                                                             dtype=torch.float32).build()
    got = pipe.generate_tokens(toks[:21], GenerationConfig.greedy(5, eos_token_id=-1))
    assert pipe.engine_kind == "gpu-kernels" and got == _greedy(cfg, w, toks[:21], 5)


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
        assert C.row_error(got.double(), ref[rows]).max() < (5e-4 if dtype == "float32" else 0.25)
