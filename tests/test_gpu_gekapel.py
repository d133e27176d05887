"""Gekapel on the GPU: each mechanism's kernel alone and the serving engine on them, against the plain statement."""
import os
import subprocess
import sys

import pytest
import torch

import gekapel_cases as C
import gekapel_plain as P

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


# ------------------------------------------------------------------------------------------------
# mechanisms
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H", [(1, 8), (3, 50), (5, 136), (7, 1000), (4, 4096), (2, 9000)])
@pytest.mark.parametrize("kind", ["layer", "rms"])
def test_residual_norm(dtype, T, H, kind):
    from unillm_b200.ops import cuda_ops as K

    Hp, Kx = (H + 7) // 8 * 8, 3
    pad = lambda t: torch.nn.functional.pad(t, (0, Hp - H))
    x, y, yx = _rand(T, H, seed=1, dtype=torch.float32, scale=3.0), _rand(T, H, seed=2), _rand(T * Kx, H, seed=3)
    w, b = _rand(H, seed=4) + 1, _rand(H, seed=5)
    r = K.MoeRouting(T, Kx, 4, 16, "cuda")
    g = torch.Generator().manual_seed(6)
    slots = torch.randperm(T * Kx, generator=g).int().reshape(T, Kx)
    slots[0, 1] = -1                                                # a choice without a row
    wt = torch.rand(T, Kx, generator=g)
    r.row_slot.copy_(slots.flatten()), r.topk_w.copy_(wt)
    dev = lambda t: pad(t).to("cuda", dtype).contiguous()
    norm = (lambda z: P.layer_norm(z, w.double(), b.double(), 1e-4)) if kind == "layer" else \
        (lambda z: P.rms_norm(z, w.double(), 1e-4))
    mix = torch.stack([sum(wt[t, k].double() * yx[slots[t, k]].double() for k in range(Kx) if slots[t, k] >= 0) for t in range(T)])
    for base, experts, rows in ((y, None, y.double()), (y, yx, y.double() + mix), (None, yx, mix)):
        xs = pad(x).cuda().contiguous()
        out = K.residual_norm(xs, None if base is None else dev(base), dev(w), dev(b) if kind == "layer" else None, eps=1e-4,
                              kind=kind, width=H, experts=None if experts is None else dev(experts),
                              routing=None if experts is None else r)
        want = x.double() + norm(rows)
        _close(xs[:, :H], want, torch.float32, f32_tol=1e-5)
        _close(out[:, :H], want, dtype)
        assert xs[:, H:].abs().sum() == 0 and out[:, H:].abs().sum() == 0
    pick = torch.tensor([T - 1, 0, T - 1], dtype=torch.int32)
    out = K.row_norm(pad(x).cuda().contiguous(), dev(w), dev(b) if kind == "layer" else None, eps=1e-4, kind=kind, width=H,
                     rows=pick.cuda())
    _close(out[:, :H], norm(x.double())[pick.long()], dtype)
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
def test_embed_residual_and_bad_ids(dtype):
    from unillm_b200.ops import cuda_ops as K

    table = _rand(37, 56, seed=1)
    ids = torch.tensor([36, 0, 5, 5], dtype=torch.int32)
    x, h = K.embed_residual(ids.cuda(), table.to("cuda", dtype))
    assert torch.equal(x.cpu(), table[ids.long()].float()) and torch.equal(h.float().cpu(), table[ids.long()].float())
    K.check_device_errors()
    K.embed_residual(torch.tensor([37], dtype=torch.int32).cuda(), table.to("cuda", dtype))
    with pytest.raises(RuntimeError):
        K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hq,Hkv,dim,vdim,dims", [(6, 3, 64, 64, 24), (6, 2, 32, 48, 8), (5, 5, 20, 12, 6), (3, 1, 40, 24, 40),
                                                  (2, 1, 128, 96, 64), (2, 1, 192, 256, 2), (1, 1, 16, 8, 0), (18, 1, 72, 136, 72)])
@pytest.mark.parametrize("scaled", [True, False])
def test_head_norm_rotation_and_append(dtype, Hq, Hkv, dim, vdim, dims, scaled):
    from unillm_b200.ops import cuda_ops as K
    from unillm_b200.precompute import rope_inv_freq

    r8 = lambda n: (n + 7) // 8 * 8
    dp, vp, T, bs, nb = r8(dim), r8(vdim), 9, 16, 7
    rot = {"base": 700.0, "dims": dims}
    if scaled:
        rot["scaling"] = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 200}
    q, k, v = _rand(T, Hq, dim, seed=1, scale=2.0), _rand(T, Hkv, dim, seed=2), _rand(T, Hkv, vdim, seed=3)
    qw, kw = _rand(dim, seed=4) + 1, _rand(dim, seed=5) + 1
    pos = torch.tensor([0, 1, 15, 16, 17, 300, 299, 1000, 3], dtype=torch.int32)
    slots = torch.tensor([40, 0, 111, -1, 16, 15, 3, 77, 50], dtype=torch.int32)
    want_q = P.rotate(P.rms_norm(q.double(), qw.double(), 1e-3), pos, rot)
    want_k = P.rotate(P.rms_norm(k.double(), kw.double(), 1e-3), pos, rot)
    padh = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1])).reshape(T, -1)
    dev = lambda t: t.to("cuda", dtype).contiguous()
    kc, vc = dev(torch.zeros(nb, Hkv, bs, dp)), dev(torch.zeros(nb, Hkv, bs, vp))
    l3 = tuple(rot["scaling"][n] for n in ("factor", "low", "high", "original")) if scaled else None
    table = rope_inv_freq(dims, 700.0, l3).cuda() if dims else None
    nw = lambda t: dev(torch.nn.functional.pad(t, (0, dp - dim)))
    kw_ = dict(head_dim=dp, rotary_dim=dims, interleaved=True, norm_eps=1e-3, v_head_dim=vp, norm_dim=dim, inv_freq=table)
    qkv = dev(torch.cat([padh(q, dp), padh(k, dp), padh(v, vp)], 1))
    K.rope_kv_append(qkv, pos.cuda(), slots.cuda(), kc, vc, num_q_heads=Hq, num_kv_heads=Hkv, q_norm_w=nw(qw), k_norm_w=nw(kw),
                     k_cache_only=True, **kw_)
    got = qkv[:, :Hq * dp].reshape(T, Hq, dp)
    tol = dict(f32_tol=3e-4)                         # angles up to 1000 radians in 32 bits
    _close(got[..., :dim], want_q, dtype, **tol)
    assert got[..., dim:].abs().sum() == 0
    keep = slots >= 0
    at = slots[keep].long()
    _close(kc[at // bs, :, at % bs][..., :dim], want_k[keep], dtype, **tol)
    _close(vc[at // bs, :, at % bs][..., :vdim], v.double()[keep], dtype)
    assert int((vc.abs().sum((1, 3)) > 0).sum()) == int(keep.sum())          # no other slot was touched
    only_q = dev(padh(q, dp))
    K.rope_kv_append(only_q, pos.cuda(), None, None, None, num_q_heads=Hq, num_kv_heads=0, q_norm_w=nw(qw), **kw_)
    assert torch.equal(only_q.reshape(T, Hq, dp), got)
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,top,H,bias", [(5, 2, 96, True), (7, 7, 56, True), (1, 1, 8, True), (64, 8, 1024, True), (256, 16, 64, False)])
@pytest.mark.parametrize("T", [1, 21, 1501])
def test_router(dtype, E, top, H, bias, T):
    from unillm_b200.ops import cuda_ops as K

    x, w = _rand(T, H, seed=1, dtype=torch.float32, scale=2.0), _rand(E, H, seed=2, scale=H ** -0.5)
    b = _rand(E, seed=3) if bias else torch.zeros(E)
    idx, wt = P.route(x.double(), w.double(), b.double(), top)
    r = K.moe_route(x.cuda(), w.to("cuda", dtype), top, round_logits_bf16=False, router_b=b.to("cuda", dtype) if bias else None)
    got = torch.zeros(T, E, dtype=torch.float64).scatter_(1, r.topk_ids.cpu().long(), r.topk_w.cpu().double())
    want = torch.zeros(T, E, dtype=torch.float64).scatter_(1, idx, wt)
    assert (got - want).abs().max() < 1e-5
    # expert order: every (token, choice) pair has a slot of its own inside its expert's rows, covered by the tile table
    ids, slot, off = r.topk_ids.cpu().flatten().long(), r.row_slot.cpu().long(), r.offsets.cpu().long()
    assert torch.equal(slot.sort().values, torch.arange(T * top)) and torch.equal(r.sorted_rows.cpu().long()[slot], torch.arange(T * top))
    assert ((slot >= off[ids]) & (slot < off[ids + 1])).all()
    assert torch.equal(r.counts.cpu().long(), torch.bincount(ids, minlength=E))
    tiles = [t for t in r.tiles.cpu().tolist() if t[0] >= 0]
    covered = [(e, x) for e, a, z, _ in tiles for x in range(a, min(z, a + r.tile_tokens))]
    assert len(covered) == T * top and all(off[e] <= x < off[e + 1] for e, x in covered)
    K.check_device_errors()


@pytest.mark.parametrize("M,N,Kd", [(1, 1, 8), (3, 37, 50), (65, 129, 40), (200, 64, 4096)])
@pytest.mark.parametrize("form", ["plain", "gated"])
def test_gemm_in_32_bits(M, N, Kd, form):
    from unillm_b200.ops import cuda_ops as K

    x = _rand(M, Kd, seed=1, dtype=torch.float32)
    w = _rand(2 * N if form == "gated" else N, Kd, seed=2, dtype=torch.float32, scale=Kd ** -0.5)
    if form == "gated":
        got = K.gemm_tn(x.cuda(), w.cuda(), dual_rows=N, act="silu")
        g, u = (x.double() @ w.double().T).chunk(2, 1)
        want = g * torch.sigmoid(g) * u
    else:
        b, res = _rand(N, seed=3, dtype=torch.float32), _rand(M, N, seed=4, dtype=torch.float32)
        got = K.gemm_tn(x.cuda(), w.cuda(), bias=b.cuda(), residual=res.cuda(), act="relu2")
        want = P.relu2(x.double() @ w.double().T + b.double()) + res.double()
    _close(got, want, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,top,H,ff,T", [(5, 2, 96, 40, 33), (3, 3, 56, 8, 1), (4, 1, 136, 200, 300), (12, 3, 256, 72, 7)])
def test_squared_relu_experts(dtype, E, top, H, ff, T):
    from unillm_b200.ops import cuda_ops as K

    x, w = _rand(T, H, seed=1), {}
    w["m.router"], w["m.router.b"] = _rand(E, H, seed=2, scale=2 * H ** -0.5), _rand(E, seed=3)
    for e in range(E):
        w[f"m.e{e}.up"], w[f"m.e{e}.down"] = _rand(ff, H, seed=10 + e, scale=H ** -0.5), _rand(H, ff, seed=50 + e, scale=ff ** -0.5)
    want = P.mixture(x.double(), {n: t.double() for n, t in w.items()}, "m", {"router": {"top": top}})
    dev = lambda t: t.to("cuda", dtype).contiguous()
    r = K.moe_route(x.float().cuda(), dev(w["m.router"]), top, round_logits_bf16=False, router_b=dev(w["m.router.b"]))
    up, dn = dev(torch.stack([w[f"m.e{e}.up"] for e in range(E)])), dev(torch.stack([w[f"m.e{e}.down"] for e in range(E)]))
    y = K.grouped_gemm(K.grouped_gemm(K.moe_gather(dev(x), r), up, r, act="relu2"), dn, r).cpu().double()
    slot, wt = r.row_slot.cpu().reshape(T, top), r.topk_w.cpu().double()
    got = sum(wt[:, k:k + 1] * y[slot[:, k].long()] for k in range(top))
    _close(got, want, dtype, bf16_tol=3e-2)
    K.check_device_errors()


# ------------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------------
def _paged(lens, Hkv, dim, vdim, dtype, bs=16, seed=0):
    """Random keys and values of several sequences in shuffled pages; unused slots hold a large value."""
    g = torch.Generator().manual_seed(seed)
    nb = sum((n + bs - 1) // bs for n in lens) + 3
    perm = torch.randperm(nb, generator=g).tolist()
    kc, vc = torch.full((nb, Hkv, bs, dim), 50.0), torch.full((nb, Hkv, bs, vdim), 50.0)
    bt = torch.full((len(lens), (max(lens) + bs - 1) // bs), -1, dtype=torch.int32)
    ks, vs = [], []
    for s, n in enumerate(lens):
        k, v = (torch.randn(n, Hkv, d, generator=g).to(torch.bfloat16) for d in (dim, vdim))
        ks.append(k), vs.append(v)
        for p in range(n):
            if p % bs == 0:
                bt[s, p // bs] = perm.pop()
            kc[bt[s, p // bs], :, p % bs], vc[bt[s, p // bs], :, p % bs] = k[p].float(), v[p].float()
    dev = lambda t: t.to("cuda", dtype)
    return kc, vc, bt, ks, vs, dev


SIZES = [(6, 2, 64, 64), (4, 1, 128, 128), (6, 2, 32, 48), (5, 5, 24, 16), (18, 1, 72, 136), (2, 1, 192, 256), (4, 2, 256, 64), (3, 3, 8, 200)]


def _plant(k, q, pos, h, g, scale):
    """Makes the score of query ``q[pos, h]`` with key ``k[.., g]`` at the returned place stand out by 12."""
    n = q[pos, h].float()
    return (n * (12.0 / (scale * n.pow(2).sum()))).to(torch.bfloat16)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hq,Hkv,dim,vdim", SIZES)
@pytest.mark.parametrize("window", [1, 16, 21, 64, 0])
def test_prompt_attention(dtype, Hq, Hkv, dim, vdim, window):
    """Portions of unequal sequences with sinks; keys that stand out just inside and just outside the window, at page
    borders and at the very start."""
    from unillm_b200.ops import cuda_ops as K

    lens, qlens, scale = [83, 5, 130, 17], [83, 2, 40, 1], 0.5 * dim ** -0.5
    kc, vc, bt, ks, vs, dev = _paged(lens, Hkv, dim, vdim, dtype, seed=window)
    q = [_rand(n, Hq, dim, seed=70 + i) for i, n in enumerate(lens)]
    per = Hq // Hkv
    for s, pos, key in ((0, 80, 80 - window), (0, 70, 70 - window + 1), (2, 120, 120 - window), (2, 110, 110 - window + 1), (2, 100, 0),
                        (2, 127, 112), (2, 95, 95), (3, 16, 15)):
        if 0 <= key <= pos and window >= 0:
            ks[s][key, 0] = _plant(ks[s], q[s], pos, per - 1, 0, scale)
            kc[bt[s, key // 16], 0, key % 16] = ks[s][key, 0].float()
    sinks = _rand(Hq, seed=9, dtype=torch.float32, scale=2.0)
    rows = torch.cat([t[n - m:] for t, n, m in zip(q, lens, qlens)])
    qs = torch.tensor([0, *torch.tensor(qlens).cumsum(0).tolist()], dtype=torch.int32).cuda()
    i32 = lambda t: torch.as_tensor(t, dtype=torch.int32).cuda()
    want = torch.cat([P.window_attention(a.double(), k.double(), v.double(), sinks.double(), scale, window or None)[n - m:]
                      for a, k, v, n, m in zip(q, ks, vs, lens, qlens)])
    for sk in (sinks, None):
        if sk is None:
            want = torch.cat([P.window_attention(a.double(), k.double(), v.double(), torch.full((Hq,), -1e4, dtype=torch.float64),
                                                 scale, window or None)[n - m:] for a, k, v, n, m in zip(q, ks, vs, lens, qlens)])
        got = K.attn_prefill(dev(rows), dev(kc), dev(vc), bt.cuda(), i32(lens), qs, max(qlens), scale=scale, window=window,
                             sinks=None if sk is None else sk.cuda())
        _close(got, want, dtype)
        K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hq,Hkv,dim,vdim", SIZES)
@pytest.mark.parametrize("window,splits", [(1, 1), (16, 1), (21, 1), (300, 1), (300, 4), (0, 1), (0, 8), (64, 3)])
def test_decode_attention(dtype, Hq, Hkv, dim, vdim, window, splits):
    from unillm_b200.ops import cuda_ops as K

    lens, scale = [1, 16, 17, 64, 333, 65], 0.5 * dim ** -0.5
    kc, vc, bt, ks, vs, dev = _paged(lens, Hkv, dim, vdim, dtype, seed=window + splits)
    q = [_rand(n, Hq, dim, seed=170 + i) for i, n in enumerate(lens)]
    for s, n in enumerate(lens):
        for key in ((n - 1 - window, n - window, 0, 48) if window else (0, n - 1)):
            if 0 <= key < n and (s + key) % 2 == 0:
                ks[s][key, -1] = _plant(ks[s], q[s], n - 1, Hq - 1, 0, scale)
                kc[bt[s, key // 16], -1, key % 16] = ks[s][key, -1].float()
    sinks = _rand(Hq, seed=9, dtype=torch.float32, scale=2.0)
    last = torch.stack([t[-1] for t in q])
    i32 = lambda t: torch.as_tensor(t, dtype=torch.int32).cuda()

    def plain(sk):
        out = []
        for a, k, v in zip(q, ks, vs):
            n = k.shape[0]
            lo = max(0, n - window) if window else 0
            pad = torch.zeros(n - lo, *a.shape[1:], dtype=torch.float64)
            pad[-1] = a[-1].double()
            out.append(P.window_attention(pad[-1:].expand(1, -1, -1).repeat(n - lo, 1, 1), k[lo:].double(), v[lo:].double(),
                                          sk.double(), scale, None)[-1])
        return torch.stack(out)

    for sk in (sinks, None):
        want = plain(sinks if sk is not None else torch.full((Hq,), -1e4))
        got = K.attn_decode(dev(last), dev(kc), dev(vc), bt.cuda(), i32(lens), scale=scale, window=window, splits=splits,
                            sinks=None if sk is None else sk.cuda())
        _close(got, want, dtype)
        K.check_device_errors()


# ------------------------------------------------------------------------------------------------
# the serving engine
# ------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=sorted(C.CASES))
def case(request):
    cfg = C.CASES[request.param]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 150, 1)
    return cfg, w, C.load_model(cfg, w), toks, P.forward(cfg, w, toks)


def _engine(m, dtype, blocks=16, **kw):
    from unillm_b200.engine.factory import build_engine

    o = dict(max_num_seqs=4, max_num_batched_tokens=256, max_model_len=256, use_cuda_graphs=False, enable_prefix_caching=False)
    o.update(kw)
    return build_engine(m, device="cuda", dtype=dtype, num_blocks=blocks, **o)


def _check_rows(got, want, dtype):
    """32-bit: every row.  bf16: a router's close call may go the other way for single tokens of these random weights (and
    nudge the tokens that attend to them), so the bulk of the rows carries the test."""
    err = C.row_error(got, want)
    if dtype == torch.float32:
        assert err.max() < 5e-4 and err.median() < 2e-5, (err.max(), err.median())
    else:
        assert err.median() < 0.03 and (err < 0.12).float().mean() > 0.8, (err.median(), err.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[150], [1], [2], [3, 1, 2], [16], [17, 2, 31], [64, 1], [120] + [1] * 30])
def test_portions_and_decoding(case, dtype, sizes):
    """Whole prompts, portions down to two tokens, token by token, and a long decoded tail give the same logits."""
    _, _, m, toks, ref = case
    eng = _engine(m, dtype)
    got = C.score(eng, toks, C.portions(len(toks), sizes))
    eng.runner.raise_on_device_error()
    _check_rows(got, ref, dtype)
    whole = C.score(eng, toks, [(0, len(toks))])
    if dtype == torch.float32:
        assert C.row_error(got, whole).max() < 5e-4
    else:
        assert C.row_error(got, whole).median() < 0.03


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_with_blocks_used_again(case, dtype):
    cfg, w, m, _, _ = case
    seqs = {k: C.tokens(cfg, n, 10 + k) for k, n in enumerate((61, 7, 33, 1, 48, 16, 2))}
    want = {k: P.forward(cfg, w, t) for k, t in seqs.items()}
    eng = _engine(m, dtype, blocks=11)
    sizes = {0: [5, 1, 2], 1: [1], 2: [17, 1], 3: [1], 4: [2, 31], 5: [16], 6: [2]}
    cuts = {k: C.portions(len(t), sizes[k]) for k, t in seqs.items()}
    queue, live, got = list(seqs), [], {k: [] for k in seqs}
    while queue or live:
        while queue and len(live) < 3:
            live.append(queue.pop(0))
        step = [(k, cuts[k].pop(0)) for k in live]
        done = [k for k, (_, b) in step if b == len(seqs[k])]
        out = eng.score_step([(k, seqs[k][a:b], range(b - a)) for k, (a, b) in step], done).double().cpu()
        for k, (a, b) in step:
            got[k].append(out[:b - a])
            out = out[b - a:]
        live = [k for k in live if k not in done]
    eng.runner.raise_on_device_error()
    assert eng.pool.num_free() == 11
    _check_rows(torch.cat([torch.cat(got[k]) for k in seqs]), torch.cat([want[k] for k in seqs]), dtype)


def _greedy(cfg, w, prompt, n):
    out = []
    for _ in range(n):
        out.append(int(P.forward(cfg, w, prompt + out)[-1].argmax()))
    return out


@pytest.mark.parametrize("graphs,ahead", [(False, False), (True, False), (True, True)])
def test_greedy_generation(case, graphs, ahead):
    """Requests through the scheduler (chunked prompts, a pool too small for all, prefix cache, CUDA graphs, the host one
    step ahead), in 32 bits token for token; in bf16 graphs and plain launches agree."""
    from unillm_b200.sampling import SamplingParams

    cfg, w, m, _, _ = case
    prompts = [C.tokens(cfg, n, 30 + n) for n in (19, 3, 34, 1, 50)]
    prompts.append(prompts[4][:40])
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    kw = dict(blocks=14, max_num_batched_tokens=24, use_cuda_graphs=graphs, async_scheduling=ahead, enable_prefix_caching=True)
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
def test_trace_runner(tmp_path, case, dtype):
    import json

    cfg, w, _, toks, ref = case
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
        err = C.row_error(got.double(), ref[rows])
        assert err.max() < (5e-4 if dtype == "float32" else 0.3)


def test_windowed_batch_with_a_shared_prefix():
    """Ten sequences that share their first blocks and have outgrown the window: the shared-prefix pass, which knows no
    window, must not be taken."""
    from unillm_b200.engine.cpu_runner import CpuModelRunner
    from unillm_b200.engine.llm_engine import LLMEngine
    from unillm_b200.engine.runner import GpuModelRunner, RunnerWeights
    from unillm_b200.models import configs as CF
    from unillm_b200.models.families import MistralModel
    from unillm_b200.sampling import SamplingParams

    cfg = CF.MistralConfig().replace(vocab_size=256, hidden_size=128, intermediate_size=128, num_hidden_layers=2, num_attention_heads=2,
                                     num_key_value_heads=1, sliding_window=24, initializer_range=0.1)
    m = MistralModel.new(cfg, init="random", seed=3)
    m.p = {k: v.to(torch.bfloat16).float() for k, v in m.p.items()}
    g = torch.Generator().manual_seed(1)
    shared = torch.randint(0, 256, (96,), generator=g).tolist()
    prompts = [shared + torch.randint(0, 256, (n,), generator=g).tolist() for n in range(3, 13)]
    res = []
    for gpu in (False, True):
        if gpu:
            run = GpuModelRunner(m.spec, RunnerWeights(m.spec, m.p, "cuda"), num_blocks=64, max_num_seqs=16, max_num_batched_tokens=256,
                                 max_model_len=256, use_cuda_graphs=False)
        else:
            run = CpuModelRunner(m, num_blocks=64, max_model_len=256)
        eng = LLMEngine(run, num_blocks=64, max_num_seqs=16, max_num_batched_tokens=256, max_model_len=256)
        res.append(eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)))
    same = sum(a == b for x, y in zip(*res) for a, b in zip(x, y))
    assert same >= 0.75 * 80, same
