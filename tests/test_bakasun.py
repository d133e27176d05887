"""Bakasun on the host: reading a model directory, the whole-model path, and the serving engine with its block pool, state
slots and batching (fp32 CPU runner) against the plain statement of the design; the plain statement's own sensitivity."""
import copy

import pytest
import torch

import bakasun_cases as C
import bakasun_plain as P

TOL = 3e-5


@pytest.fixture(scope="module", params=sorted(C.CASES))
def case(request):
    cfg = C.CASES[request.param]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 70, 1)
    return request.param, cfg, w, C.load_model(cfg, w), toks, P.forward(cfg, w, toks)


def _engine(m, blocks=16, **kw):
    from unillm_b200.engine.factory import build_cpu_engine

    return build_cpu_engine(m, num_blocks=blocks, **kw)


def test_model_directory_loads_and_exports(tmp_path, case):
    from unillm_b200.models import BakasunModel
    from unillm_b200.weights import ModelLoader

    _, cfg, w, _, toks, ref = case
    m = ModelLoader().load_model(C.write_model(tmp_path / "m", cfg, w))
    assert isinstance(m, BakasunModel)
    with torch.no_grad():
        y = m.forward_with_cache(torch.tensor(toks))[0]
    assert C.row_error(y.double(), ref).max() < TOL
    out = m.export_hf().tensors
    assert set(out) == set(w)
    assert all(torch.equal(out[n].float(), t.float()) for n, t in w.items())


def test_layers_one_by_one(case):
    _, cfg, w, m, toks, _ = case
    _, after = P.forward(cfg, w, toks[:30], keep_layers=True)
    with torch.no_grad():
        x = m.p["embed"][torch.tensor(toks[:30])][None]
        for i in range(m.spec.num_layers):
            st = {}
            x = m.block(i, x, lambda h: m.mixer(i, h, 0, None, {}, st))
            assert (x[0].double() - after[i]).abs().max() < 1e-4 * after[i].abs().max(), i


def test_whole_model_path_continues_from_its_cache(case):
    _, _, _, m, toks, ref = case
    cache, got = m.new_cache(128), []
    with torch.no_grad():
        for a, b in C.portions(len(toks), [9, 1, 2, 1]):
            got.append(m.forward_with_cache(torch.tensor(toks[a:b]), cache)[0])
    assert C.row_error(torch.cat(got).double(), ref).max() < TOL
    cache.clear()
    with torch.no_grad():
        again = m.forward_with_cache(torch.tensor(toks), cache)[0]
    assert C.row_error(again.double(), ref).max() < TOL


def test_costs_of_cache_and_state(case):
    from unillm_b200.engine.runner import RunnerWeights
    from unillm_b200.scheduler.policies import KvShape

    _, cfg, _, m, _, _ = case
    row = state = 0
    for x in cfg["layers"]:
        a = x["mixer"] if x["type"] == "attention" else x["mixer"]["left"]
        row += a["kv_heads"] * (a["dim"] + a["vdim"])
        if x["type"] == "parallel":
            r = x["mixer"]["right"]
            state += r["heads"] * r["dim"] * r["vdim"] + (r["conv"] - 1) * (2 * r["kv_heads"] * r["dim"] + r["heads"] * r["vdim"])
    assert KvShape.from_spec(m.spec).bytes_per_token() == 2 * row
    assert m.spec.state_elements == state and m.spec.has_state == (state > 0)
    rw = RunnerWeights(m.spec, m.p, "cpu")
    assert rw.state_bytes_per_seq() >= 8 * state and rw.kv_bytes_per_token() >= 2 * row


def test_random_kernel_weights_have_the_loaded_ones_shapes(case):
    from unillm_b200.engine.runner import RunnerWeights

    _, cfg, _, m, _, _ = case
    if cfg["width"] % 8:
        pytest.skip("random weights are for widths that need no padding")
    a, b = RunnerWeights(m.spec, m.p, "cpu"), RunnerWeights.random(m.spec, "cpu")
    assert all(n in b.t and (b.t[n].shape, b.t[n].dtype) == (t.shape, t.dtype) for n, t in a.t.items())


def _first(cfg, kind):
    return next(x for x in cfg["layers"] if x["type"] == kind)


def test_bad_configurations_are_refused():
    from unillm_b200.types import ConfigurationError

    edits = [lambda c: c["layers"][0].update(type="latent"), lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
             lambda c: c["layers"][0]["mixer"].update(kv_heads=3), lambda c: _first(c, "parallel")["mixer"]["right"].update(kv_heads=3),
             lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
             lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5), lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=5),
             lambda c: c["layers"][1]["mlp"]["router"].update(top=7)]
    for edit in edits:
        cfg = copy.deepcopy(C.CASES["mixed"])
        edit(cfg)
        with pytest.raises(ConfigurationError):
            C.load_model(cfg, {})


@pytest.mark.parametrize("missing", ["l0.mix.q.norm", "l1.mix.left.k", "l1.mix.right.v.conv", "l1.mix.right.A_log", "l1.mlp.correction",
                                     "l1.mlp.shared.sg", "l1.mlp.e11.up", "l0.norm2b", "l2.mix.right.o"])
def test_missing_tensors_are_named(missing):
    from unillm_b200.types import LoadingError

    w = C.make_weights(C.CASES["mixed"])
    del w[missing]
    with pytest.raises(LoadingError):
        C.load_model(C.CASES["mixed"], w)


@pytest.mark.parametrize("sizes", [[70], [1], [2], [3, 1, 2], [17, 2, 31]])
def test_portions_through_the_engine(case, sizes):
    _, _, _, m, toks, ref = case
    got = C.score(_engine(m), toks, C.portions(len(toks), sizes))
    assert C.row_error(got, ref).max() < TOL


def test_unequal_batch_with_blocks_and_slots_used_again(case):
    """Sequences in one batch, in portions of different sizes; finished ones make room for others in a pool and in state
    slots that hold no more than the live ones need."""
    _, cfg, w, m, _, _ = case
    seqs = {k: C.tokens(cfg, n, 10 + k) for k, n in C.BATCH.items()}
    eng = _engine(m, blocks=11, max_num_seqs=3)
    got = C.score_batch(eng, seqs, C.BATCH_SIZES)
    assert eng.pool.num_free() == 11 and (eng.slots is None or eng.slots.num_free() == 3)
    for k in seqs:
        assert C.row_error(got[k], P.forward(cfg, w, seqs[k])).max() < TOL, k


def test_a_sequence_may_pause(case):
    _, cfg, w, m, toks, ref = case
    eng, other = _engine(m), C.tokens(cfg, 30, 5)
    a = eng.score_step([("x", toks[:11], range(11))])
    b = eng.score_step([("y", other[:30], range(30))], ["y"])
    c = eng.score_step([("x", toks[11:12], [0]), ("z", other[:1], [0])], ["x", "z"])
    want = P.forward(cfg, w, other)
    assert C.row_error(torch.cat([a, c[:1]]).double(), ref[:12]).max() < TOL
    assert C.row_error(b.double(), want).max() < TOL and C.row_error(c[1:].double(), want[:1]).max() < TOL


@pytest.mark.parametrize("ahead", [False, True])
def test_greedy_generation_through_the_scheduler(case, ahead):
    """Chunked prompts, a pool too small for all of them, prompts that share a prefix: without carried state cached blocks are
    used, with it they must not be."""
    from unillm_b200.engine.cpu_runner import CpuModelRunner
    from unillm_b200.engine.llm_engine import LLMEngine
    from unillm_b200.sampling import SamplingParams

    name, _, _, m, _, _ = case
    prompts, want = C.expected_generation(name)
    eng = LLMEngine(CpuModelRunner(m, num_blocks=9, max_model_len=256), num_blocks=9, max_num_seqs=4, max_num_batched_tokens=24,
                    max_model_len=256, async_scheduling=ahead)
    assert eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)) == want
    if m.spec.has_state:
        assert eng.radix is None and eng.stats.cached_tokens == 0 and eng.slots.num_free() == 4
    elif not ahead:
        assert eng.stats.cached_tokens > 0


def test_preempted_sequences_start_over(case):
    from unillm_b200.sampling import SamplingParams

    _, cfg, w, m, _, _ = case
    prompts = [C.tokens(cfg, n, 60 + n) for n in (27, 30)]
    eng = _engine(m, blocks=5, max_num_seqs=2)          # both grow over a block's edge, and only one of them can
    got = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=7, ignore_eos=True))
    assert got == [C.greedy(cfg, w, p, 7) for p in prompts] and eng.stats.preemptions > 0
    assert eng.slots is None or eng.slots.num_free() == 2


def test_command_line_generates(tmp_path, capsys):
    from unillm_b200.cli import main

    cfg = C.CASES["mixed"]
    d = C.write_model(tmp_path / "m", cfg, C.make_weights(cfg))
    assert main(["generate", "-m", d, "-p", "ab", "--max-tokens", "3", "--temperature", "0", "--engine"]) == 0
    assert main(["models"]) == 0
    assert "bakasun" in capsys.readouterr().out


@pytest.mark.parametrize("layer,what", [(1, "cap"), (1, "linear"), (0, "row norm"), (1, "bias"), (0, "window+1"), (1, "window-1"), (2, "window+1"),
                                        (3, "window-1"), (0, "sink"), (1, "conv"), (1, "taps"), (1, "unit"), (1, "decay"), (2, "beta"), (1, "order"),
                                        (2, "lost"), (1, "head norm"), (1, "scales"), (1, "groups"), (1, "correction"), (1, "weights"),
                                        (3, "shared gate"), (0, "gelu"), (0, "eps"), (0, "out norm")])
def test_planted_mistakes_show(layer, what, monkeypatch):
    """The weights are sharp enough: a mistake planted in the plain statement moves the logits far beyond the tolerances."""
    cfg = C.CASES["mixed"]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 60, 1)
    ref = P.forward(cfg, w, toks)
    c2, w2, L = copy.deepcopy(cfg), dict(w), f"l{layer}."
    mx = c2["layers"][layer]["mixer"]
    left, right = mx.get("left", mx), mx.get("right")
    if what == "cap":
        del left["softcap"]
    elif what == "linear":
        del left["rot"]["scaling"]
    elif what == "row norm":                             # per head instead of over the whole projection
        f = P.attention
        def per_head(h, w, name, m, eps, bias, qk_norm):
            if not qk_norm:
                return f(h, w, name, m, eps, bias, qk_norm)
            q = (h @ w[name + ".q"].T).reshape(len(h), m["heads"], m["dim"])
            r = P.rms(q, eps).reshape(len(h), -1) / P.rms(q.reshape(len(h), -1), eps)
            keep = dict(w)
            real = P.rms
            monkeypatch.setattr(P, "rms", lambda x, e: real(x, e) * r if x.shape == r.shape else real(x, e))
            y = f(h, keep, name, m, eps, bias, qk_norm)
            monkeypatch.setattr(P, "rms", real)
            return y
        monkeypatch.setattr(P, "attention", per_head)
    elif what == "bias":
        w2[L + "mix.left.k.b"] = torch.zeros_like(w[L + "mix.left.k.b"])
        w2[L + "mix.left.v.b"] = torch.zeros_like(w[L + "mix.left.v.b"])
    elif what.startswith("window"):
        left["mask"]["size"] += int(what[6:])
    elif what == "sink":
        monkeypatch.setattr(P, "off_by_one_softmax", lambda s: torch.softmax(s, -1))
    elif what == "conv":                                 # one token off
        t = w[L + "mix.right.v.conv"]
        w2[L + "mix.right.v.conv"] = torch.cat([t[:, 1:], torch.zeros_like(t[:, :1])], 1)
    elif what == "taps":
        w2[L + "mix.right.k.conv"] = w[L + "mix.right.k.conv"].flip(1)
    elif what == "unit":
        monkeypatch.setattr(P, "unit", lambda x: x)
    elif what == "decay":
        w2[L + "mix.right.a"] = torch.zeros_like(w[L + "mix.right.a"])
    elif what == "beta":
        w2[L + "mix.right.b"] = torch.zeros_like(w[L + "mix.right.b"])
    elif what == "order":                                # the read-out comes before the write
        def early(q, k, v, g, beta):
            S, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype), torch.zeros_like(v)
            for t in range(len(q)):
                S = S * g[t, :, None, None]
                out[t] = (S * q[t, :, :, None]).sum(1)
                S = S + k[t, :, :, None] * (beta[t, :, None] * (v[t] - (S * k[t, :, :, None]).sum(1)))[:, None]
            return out
        monkeypatch.setattr(P, "delta_recurrence", early)
    elif what == "lost":                                 # the state starts again at token 30
        f = P.delta_recurrence
        monkeypatch.setattr(P, "delta_recurrence", lambda *t: torch.cat([f(*(x[a:b] for x in t)) for a, b in ((0, 30), (30, 60))])
                            if t[0].shape[1] == 3 else f(*t))
    elif what == "head norm":
        w2[L + "mix.right.norm"] = w[L + "mix.right.norm"].flip(0)
    elif what == "scales":
        mx["left_scale"], mx["right_scale"] = mx["right_scale"], mx["left_scale"]
    elif what == "groups":
        c2["layers"][layer]["mlp"]["router"]["groups"]["keep"] = 4
    elif what == "correction":
        w2[L + "mlp.correction"] = torch.zeros_like(w[L + "mlp.correction"])
    elif what == "weights":                              # the correction joins the weights
        f, n = P.mixture, 0
        def biased(h, w, name, mlp):
            s = torch.softmax(h @ w[name + ".router"].T, -1) + w[name + ".correction"]
            w = dict(w)
            w[name + ".router"], w[name + ".correction"] = torch.zeros_like(w[name + ".router"]), torch.zeros_like(w[name + ".correction"])
            out = []
            real = torch.softmax
            for t in range(len(h)):
                monkeypatch.setattr(torch, "softmax", lambda x, d, t=t: s[t:t + 1])
                out.append(f(h[t:t + 1], w, name, mlp))
            monkeypatch.setattr(torch, "softmax", real)
            return torch.cat(out)
        monkeypatch.setattr(P, "mixture", biased)
    elif what == "shared gate":
        w2[L + "mlp.shared.sg"] = torch.zeros_like(w[L + "mlp.shared.sg"])
    elif what == "gelu":
        monkeypatch.setattr(P, "gelu_tanh", P.silu)
    elif what == "out norm":
        w2[L + "norm1b"] = torch.zeros_like(w[L + "norm1b"])
    else:
        c2["norm"]["eps"] = 0.1
    err = C.row_error(P.forward(c2, w2, toks), ref)
    assert err.max() > 0.05, err.max()
