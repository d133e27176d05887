"""Tasadra on the host: reading a model directory, the whole-model path, and the serving engine with its block pool, state
slots and batching (fp32 CPU runner) against the plain statement of the design; the plain statement's own sensitivity."""
import copy

import pytest
import torch

import tasadra_cases as C
import tasadra_plain as P

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
    from unillm_b200.models import TasadraModel
    from unillm_b200.weights import ModelLoader

    _, cfg, w, _, toks, ref = case
    m = ModelLoader().load_model(C.write_model(tmp_path / "m", cfg, w))
    assert isinstance(m, TasadraModel)
    with torch.no_grad():
        y = m.forward_with_cache(torch.tensor(toks))[0]
    assert C.row_error(y.double(), ref).max() < TOL
    out = m.export_hf().tensors
    assert set(out) == set(w)
    assert all(torch.equal(out[n].float(), t.float()) for n, t in w.items())


def test_layers_one_by_one(case):
    _, cfg, w, m, toks, _ = case
    from unillm_b200.models import mixers as MX

    _, after = P.forward(cfg, w, toks[:30], keep_layers=True)
    with torch.no_grad():
        x = m.p["embed"][torch.tensor(toks[:30])][None]
        streams, shared = [x], {}
        for i in range(m.spec.num_layers):
            st = {}
            x = m.block(i, x, lambda h: m.mixer(i, h, 0, None, shared, st),
                        lambda h, n: MX.before_sublayer(h, m.p[f"layers.{i}.{n}"], st, n))
            x = m.after_layer(i, x, streams)
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
        a = x["mixer"]
        state += cfg["width"]                            # every mixer's token shift
        if x["type"] == "channel_delta":
            state += a["heads"] * a["dim"] * a["vdim"] + (a["conv"] - 1) * (2 * a["kv_heads"] * a["dim"] + a["heads"] * a["vdim"])
        elif a.get("kv_from") is None:
            row += a["kv_heads"] * (a["dim"] * (2 if x["type"] == "attention_2" else 1) + a["vdim"])
    assert KvShape.from_spec(m.spec).bytes_per_token() == 2 * row
    assert m.spec.state_elements == state and m.spec.has_state
    rw = RunnerWeights(m.spec, m.p, "cpu")
    assert rw.state_bytes_per_seq() >= 8 * state and rw.kv_bytes_per_token() >= 2 * row


def test_random_kernel_weights_have_the_loaded_ones_shapes(case):
    from unillm_b200.engine.runner import RunnerWeights

    _, cfg, _, m, _, _ = case
    if cfg["width"] % 8:
        pytest.skip("random weights are for widths that need no padding")
    a, b = RunnerWeights(m.spec, m.p, "cpu"), RunnerWeights.random(m.spec, "cpu")
    assert all(n in b.t and (b.t[n].shape, b.t[n].dtype) == (t.shape, t.dtype) for n, t in a.t.items())
    assert set(a.slopes) <= set(b.slopes) and set(a.lams) == set(b.lams)


def test_bad_configurations_are_refused():
    from unillm_b200.types import ConfigurationError

    edits = [lambda c: c["layers"][0].update(type="latent"), lambda c: c["layers"][0]["mlp"].update(kind="moe"),
             lambda c: c["layers"][1]["mixer"].update(kv_heads=4), lambda c: c["layers"][2]["mixer"].update(kv_heads=3),
             lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
             lambda c: c["layers"][1]["mixer"].update(vdim=33), lambda c: c["layers"][3]["mixer"].update(kv_from=1),
             lambda c: c["layers"][3]["mixer"].update(kv_from=3), lambda c: c["layers"][3]["mixer"].update(vdim=48)]
    for edit in edits:
        cfg = copy.deepcopy(C.CASES["mixed"])
        edit(cfg)
        with pytest.raises(ConfigurationError):
            C.load_model(cfg, {})


@pytest.mark.parametrize("missing", ["l1.mix.q.norm", "l0.mix.k", "l0.mix.lk2", "l1.mix.g", "l2.mix.v.conv", "l2.mix.a1", "l2.mix.g2", "l0.norm1.alpha",
                                     "l0.shift", "l3.dwa", "l2.mix.dt_bias", "final.norm.alpha", "l3.mix.o"])
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
    assert eng.pool.num_free() == 11 and eng.slots.num_free() == 3
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
    """Chunked prompts, a pool too small for all of them, prompts that share a prefix (whose cached blocks must not be used: the
    state at their end is not cached)."""
    from unillm_b200.engine.cpu_runner import CpuModelRunner
    from unillm_b200.engine.llm_engine import LLMEngine
    from unillm_b200.sampling import SamplingParams

    name, _, _, m, _, _ = case
    prompts, want = C.expected_generation(name)
    eng = LLMEngine(CpuModelRunner(m, num_blocks=9, max_model_len=256), num_blocks=9, max_num_seqs=4, max_num_batched_tokens=24,
                    max_model_len=256, async_scheduling=ahead)
    assert eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)) == want
    assert eng.radix is None and eng.stats.cached_tokens == 0 and eng.slots.num_free() == 4


def test_preempted_sequences_start_over(case):
    from unillm_b200.sampling import SamplingParams

    _, cfg, w, m, _, _ = case
    prompts = [C.tokens(cfg, n, 60 + n) for n in (27, 30)]
    eng = _engine(m, blocks=5, max_num_seqs=2)          # both grow over a block's edge, and only one of them can
    got = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=7, ignore_eos=True))
    assert got == [C.greedy(cfg, w, p, 7) for p in prompts] and eng.stats.preemptions > 0
    assert eng.slots.num_free() == 2


def test_command_line_generates(tmp_path, capsys):
    from unillm_b200.cli import main

    cfg = C.CASES["mixed"]
    d = C.write_model(tmp_path / "m", cfg, C.make_weights(cfg))
    assert main(["generate", "-m", d, "-p", "ab", "--max-tokens", "3", "--temperature", "0", "--engine"]) == 0
    assert main(["models"]) == 0
    assert "tasadra" in capsys.readouterr().out


@pytest.mark.parametrize("layer,what", [(1, "cap"), (1, "yarn"), (1, "gain"), (1, "q norm"), (1, "value turn"), (1, "turn back"), (1, "head gate"),
                                        (0, "chunk+1"), (0, "chunk-1"), (3, "chunk+1"), (3, "chunk-1"), (0, "one map"), (0, "lambda"), (0, "difference norm"),
                                        (3, "element gate"), (3, "own keys"), (2, "conv"), (2, "taps"), (2, "unit"), (2, "decay"), (2, "head decay"),
                                        (2, "beta"), (2, "order"), (2, "lost"), (2, "head norm"), (2, "low gate"), (0, "shift"), (4, "shift"), (2, "slope"),
                                        (1, "norm bias"), (3, "average"), (0, "average"), (0, "mult"), (0, "ff bias"), (0, "relu"), (0, "eps")])
def test_planted_mistakes_show(layer, what, monkeypatch):
    """The weights are sharp enough: a mistake planted in the plain statement moves the logits far beyond the tolerances."""
    cfg = C.CASES["mixed"]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 60, 1)
    ref = P.forward(cfg, w, toks)
    c2, w2, L = copy.deepcopy(cfg), dict(w), f"l{layer}."
    mx = c2["layers"][layer]["mixer"]
    zero = lambda n: w2.update({n: torch.zeros_like(w[n])})
    if what == "cap":
        del mx["softcap"]
    elif what == "yarn":
        del mx["rot"]["scaling"]
    elif what == "gain":
        f = P.yarn_frequencies
        monkeypatch.setattr(P, "yarn_frequencies", lambda rot: (f(rot)[0], 1.0))
    elif what == "q norm":
        w2[L + "mix.q.norm"] = torch.ones_like(w[L + "mix.q.norm"])
    elif what == "value turn":
        monkeypatch.setattr(P, "value_frequencies", lambda base, n: [0.0] * (n // 2))
    elif what == "turn back":                            # values keep their rotation
        f = P.turn
        monkeypatch.setattr(P, "turn", lambda v, pos, fr, gain=1.0: v if pos[-1] < 0 else f(v, pos, fr, gain))
    elif what in ("head gate", "element gate"):
        zero(L + "mix.g")
    elif what.startswith("chunk"):
        mx["mask"]["size"] += int(what[5:])
    elif what == "one map":
        monkeypatch.setattr(P, "difference", lambda a1, a2, lam, diff, eps: P.rms(a1, eps) * (1 - diff))
    elif what == "lambda":
        for c in ("lq1", "lq2"):
            zero(L + "mix." + c)
    elif what == "difference norm":
        monkeypatch.setattr(P, "difference", lambda a1, a2, lam, diff, eps: (a1 - lam * a2) * (1 - diff))
    elif what == "own keys":                             # made from the reading layer's own input
        del mx["kv_from"]
        for c in "kv":
            w2[L + "mix." + c] = w[f"l0.mix.{c}"]
    elif what == "conv":                                 # one token off
        t = w[L + "mix.v.conv"]
        w2[L + "mix.v.conv"] = torch.cat([t[:, 1:], torch.zeros_like(t[:, :1])], 1)
    elif what == "taps":
        w2[L + "mix.k.conv"] = w[L + "mix.k.conv"].flip(1)
    elif what == "unit":
        monkeypatch.setattr(P, "unit", lambda x: x)
    elif what == "decay":
        zero(L + "mix.a2")
    elif what == "head decay":                           # one decay for all channels of a head
        f = P.channel_decay
        monkeypatch.setattr(P, "channel_decay", lambda *a: f(*a).mean(-1, keepdim=True).expand(-1, -1, a[4]))
    elif what == "beta":
        zero(L + "mix.b")
    elif what == "order":                                # the read-out comes before the write
        def early(q, k, v, g, beta):
            S, out = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype), torch.zeros_like(v)
            for t in range(len(q)):
                S = S * g[t, :, :, None]
                out[t] = (S * q[t, :, :, None]).sum(1)
                S = S + k[t, :, :, None] * (beta[t, :, None] * (v[t] - (S * k[t, :, :, None]).sum(1)))[:, None]
            return out
        monkeypatch.setattr(P, "delta_recurrence", early)
    elif what == "lost":                                 # the state starts again at token 30
        f = P.delta_recurrence
        monkeypatch.setattr(P, "delta_recurrence", lambda *t: torch.cat([f(*(x[a:b] for x in t)) for a, b in ((0, 30), (30, 60))]))
    elif what == "head norm":
        w2[L + "mix.norm"] = w[L + "mix.norm"].flip(0)
    elif what == "low gate":
        zero(L + "mix.g2")
    elif what == "shift":
        zero(L + "shift")
    elif what == "slope":
        w2[L + "norm1.alpha"] = w[L + "norm1.alpha"] * 1.5
    elif what == "norm bias":
        zero(L + "norm1.b")
    elif what == "average":                              # without the embedding
        w2[L + "dwa"] = w[L + "dwa"].clone()
        w2[L + "dwa"][0] = 0
    elif what == "mult":
        c2["residual_mult"] = 1.0
    elif what == "ff bias":
        zero(L + "mlp.down.b")
    elif what == "relu":
        monkeypatch.setattr(P, "feed_forward", lambda h, w, n: torch.clamp(h @ w[n + ".up"].T + w[n + ".up.b"], min=0.0) @ w[n + ".down"].T + w[n + ".down.b"])
    else:
        c2["norm"]["eps"] = 0.1
    err = C.row_error(P.forward(c2, w2, toks), ref)
    assert err.max() > 0.05, err.max()
