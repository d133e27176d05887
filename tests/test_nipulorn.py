"""Nipulorn on the host: reading a model directory, the whole-model path, and the serving engine with its block pool, state
slots and batching (fp32 CPU runner) against the plain statement of the design; the plain statement's own sensitivity."""
import copy

import pytest
import torch

import nipulorn_cases as C
import nipulorn_plain as P

TOL = 3e-5


@pytest.fixture(scope="module", params=sorted(C.CASES))
def case(request):
    cfg = C.CASES[request.param]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 70, 1)
    return cfg, w, C.load_model(cfg, w), toks, P.forward(cfg, w, toks)


def _engine(m, blocks=16, **kw):
    from unillm_b200.engine.factory import build_cpu_engine

    return build_cpu_engine(m, num_blocks=blocks, **kw)


def test_model_directory_loads_and_exports(tmp_path, case):
    from unillm_b200.models import NipulornModel
    from unillm_b200.weights import ModelLoader

    cfg, w, _, toks, ref = case
    m = ModelLoader().load_model(C.write_model(tmp_path / "m", cfg, w))
    assert isinstance(m, NipulornModel)
    with torch.no_grad():
        y = m.forward_with_cache(torch.tensor(toks))[0]
    assert C.row_error(y.double(), ref).max() < TOL
    out = m.export_hf().tensors
    assert set(out) == set(w)
    assert all(torch.equal(out[n].float(), t.float()) for n, t in w.items())


def test_layers_one_by_one(case):
    cfg, w, m, toks, _ = case
    _, after = P.forward(cfg, w, toks[:20], keep_layers=True)
    from unillm_b200.models import mixers as MX

    with torch.no_grad():
        x = m.p["embed"][torch.tensor(toks[:20])][None] * m.spec.embed_scale
        for i in range(m.spec.num_layers):
            st = {}
            x = m.block(i, x, lambda h: m.mixer(i, h, 0, None, {}, st),
                        lambda h, n: MX.input_conv(h, m.p[f"layers.{i}.{n}"], st, n))
            assert (x[0].double() - after[i]).abs().max() < 1e-4 * after[i].abs().max(), i


def test_whole_model_path_continues_from_its_cache(case):
    _, _, m, toks, ref = case
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

    cfg, _, m, _, _ = case
    row = sum(x["mixer"]["kv_rank"] + x["mixer"]["rot_dim"] for x in cfg["layers"] if x["type"] == "latent_attention")
    assert KvShape.from_spec(m.spec).bytes_per_token() == 2 * row
    state = 0
    for x in cfg["layers"]:
        state += (cfg["canon"]["taps"] - 1) * cfg["width"] * (1 if x["mlp"] is None else 2)
        if x["type"] == "wkv":
            state += cfg["width"] + x["mixer"]["heads"] * x["mixer"]["dim"] ** 2
    assert m.spec.state_elements == state and m.spec.has_state == (state > 0)
    assert RunnerWeights(m.spec, m.p, "cpu").state_bytes_per_seq() >= 8 * state


def test_bad_configurations_are_refused():
    from unillm_b200.types import ConfigurationError

    for edit in (lambda c: c["layers"][0].update(type="attention"), lambda c: c["layers"][1]["mlp"].update(kind="moe"),
                 lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7)):
        cfg = copy.deepcopy(C.CASES["mixed"])
        edit(cfg)
        with pytest.raises(ConfigurationError):
            C.load_model(cfg, {})


@pytest.mark.parametrize("missing", ["l0.mix.w1", "l0.mix.mu.g", "l1.mix.dkv.norm", "l1.norm2b", "l2.canon1", "l1.mlp.act"])
def test_missing_tensors_are_named(missing):
    from unillm_b200.types import LoadingError

    w = C.make_weights(C.CASES["mixed"])
    del w[missing]
    with pytest.raises(LoadingError):
        C.load_model(C.CASES["mixed"], w)


@pytest.mark.parametrize("sizes", [[70], [1], [2], [3, 1, 2], [16], [17, 2, 31], [64, 1]])
def test_portions_through_the_engine(case, sizes):
    cfg, _, m, toks, ref = case
    got = C.score(_engine(m), toks, C.portions(len(toks), sizes))
    assert C.row_error(got, ref).max() < TOL


def test_unequal_batch_with_blocks_and_slots_used_again(case):
    """Sequences in one batch, in portions of different sizes; finished ones make room for others in a pool and in state
    slots that hold no more than the live ones need."""
    cfg, w, m, _, _ = case
    seqs = {k: C.tokens(cfg, n, 10 + k) for k, n in C.BATCH.items()}
    eng = _engine(m, blocks=11, max_num_seqs=3)
    got = C.score_batch(eng, seqs, C.BATCH_SIZES)
    assert eng.pool.num_free() == 11 and (eng.slots is None or eng.slots.num_free() == 3)
    for k in seqs:
        assert C.row_error(got[k], P.forward(cfg, w, seqs[k])).max() < TOL, k


def test_a_sequence_may_pause(case):
    cfg, w, m, toks, ref = case
    eng, other = _engine(m), C.tokens(cfg, 30, 5)
    a = eng.score_step([("x", toks[:11], range(11))])
    b = eng.score_step([("y", other[:30], range(30))], ["y"])
    c = eng.score_step([("x", toks[11:12], [0]), ("z", other[:1], [0])], ["x", "z"])
    want = P.forward(cfg, w, other)
    assert C.row_error(torch.cat([a, c[:1]]).double(), ref[:12]).max() < TOL
    assert C.row_error(b.double(), want).max() < TOL and C.row_error(c[1:].double(), want[:1]).max() < TOL


def greedy(cfg, w, prompt, n):
    out = []
    for _ in range(n):
        out.append(int(P.forward(cfg, w, prompt + out)[-1].argmax()))
    return out


@pytest.mark.parametrize("ahead", [False, True])
def test_greedy_generation_through_the_scheduler(case, ahead):
    """Chunked prompts, a pool too small for all of them, prompts that share a prefix: without carried state cached blocks are
    used, with it they must not be."""
    from unillm_b200.sampling import SamplingParams

    cfg, w, m, _, _ = case
    prompts = [C.tokens(cfg, n, 30 + n) for n in (19, 3, 34, 1, 50)]
    prompts.append(prompts[4][:40])
    from unillm_b200.engine.cpu_runner import CpuModelRunner
    from unillm_b200.engine.llm_engine import LLMEngine

    eng = LLMEngine(CpuModelRunner(m, num_blocks=9, max_model_len=256), num_blocks=9, max_num_seqs=4, max_num_batched_tokens=24,
                    max_model_len=256, async_scheduling=ahead)
    got = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    assert got == [greedy(cfg, w, p, 6) for p in prompts]
    if m.spec.has_state:
        assert eng.radix is None and eng.stats.cached_tokens == 0 and eng.slots.num_free() == 4
    elif not ahead:
        assert eng.stats.cached_tokens > 0


def test_preempted_sequences_start_over(case):
    from unillm_b200.sampling import SamplingParams

    cfg, w, m, _, _ = case
    prompts = [C.tokens(cfg, n, 60 + n) for n in (27, 30)]
    eng = _engine(m, blocks=5, max_num_seqs=2)          # both grow over a block's edge, and only one of them can
    got = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=7, ignore_eos=True))
    assert got == [greedy(cfg, w, p, 7) for p in prompts] and eng.stats.preemptions > 0
    assert eng.slots is None or eng.slots.num_free() == 2


def test_command_line_generates(tmp_path, capsys, case):
    from unillm_b200.cli import main

    cfg, w, _, _, _ = case
    if cfg["vocab"] < 128:
        pytest.skip("the fallback tokenizer needs more ids")
    d = C.write_model(tmp_path / "m", cfg, w)
    assert main(["generate", "-m", d, "-p", "ab", "--max-tokens", "3", "--temperature", "0", "--engine"]) == 0
    assert main(["models"]) == 0
    assert "nipulorn" in capsys.readouterr().out


def test_state_slots():
    from unillm_b200.kv.state_slots import StateSlots
    from unillm_b200.types import MemoryError_

    s = StateSlots(2)
    a, b = s.allocate(), s.allocate()
    with pytest.raises(MemoryError_):
        s.allocate()
    r0, w0 = s.advance(a, fresh=True)
    r1, w1 = s.advance(a, fresh=False)
    assert r0 == s.FRESH and r1 == w0 and w1 != w0 and {w0, w1} == {2 * a, 2 * a + 1}
    assert s.advance(b, fresh=True)[1] not in (w0, w1)
    s.free(a)
    with pytest.raises(MemoryError_):
        s.free(a)
    assert s.num_free() == 1 and s.allocate() == a


def test_packed_metadata_carries_state_rows():
    from unillm_b200.engine.runner import StepBatch, StepPacker

    b = StepBatch([1, 2, 3, 4, 5, 6], [4, 9, 2, 0, 1, 2], [4, 25, 34, 48, 49, 50], 3, [5, 10, 3, 3], [[0], [1], [2], [3]], [3], [2],
                  state_in=[0, 3, 5, -1], state_out=[1, 2, 4, 7])
    for bucketed in (False, True):
        pk = StepPacker(torch.zeros(4096, dtype=torch.int32), 16)
        lay = pk.pack(b, bucketed)
        get = lambda n: pk.np[lay[n][0]:lay[n][0] + lay[n][1]].tolist()
        D, n = lay["_Dp"], lay["_Dp"] + lay["_P"]
        si, so = get("state_in"), get("state_out")
        assert len(si) == len(so) == n and si[:3] == [0, 3, 5] and so[:3] == [1, 2, 4] and si[D] == -1 and so[D] == 7
        assert all(v == -1 for v in si[3:D] + so[3:D] + si[D + 1:] + so[D + 1:])
    dup = [v for v in b.state_out if v >= 0]
    assert len(set(dup)) == len(dup) and not set(dup) & set(b.state_in)


@pytest.mark.parametrize("layer,what", [(0, "decay"), (0, "bonus"), (2, "shift"), (0, "conv"), (1, "conv"), (1, "sink"), (3, "sink"),
                                        (1, "yarn"), (1, "gain"), (1, "scale"), (1, "far"), (3, "far"), (1, "act"), (2, "lost"), (0, "eps")])
def test_planted_mistakes_show(layer, what, monkeypatch):
    """The weights are sharp enough: a mistake planted in the plain statement moves the logits far beyond the tolerances."""
    cfg = C.CASES["mixed"]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 60, 1)
    ref = P.forward(cfg, w, toks)
    c2, w2, L = copy.deepcopy(cfg), dict(w), f"l{layer}."
    if what == "decay":
        w2[L + "mix.w2"] = torch.zeros_like(w[L + "mix.w2"])
    elif what == "bonus":
        w2[L + "mix.u"] = torch.zeros_like(w[L + "mix.u"])
    elif what == "shift":
        w2[L + "mix.mu.k"] = torch.zeros_like(w[L + "mix.mu.k"])
    elif what == "conv":                                 # one token off
        t = w[L + "canon1"].clone()
        w2[L + "canon1"] = torch.cat([t[:, 1:], torch.zeros_like(t[:, :1])], 1)
    elif what == "sink":
        w2[L + "mix.sink"] = torch.full_like(w[L + "mix.sink"], -40.0)
    elif what == "yarn":
        del c2["layers"][layer]["mixer"]["rot"]["scaling"]
    elif what == "gain":
        f = P.yarn_frequencies
        monkeypatch.setattr(P, "yarn_frequencies", lambda rot: (f(rot)[0], 1.0))
    elif what == "scale":
        c2["layers"][layer]["mixer"]["scale"] *= 1.3
    elif what == "far":                                  # the first 16 cached rows are another token's
        f = P.latent_attention
        monkeypatch.setattr(P, "latent_attention", lambda qn, qr, c, *a: f(qn, qr, torch.cat([c[15:16].expand(16, -1), c[16:]]), *a)
                            if c.shape[1] == cfg["layers"][layer]["mixer"]["kv_rank"] else f(qn, qr, c, *a))
    elif what == "act":
        w2[L + "mlp.act"] = w[L + "mlp.act"].flip(0)
    elif what == "lost":                                 # the state starts again at token 30
        f = P.wkv_recurrence
        monkeypatch.setattr(P, "wkv_recurrence", lambda r, k, v, d, u: torch.cat(
            [f(*(t[a:b] for t in (r, k, v, d)), u) for a, b in ((0, 30), (30, 60))]) if k.shape[1] == 2 else f(r, k, v, d, u))
    else:
        c2["norm"]["eps"] = 0.1
    err = C.row_error(P.forward(c2, w2, toks), ref)
    assert err.max() > 0.05, err.max()
