"""Gekapel on the host: reading a model directory, the whole-model path, and the serving engine with its block pool and
batching (fp32 CPU runner) against the plain statement of the design; the plain statement's own sensitivity."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import gekapel_cases as C
import gekapel_plain as P

TOL = 2e-5


@pytest.fixture(scope="module", params=sorted(C.CASES))
def case(request):
    cfg = C.CASES[request.param]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 90, 1)
    return cfg, w, C.load_model(cfg, w), toks, P.forward(cfg, w, toks)


def _engine(m, blocks=16, **kw):
    from unillm_b200.engine.factory import build_cpu_engine

    return build_cpu_engine(m, num_blocks=blocks, **kw)


def test_model_directory_loads_and_exports(tmp_path, case):
    from unillm_b200.models import GekapelModel
    from unillm_b200.weights import ModelLoader

    cfg, w, _, toks, ref = case
    m = ModelLoader().load_model(C.write_model(tmp_path / "m", cfg, w))
    assert isinstance(m, GekapelModel)
    with torch.no_grad():
        y = m.forward_with_cache(torch.tensor(toks))[0]
    assert C.row_error(y.double(), ref).max() < TOL
    out = m.export_hf().tensors
    assert set(out) == set(w)
    assert all(torch.equal(out[n].float(), t.float()) for n, t in w.items())


def test_cache_cost_counts_only_layers_with_keys(case):
    from unillm_b200.scheduler.policies import KvShape

    cfg, _, m, _, _ = case
    per_token = sum(x["mixer"]["kv_heads"] * (x["mixer"]["dim"] + x["mixer"]["vdim"]) for x in cfg["layers"]
                    if x["mixer"].get("kv_from") is None)
    assert KvShape.from_spec(m.spec).bytes_per_token() == 2 * per_token
    assert m.memory_requirements().kv_cache_memory == 2 * per_token * m.spec.max_position_embeddings


def test_bad_configurations_are_refused():
    from unillm_b200.types import ConfigurationError

    for edit in (lambda c: c["layers"][3]["mixer"].update(kv_from=4), lambda c: c["layers"][4]["mixer"].update(kv_from=3),
                 lambda c: c["layers"][3]["mixer"].update(vdim=8), lambda c: c["layers"][0]["mixer"].update(heads=5),
                 lambda c: c["layers"][0].update(type="other")):
        cfg = copy.deepcopy(C.CASES["mixed"])
        edit(cfg)
        with pytest.raises(ConfigurationError):
            C.load_model(cfg, {})


@pytest.mark.parametrize("sizes", [[90], [1], [2], [3, 1, 2], [16], [17, 2, 31], [64, 1]])
def test_portions_through_the_engine(case, sizes):
    cfg, _, m, toks, ref = case
    got = C.score(_engine(m), toks, C.portions(len(toks), sizes))
    assert C.row_error(got, ref).max() < TOL


def test_unequal_batch_with_blocks_used_again(case):
    """Four sequences in one batch, in portions of different sizes; finished ones make room for others in a pool that
    holds no more than the live ones need."""
    cfg, w, m, _, _ = case
    seqs = {k: C.tokens(cfg, n, 10 + k) for k, n in enumerate((61, 7, 33, 1, 48, 16, 2))}
    want = {k: P.forward(cfg, w, t) for k, t in seqs.items()}
    eng = _engine(m, blocks=4 + 1 + 3 + 3)
    sizes = {0: [5, 1, 2], 1: [1], 2: [17, 1], 3: [1], 4: [2, 31], 5: [16], 6: [2]}
    cuts = {k: C.portions(len(t), sizes[k]) for k, t in seqs.items()}
    queue, live, got = list(seqs), [], {k: [] for k in seqs}
    while queue or live:
        while queue and len(live) < 3:
            live.append(queue.pop(0))
        step = [(k, cuts[k].pop(0)) for k in live]
        done = [k for k, (_, b) in step if b == len(seqs[k])]
        out = eng.score_step([(k, seqs[k][a:b], range(b - a)) for k, (a, b) in step], done).double()
        for k, (a, b) in step:
            got[k].append(out[:b - a])
            out = out[b - a:]
        live = [k for k in live if k not in done]
    assert eng.pool.num_free() == 11
    for k in seqs:
        assert C.row_error(torch.cat(got[k]), want[k]).max() < TOL, k


def test_score_step_refuses_bad_steps(case):
    from unillm_b200.types import InvalidInput, MemoryError_

    eng = _engine(case[2], blocks=2, max_num_seqs=2, max_num_batched_tokens=64)
    for entries, end in (([("a", [], [])], []), ([("a", [1], [1])], []), ([("a", [1], []), ("a", [2], [])], []),
                         ([(k, [1], []) for k in "abc"], []), ([("a", [1] * 65, [])], []), ([], ["a"])):
        with pytest.raises(InvalidInput):
            eng.score_step(entries, end)
    eng.score_step([("a", [1] * 20, [])], [])
    with pytest.raises(MemoryError_):
        eng.score_step([("b", [1], [])], [])


def greedy(cfg, w, prompt, n):
    out = []
    for _ in range(n):
        out.append(int(P.forward(cfg, w, prompt + out)[-1].argmax()))
    return out


def test_greedy_generation_through_the_scheduler(case):
    from unillm_b200.sampling import SamplingParams

    cfg, w, m, _, _ = case
    prompts = [C.tokens(cfg, n, 30 + n) for n in (19, 3, 34, 1, 50)]
    prompts.append(prompts[4][:40])                     # shares whole cached blocks with an earlier prompt
    eng = _engine(m, blocks=14, max_num_seqs=4, max_num_batched_tokens=24)      # chunked prompts, tight pool
    got = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    assert got == [greedy(cfg, w, p, 6) for p in prompts]
    assert eng.stats.cached_tokens > 0


def test_command_line_generates(tmp_path, capsys, case):
    from unillm_b200.cli import main

    cfg, w, m, _, _ = case
    if cfg["vocab"] < 128:
        pytest.skip("the fallback tokenizer needs more ids")
    d = C.write_model(tmp_path / "m", cfg, w)
    assert main(["generate", "-m", d, "-p", "ab", "--max-tokens", "3", "--temperature", "0", "--engine"]) == 0
    assert main(["models"]) == 0
    assert "gekapel" in capsys.readouterr().out


def test_kernel_layout_pads_and_shards(case):
    """The weights in kernel layout (padded rows and heads) still give the model: checked by undoing the layout of one
    rank, and by summing the partial products of two."""
    from unillm_b200.engine.runner import RunnerWeights
    from unillm_b200.types import InvalidInput

    cfg, w, m, _, _ = case
    one = RunnerWeights(m.spec, m.p, "cpu", dtype=torch.float32)
    H = cfg["width"]
    for i, ls in enumerate(m.spec.layers):
        L, kh = f"layers.{i}.", one.heads[i]
        q = one.t[L + "wqkv"][:kh.hq * kh.dk].reshape(kh.hq, kh.dk, -1)
        assert torch.equal(q[:, :ls.head_dim, :H].reshape(-1, H), m.p[L + "wqkv"][:ls.q_size])
        assert q[:, ls.head_dim:].abs().sum() == 0 and one.t[L + "wqkv"][:, H:].abs().sum() == 0
        wo = one.t[L + "wo"].reshape(-1, kh.hq, kh.dv)
        assert torch.equal(wo[:H, :, :ls.v_head_dim].reshape(H, -1), m.p[L + "wo"]) and wo[H:].abs().sum() == 0
        assert kh.dk % 8 == 0 and kh.dv % 8 == 0 and kh.own_kv == (ls.kv_from is None)
    try:
        two = [RunnerWeights(m.spec, m.p, "cpu", r, 2, dtype=torch.float32) for r in range(2)]
    except InvalidInput:
        return                                          # sizes that two ranks do not divide
    x = torch.randn(3, one.width)
    for i in range(m.spec.num_layers):
        for n in ("shared_gate_up", "experts_gate_up"):
            L = f"layers.{i}."
            if L + n not in one.t:
                continue
            dn = n.split("_")[0] + "_down"
            f = lambda r: torch.relu(x @ r.t[L + n].transpose(-1, -2)) ** 2 @ r.t[L + dn].transpose(-1, -2)
            assert torch.allclose(f(one), f(two[0]) + f(two[1]), atol=1e-4)


@pytest.mark.parametrize("layer,what", [(0, "wider"), (0, "narrower"), (0, "sink"), (1, "wider"), (2, "narrower"), (3, "sink"),
                                        (3, "kv"), (0, "route"), (2, "freq")])
def test_planted_mistakes_show(layer, what):
    """The weights are sharp enough: a mistake planted in the plain statement moves the logits far beyond the tolerances."""
    cfg = C.CASES["mixed"]
    w = C.make_weights(cfg)
    toks = C.tokens(cfg, 75, 1)
    c2, w2 = copy.deepcopy(cfg), dict(w)
    mx = c2["layers"][layer]["mixer"]
    if what in ("wider", "narrower"):
        mx["mask"]["size"] += 1 if what == "wider" else -1
    elif what == "sink":
        w2[f"l{layer}.mix.sink"] = torch.full_like(w[f"l{layer}.mix.sink"], -40.0)
    elif what == "kv":
        del mx["kv_from"]
        for n in ("k", "v", "k.norm"):
            w2[f"l{layer}.mix.{n}"] = w[f"l0.mix.{n}"]   # its own keys instead of the cached ones of layer 0
    elif what == "route":
        w2["l0.mlp.router.b"] = torch.zeros_like(w["l0.mlp.router.b"])
    else:
        del mx["rot"]["scaling"]
    err = C.row_error(P.forward(c2, w2, toks), P.forward(cfg, w, toks))
    assert err.max() > 0.2


def test_trace_runner_arguments():
    r = subprocess.run([sys.executable, os.path.join(os.path.dirname(__file__), "..", "bin", "trace_run"), "--help"],
                       capture_output=True, text=True, timeout=120)
    assert r.returncode == 0 and "--max-tokens" in r.stdout


def test_replay_writes_wanted_logits_in_order(tmp_path, case):
    from unillm_b200.engine.replay import replay

    cfg, _, m, toks, ref = case
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:20], "want": [3, 19]}, {"id": "y", "tokens": toks[:1], "want": [0]}],
              "end": ["y"]},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[20:21], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": toks[:9], "want": [8]}, {"id": "x", "tokens": toks[21:22], "want": [0]}],
              "end": ["x", "y"]}]
    said = []
    replay(_engine(m), [json.dumps(d) for d in lines], str(tmp_path), write=lambda s, flush: said.append(s))
    assert said == ["done 0", "done 1", "done 2"]
    assert not os.path.exists(tmp_path / "1.f32")
    for step, rows in ((0, [3, 19, 0]), (2, [8, 21])):
        got = torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32).reshape(len(rows), -1)
        assert C.row_error(got.double(), ref[rows]).max() < TOL
