"""Gedilorn through the engine's own step function, cache manager, scheduler and entry points, against the plain
model: whole prompts, decoding token by token, portions down to two tokens, unequal requests in one batch, long
portions beside decoding requests, pages and slots used again, long decoding, greedy generation."""

import json
import os
import subprocess
import sys

import pytest
import torch

import gedilorn_tiny as gt
import plain_gedilorn as pg
import traces
from engine_harness import run_trace

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 4e-5                 # float32: of a request's largest logit
ROUNDINGS = 2.5            # bfloat16: of the largest error that the rounding of the stored numbers alone causes


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in gt.CONFIGS.items():
        w = gt.make_weights(cfg, seed=7 + ord(name))
        folder = gt.write_folder(str(tmp_path_factory.mktemp("gd_" + name)), cfg, w)
        out[name] = (folder, cfg, w)
    return out


def runner_for(folder, dtype, **kw):
    from mini_infer_b200.engine.loading import load_model
    from mini_infer_b200.engine.step import ModelRunner
    model, rt, _ = load_model(folder, dtype, "cuda:0")
    args = dict(page_size=8, num_pages=40, max_requests=4, max_tokens_per_step=256, max_context=352)
    args.update(kw)
    return ModelRunner(model, rt, **args)


def rms(x):
    return x.pow(2).mean(dim=-1).sqrt()


def check(got, cfg, w, reqs, dtype, plain_dtype=torch.float64):
    """Float32: every logit.  Bfloat16: every position's root mean square error, beside the largest one of the plain
    model that rounds what the engine stores in 16 bits."""
    exact = {rid: pg.forward(cfg, w, toks, plain_dtype).double() for rid, toks in reqs.items()}
    if dtype == "bfloat16":
        limit = max(float(rms(pg.forward(cfg, w, toks, plain_dtype, pg.as_bfloat16).double() - exact[rid]).max() /
                          rms(exact[rid]).mean()) for rid, toks in reqs.items())
        assert limit < 0.12, "the model is too sensitive for its rounding to tell a fault"
    for (rid, pos), row in sorted(got.items()):
        diff, ref = row.double() - exact[rid][pos], exact[rid]
        if dtype == "float32":
            err, tol = float(diff.abs().max() / ref.abs().max()), TOL
        else:
            err, tol = float(rms(diff) / rms(ref).mean()), ROUNDINGS * limit
        assert err <= tol, f"request {rid} position {pos}: {err:.2e}, at most {tol:.2e} (first failing place)"


def run_and_check(runner, steps, cfg, w, reqs, dtype):
    got = run_trace(runner, steps)
    check(got, cfg, w, reqs, dtype)
    return got


@pytest.mark.parametrize("name", sorted(gt.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_cutting_against_the_plain_model(models, name, dtype):
    folder, cfg, w = models[name]
    runner = runner_for(folder, dtype, max_requests=6, num_pages=60)
    reqs = gt.random_requests(cfg, [70, 1, 23, 2, 150, 9], seed=ord(name))
    results = []
    for steps in (traces.whole(reqs), traces.tail_decoded(reqs, tail=36), traces.portions(reqs),
                  traces.portions(reqs, (2,)), traces.mixed(reqs, max_live=3, seed=2, decode_tail=14),
                  traces.decoded_together({r: t for r, t in reqs.items() if len(t) > 1},
                                          {"r0": 30, "r2": 12, "r3": 1, "r4": 40, "r5": 3})):
        results.append(run_and_check(runner, steps, cfg, w, reqs, dtype))
        assert runner.cache.used_pages() == [0] * len(runner.cache.pools)
    if dtype == "float32":
        # the 32-bit path gives the same bits however the work was cut and batched
        for other in results[1:]:
            for key, row in other.items():
                assert torch.equal(row, results[0][key]), key
    if dtype == "bfloat16" and name in "AB":
        # which kernels the sizes take: none of the tensor-core forms, or all of them
        forms = {(m._tensor_cores, m._small_max > 0, m._unfold) for m in (l.parts["mixer"] for l in runner.model.layers)}
        assert forms == {(name == "B",) * 3}


def test_layer_by_layer(models):
    """The sum of the streams after every run of a layer."""
    from mini_infer_b200.engine.step import StepEntry
    for name in sorted(gt.CONFIGS):
        folder, cfg, w = models[name]
        runner = runner_for(folder, "float32")
        toks = gt.random_requests(cfg, [29], 3)["r0"]
        want = []
        pg.forward(cfg, w, toks, layers_out=want)
        seen = {}
        runner.model.layer_observer = lambda pos, hidden: seen.__setitem__(pos, hidden.cpu().double())
        runner.add_request("a")
        runner.step([StepEntry("a", toks, [])])
        assert len(seen) == len(want) == len(cfg["layers"])
        for n in range(len(want)):
            assert float((seen[n] - want[n]).abs().max()) <= 3e-5 * float(want[n].abs().max()), (name, n)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_slots_and_pages_used_again(models, dtype):
    """Four requests decode 150 tokens each through replayed decode passes; two more follow in their pages."""
    folder, cfg, w = models["A" if dtype == "float32" else "B"]
    runner = runner_for(folder, dtype, num_pages=92, max_requests=4, max_context=200)
    reqs = gt.random_requests(cfg, [160, 170, 158, 165, 175, 181], seed=9)
    first, second = dict(list(reqs.items())[:4]), dict(list(reqs.items())[4:])
    for part in (first, second):
        run_and_check(runner, traces.decoded_together(part, 150), cfg, w, part, dtype)
    assert runner.graph_replays > 100


def test_a_slot_and_its_pages_serve_one_request_after_another(models):
    folder, cfg, w = models["B"]
    for dtype in ("float32", "bfloat16"):
        runner = runner_for(folder, dtype, max_requests=1, num_pages=6)
        reqs = gt.random_requests(cfg, [33, 20, 47], seed=1)
        for rid, toks in reqs.items():
            run_and_check(runner, traces.portions({rid: toks}, (5, 2, 11)), cfg, w, {rid: toks}, dtype)


@pytest.mark.parametrize("name", ["B", "C"])
@pytest.mark.parametrize("decoding", [1, 3, 20])
def test_long_portions_beside_decoding_requests(models, name, decoding):
    """A step whose first requests decode and whose last ones bring long portions takes both forms of the latent
    attention at once; the portions go on later, in the middle of pages."""
    folder, cfg, w = models[name]
    runner = runner_for(folder, "bfloat16", max_requests=decoding + 2, num_pages=decoding * 4 + 120, max_tokens_per_step=512,
                        max_context=500)
    lens = [12 + (5 * i) % 11 for i in range(decoding)] + [430, 290]
    reqs = gt.random_requests(cfg, lens, seed=decoding)
    ids = list(reqs)
    short, (a, b) = ids[:decoding], ids[decoding:]
    steps = [{"entries": [(r, reqs[r][:-3], []) for r in short], "end": []}]
    cuts = [((0, 203), (0, 150)), ((203, 401), (150, 151)), ((401, 430), (151, 290))]
    for i, (ca, cb) in enumerate(cuts):
        entries = [(r, [reqs[r][len(reqs[r]) - 3 + i]], [0]) for r in short]
        for r, (lo, hi) in ((a, ca), (b, cb)):
            entries.append((r, reqs[r][lo:hi], list(range(0, hi - lo, 7)) + [hi - lo - 1]))
        steps.append({"entries": entries, "end": ids if i == 2 else []})
    run_and_check(runner, steps, cfg, w, reqs, "bfloat16")


def test_full_portions_replayed_from_a_captured_pass(models):
    """A long prompt in equal portions, captured once per power of two of the context and replayed."""
    folder, cfg, w = models["C"]
    toks = gt.random_requests(cfg, [1300], 4)["r0"]
    runner = runner_for(folder, "bfloat16", max_requests=2, num_pages=400, max_context=1400, graph_chunk_tokens=256)
    steps, i = [], 0
    while i < len(toks):
        n = min(256, len(toks) - i)
        steps.append({"entries": [("a", toks[i:i + n], [n - 1])], "end": []})
        i += n
    steps[-1]["end"] = ["a"]
    got = run_trace(runner, steps)
    replayed = runner.graph_replays
    assert replayed == 5
    check(got, cfg, w, {"a": toks}, "bfloat16", torch.float32)


@pytest.mark.parametrize("seed", range(8))
def test_random_configurations(tmp_path, seed):
    cfg = gt.random_config(100 + seed)
    w = gt.make_weights(cfg, seed)
    folder = gt.write_folder(str(tmp_path / "m"), cfg, w)
    reqs = gt.random_requests(cfg, [5, 141, 40, 19], seed)
    for dtype in ("float32", "bfloat16"):
        runner = runner_for(folder, dtype, num_pages=48)
        for steps in (traces.whole(reqs), traces.tail_decoded(reqs, 10), traces.mixed(reqs, seed=seed)):
            run_and_check(runner, steps, cfg, w, reqs, dtype)


def clear_greedy(cfg, w, length, n, seed):
    """A prompt and its ``n`` greedy tokens, without a near-tie that rounding could turn."""
    while True:
        seed += 1
        p = gt.random_requests(cfg, [length], seed)["r0"]
        gen = pg.greedy(cfg, w, p, n)
        top2 = torch.topk(pg.forward(cfg, w, p + gen)[len(p) - 1:-1], 2, dim=-1).values
        if float((top2[:, 0] - top2[:, 1]).min()) > 1e-3:
            return p, gen


@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_greedy_generation_through_the_scheduler(models, name):
    from mini_infer_b200.engine.llm import LLM
    from mini_infer_b200.sampling import SamplingParams
    folder, cfg, w = models[name]
    pairs = [clear_greedy(cfg, w, 3 + 7 * i, 10, 50 * i) for i in range(4)]
    prompts, wants = [p for p, _ in pairs], [g for _, g in pairs]
    llm = LLM(folder, dtype="float32", max_seq_len=96, max_running=3, max_tokens_per_step=16, prefill_chunk=8,
              page_size=8)
    outs = llm.generate(prompts, SamplingParams(greedy=True, max_new_tokens=10))
    assert [o.token_ids for o in outs] == wants
    assert any(s.prefill_tokens and s.decode_tokens for s in llm.last_history)      # portions beside decodes
    # nothing is kept per request but pages: steps are launched ahead of the scheduler's decision
    assert llm.runner.can_step_ahead([]) is True and not llm.runner.state_tensors
    assert llm.runner.cache.used_pages() == [0] * len(llm.runner.cache.pools)
    # a pool that the running requests outgrow: some are preempted and computed again
    small = LLM(folder, dtype="float32", max_seq_len=40, max_running=3, max_tokens_per_step=16, page_size=4, num_pages=12)
    outs = small.generate(prompts, SamplingParams(greedy=True, max_new_tokens=10))
    assert [o.token_ids for o in outs] == wants
    llm16 = LLM(folder, dtype="bfloat16", max_seq_len=96, max_running=3, max_tokens_per_step=16, page_size=8)
    outs16 = llm16.generate(prompts[:2], SamplingParams(greedy=True, max_new_tokens=4))
    assert all(len(o.token_ids) == 4 for o in outs16)


def test_trace_runner_and_command_line(models, tmp_path):
    import numpy as np
    folder, cfg, w = models["A"]
    toks = gt.random_requests(cfg, [19], 2)["r0"]
    ref = pg.forward(cfg, w, toks)
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": toks[:12], "want": [0, 11]}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": toks[12:], "want": [6]}], "end": ["a"]})]
    out = str(tmp_path / "out")
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                        "--out", out, "--max-tokens", "64", "--dump-intermediates"], input="\n".join(lines) + "\n", text=True,
                       capture_output=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
    a = torch.from_numpy(np.fromfile(os.path.join(out, "0.f32"), dtype="<f4").reshape(2, -1).copy())
    b = torch.from_numpy(np.fromfile(os.path.join(out, "1.f32"), dtype="<f4").reshape(1, -1).copy())
    scale = float(ref.abs().max())
    assert float((a.double() - ref[[0, 11]]).abs().max()) <= 4e-5 * scale
    assert float((b.double() - ref[[18]]).abs().max()) <= 4e-5 * scale
    last = len(cfg["layers"]) - 1
    assert os.path.getsize(os.path.join(out, f"0.layer{last}.f32")) == 12 * cfg["width"] * 4
    prompt, gen = clear_greedy(cfg, w, 6, 6, 0)
    cmd = [sys.executable, os.path.join(ROOT, "bin", "mini_infer"), "generate", "--model", folder, "--prompt-ids",
           ",".join(map(str, prompt)), "--max-new-tokens", "6", "--greedy", "--dtype", "float32", "--max-seq-len", "64",
           "--json"]
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = r.stdout.splitlines()
    assert json.loads(lines[lines.index("--- end ---") + 2])["token_ids"] == gen


def test_random_weights_of_a_configuration_are_served(tmp_path):
    from mini_infer_b200.engine.step import StepEntry
    cfg_path = str(tmp_path / "config.json")
    with open(cfg_path, "w") as f:
        json.dump(gt.CONFIG_B, f)
    out = str(tmp_path / "made")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "mini_infer"), "random-weights", "--config", cfg_path,
                        "--seed", "5", "--out", out], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    runner = runner_for(out, "bfloat16")
    runner.add_request("a")
    res = runner.step([StepEntry("a", [1, 2, 3], [2])])
    assert res.logits.shape == (1, gt.CONFIG_B["vocab"]) and bool(torch.isfinite(res.logits).all())


def test_a_step_that_fails_leaves_the_kept_token_ids_usable(models, monkeypatch):
    """A forward pass that raises after the embedding has written its token ids: the same step runs again."""
    from mini_infer_b200.engine.step import StepEntry
    folder, cfg, w = models["B"]
    runner = runner_for(folder, "float32")
    toks = gt.random_requests(cfg, [30], 8)["r0"]
    ref = pg.forward(cfg, w, toks)
    runner.add_request("a")
    runner.step([StepEntry("a", toks[:17], [])])
    part = runner.model.layers[-1].parts["mixer"]
    kept = part.forward
    monkeypatch.setattr(part, "forward", lambda *a: (_ for _ in ()).throw(RuntimeError("planted on the host")))
    with pytest.raises(RuntimeError, match="planted"):
        runner.step([StepEntry("a", [t ^ 1 for t in toks[17:25]], [7])])
    monkeypatch.setattr(part, "forward", kept)
    res = runner.step([StepEntry("a", toks[17:], [0, 12])])
    assert float((res.logits.double().cpu() - ref[[17, 29]]).abs().max()) <= 4e-5 * float(ref.abs().max())
