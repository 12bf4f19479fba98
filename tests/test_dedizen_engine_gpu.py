"""Dedizen through the engine's own step function, cache and state manager, scheduler and entry points, against the plain
model: whole prompts, decoding token by token, portions down to two tokens, unequal requests in one batch, pages and
slots used again, long decoding past every chunk, greedy generation; and models of random shape."""

import json
import os
import random
import subprocess
import sys

import pytest
import torch

import dedizen_tiny as dt
import plain_dedizen as pd
import traces
from engine_harness import run_trace

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# of the largest logit; plus, at every position, a multiple of what rounding alone (32 bits, or 16 where the engine's
# bfloat16 path stores 16) does to the plain model there: a head's first read-out is a multiple of one vector that is then
# normalised, so it hangs on the sign of one dot product, whoever computes it
TOL = {"float32": 4e-5, "bfloat16": 2e-2}
SLACK = {"float32": 8.0, "bfloat16": 1.5}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in dt.CONFIGS.items():
        w = dt.make_weights(cfg, seed=31 + ord(name))
        out[name] = (dt.write_folder(str(tmp_path_factory.mktemp("dz_" + name)), cfg, w), cfg, w)
    return out


def runner_for(folder, dtype, **kw):
    from mini_infer_b200.engine.loading import load_model
    from mini_infer_b200.engine.step import ModelRunner
    model, rt, _ = load_model(folder, dtype, "cuda:0")
    args = dict(page_size=8, num_pages=40, max_requests=4, max_tokens_per_step=256, max_context=352)
    args.update(kw)
    return ModelRunner(model, rt, **args)


def jitter(seed):
    """Every number off by up to half a unit in bfloat16's last place, at random."""
    g = torch.Generator().manual_seed(seed)
    return lambda x: x * (1 + (torch.rand(x.shape, generator=g, dtype=x.dtype) - 0.5) * 2 ** -8)


_references = {}


def reference(cfg, w, toks, dtype):
    """Plain logits, and how far rounding alone moves them at every position."""
    key = (id(w), dtype, tuple(toks))
    if key not in _references:
        out = pd.forward(cfg, w, toks)
        if dtype == "float32":
            others = [pd.forward(cfg, w, toks, dtype=torch.float32).double()]
        else:
            others = [pd.forward(cfg, w, toks, rnd=r) for r in [pd.as_bfloat16] + [jitter(i) for i in range(4)]]
        moved = torch.stack([(o - out).abs().max(dim=1).values for o in others]).max(dim=0).values
        _references[key] = (out, moved)
    return _references[key]


def run_and_check(runner, steps, cfg, w, reqs, dtype):
    got = run_trace(runner, steps)
    for (rid, pos), row in sorted(got.items()):
        want, moved = reference(cfg, w, reqs[rid], dtype)
        scale = float(want.abs().max())
        err = float((row.double() - want[pos]).abs().max()) / scale
        allowed = TOL[dtype] + SLACK[dtype] * float(moved[pos]) / scale
        assert err <= allowed, f"request {rid} position {pos}: {err:.2e} of the largest logit, {allowed:.2e} allowed"
    assert runner.cache.used_pages() == [0] * len(runner.cache.pools)
    return got


@pytest.mark.parametrize("name", sorted(dt.CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_cutting_against_the_plain_model(models, name, dtype):
    folder, cfg, w = models[name]
    runner = runner_for(folder, dtype, max_requests=6, num_pages=90)
    reqs = dt.random_requests(cfg, [150, 1, 23, 2, 41, 9], seed=ord(name))
    results = []
    for steps in (traces.whole(reqs), traces.tail_decoded(reqs, tail=36), traces.portions(reqs),
                  traces.portions(reqs, (2,)), traces.portions(reqs, (64, 3, 65)),
                  traces.mixed(reqs, max_live=3, seed=2, decode_tail=14),
                  traces.decoded_together({r: t for r, t in reqs.items() if len(t) > 1},
                                          {"r0": 30, "r2": 12, "r3": 1, "r4": 40, "r5": 3})):
        results.append(run_and_check(runner, steps, cfg, w, reqs, dtype))
    if name == "C" and dtype == "bfloat16":
        from mini_infer_b200.ops import functional as F
        left = [l.parts["mixer"] for l in runner.model.layers if "mixer_b" in l.parts]
        assert all(p._tensor_cores and p._split_decode and F.prefill_attention_tc_supported(p.dk, 8) for p in left)
    if dtype == "float32":
        # the 32-bit path gives the same bits however the work was cut and batched
        for other in results[1:]:
            for key, row in other.items():
                assert torch.equal(row, results[0][key]), key


def test_layer_by_layer(models):
    """The residual stream after every layer (a pair of normalised outputs may still be on its way to it)."""
    from mini_infer_b200.engine.step import StepEntry
    for name in ("A", "B", "D"):
        folder, cfg, w = models[name]
        runner = runner_for(folder, "float32")
        toks = dt.random_requests(cfg, [29], 3)["r0"]
        want, low = [], []
        pd.forward(cfg, w, toks, layers_out=want)
        pd.forward(cfg, w, toks, layers_out=low, dtype=torch.float32)
        seen = {}
        runner.model.layer_observer = lambda pos, hidden: seen.__setitem__(pos, hidden.cpu().double())
        runner.add_request("a")
        runner.step([StepEntry("a", toks, [])])
        runner.release("a")
        runner.model.layer_observer = None
        assert len(seen) == len(want)
        for n in range(len(want)):
            moved = float((low[n].double() - want[n]).abs().max())
            assert float((seen[n] - want[n]).abs().max()) <= 3e-5 * float(want[n].abs().max()) + 8 * moved, (name, n)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_slots_and_pages_used_again(models, dtype):
    """Four requests decode 150 tokens each through replayed decode passes, past many chunks, then two more in their
    pages and state slots (which must start from zero)."""
    folder, cfg, w = models["A" if dtype == "float32" else "C"]
    runner = runner_for(folder, dtype, num_pages=100, max_requests=4, max_context=200)
    reqs = dt.random_requests(cfg, [160, 170, 158, 165, 175, 181], seed=9)
    for part in (dict(list(reqs.items())[:4]), dict(list(reqs.items())[4:])):
        run_and_check(runner, traces.decoded_together(part, 150), cfg, w, part, dtype)
    assert runner.graph_replays > 100


def test_one_slot_and_its_pages_serve_one_request_after_another(models):
    folder, cfg, w = models["B"]
    runner = runner_for(folder, "float32", max_requests=1, num_pages=12)
    reqs = dt.random_requests(cfg, [33, 20, 27], seed=1)
    for rid, toks in reqs.items():
        run_and_check(runner, traces.portions({rid: toks}, (5, 2, 11)), cfg, w, {rid: toks}, "float32")


def test_a_pool_that_holds_no_more_than_the_chunks_need(models):
    """The pages of passed chunks serve later tokens of the same requests: 590 tokens through 26 pages of eight."""
    folder, cfg, w = models["C"]
    reqs = dt.random_requests(cfg, [300, 290], seed=4)
    runner = runner_for(folder, "bfloat16", max_requests=2, num_pages=26, max_tokens_per_step=32)
    run_and_check(runner, traces.portions(reqs, (16, 2, 13, 1)), cfg, w, reqs, "bfloat16")


@pytest.mark.parametrize("name", ["A", "E"])
def test_greedy_generation_through_the_scheduler(models, name):
    from mini_infer_b200.engine.llm import LLM
    from mini_infer_b200.sampling import SamplingParams
    folder, cfg, w = models[name]
    prompts, wants, seed = [], [], 0
    while len(prompts) < 4:
        seed += 1
        p = dt.random_requests(cfg, [3 + 7 * len(prompts)], seed)["r0"]
        gen = pd.greedy(cfg, w, p, 10)
        top2 = torch.topk(pd.forward(cfg, w, p + gen)[len(p) - 1:-1], 2, dim=-1).values
        if float((top2[:, 0] - top2[:, 1]).min()) > 1e-2:        # no near-tie that rounding could turn
            prompts.append(p)
            wants.append(gen)
    llm = LLM(folder, dtype="float32", max_seq_len=96, max_running=3, max_tokens_per_step=16, prefill_chunk=8, page_size=8)
    outs = llm.generate(prompts, SamplingParams(greedy=True, max_new_tokens=10))
    assert [o.token_ids for o in outs] == wants
    assert any(s.prefill_tokens and s.decode_tokens for s in llm.last_history)      # portions beside decodes
    assert llm.runner.cache.used_pages() == [0] * len(llm.runner.cache.pools)
    llm16 = LLM(folder, dtype="bfloat16", max_seq_len=96, max_running=3, max_tokens_per_step=16, page_size=8)
    assert all(len(o.token_ids) == 4 for o in llm16.generate(prompts[:2], SamplingParams(greedy=True, max_new_tokens=4)))


def test_trace_runner_and_command_line(models, tmp_path):
    import numpy as np
    folder, cfg, w = models["D"]
    toks = dt.random_requests(cfg, [19], 2)["r0"]
    ref = pd.forward(cfg, w, toks)
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": toks[:12], "want": [0, 11]}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": toks[12:], "want": [6]}], "end": ["a"]})]
    out = str(tmp_path / "out")
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                        "--out", out, "--max-tokens", "64"], input="\n".join(lines) + "\n", text=True,
                       capture_output=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
    for step, places in ((0, [0, 11]), (1, [18])):
        got = torch.from_numpy(np.fromfile(os.path.join(out, f"{step}.f32"), dtype="<f4").reshape(len(places), -1).copy())
        assert float((got.double() - ref[places]).abs().max()) <= 1e-4 * float(ref.abs().max())
    seed = 0
    while True:
        seed += 1
        prompt = dt.random_requests(cfg, [6], seed)["r0"]
        gen = pd.greedy(cfg, w, prompt, 6)
        top2 = torch.topk(pd.forward(cfg, w, prompt + gen)[len(prompt) - 1:-1], 2, dim=-1).values
        if float((top2[:, 0] - top2[:, 1]).min()) > 1e-2:
            break
    cmd = [sys.executable, os.path.join(ROOT, "bin", "mini_infer"), "generate", "--model", folder, "--prompt-ids",
           ",".join(map(str, prompt)), "--max-new-tokens", "6", "--greedy", "--dtype", "float32", "--max-seq-len", "64", "--json"]
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = r.stdout.splitlines()
    assert json.loads(lines[lines.index("--- end ---") + 2])["token_ids"] == gen


def test_random_weights_of_a_configuration_are_served(tmp_path):
    from mini_infer_b200.engine.step import StepEntry
    cfg_path, out = str(tmp_path / "config.json"), str(tmp_path / "made")
    with open(cfg_path, "w") as f:
        json.dump(dt.CONFIG_A, f)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "mini_infer"), "random-weights", "--config", cfg_path,
                        "--seed", "5", "--out", out], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    runner = runner_for(out, "bfloat16")
    runner.add_request("a")
    res = runner.step([StepEntry("a", [1, 2, 3], [2])])
    assert res.logits.shape == (1, dt.CONFIG_A["vocab"]) and bool(torch.isfinite(res.logits).all())


# ---- models of random shape ------------------------------------------------------------------------------ #

def random_config(seed: int) -> dict:
    r = random.Random(seed)
    wide = r.random() < 0.35                                     # sizes the tensor-core kernels take
    layers = []
    for _ in range(r.randint(1, 5)):
        ff = None if r.random() < 0.25 else r.choice([8, 20, 33, 64, 96])
        kind = r.choice(["mlstm", "rglru", "parallel", "parallel"])
        if kind == "mlstm":
            layers.append(dt._mlstm(r.randint(1, 5), r.choice([3, 8, 17, 32, 66, 130] if wide else [3, 8, 17, 32]),
                                    r.choice([5, 8, 24, 65, 128] if wide else [5, 8, 24]), r.choice([1.0, 4.0, 15.0, 30.0]), ff))
        elif kind == "rglru":
            blocks = r.choice([1, 2, 3, 5])
            layers.append(dt._rglru(blocks * r.choice([1, 7, 16, 33, 70] if wide else [1, 7, 16]), blocks, r.randint(1, 6), ff))
        else:
            kv = r.choice([1, 1, 2, 3])
            dim = r.choice([64, 128] if wide else [4, 10, 24, 34, 96])
            rot = None
            if r.random() < 0.85:
                scaling = None if r.random() < 0.2 else (r.choice([1.5, 4.0, 16.0]), r.choice([32, 100, 4096]),
                                                         r.choice([8.0, 32.0]), r.choice([0.5, 1.0]))
                rot = dt._rot(r.choice([d for d in range(2, dim + 1, 2)]), r.choice([30.0, 1000.0, 5e5]), scaling)
            decay = [r.choice([0.1, 0.5, 0.9, 0.99, 0.9999, 1.0]) for _ in range(r.randint(1, 4))]
            layers.append(dt._parallel(kv * r.choice([1, 1, 2, 4]), kv, dim, r.choice([1, 2, 5, 16, 17, 31, 64, 100]),
                                       r.choice([0.05, 0.1, 0.3]), rot, decay, r.choice([1, 4, 16, 40]), r.choice([3, 8, 32, 70]), ff))
    return {"architecture": "Dedizen", "vocab": r.randint(40, 300), "width": r.choice([64, 96, 128] if wide else [20, 33, 48, 70]),
            "norm": {"eps": r.choice([1e-6, 1e-5])}, "layers": layers}


@pytest.mark.parametrize("seed", list(range(10)))
def test_models_of_random_shape_in_several_cuttings(seed, tmp_path):
    cfg = random_config(seed)
    w = dt.make_weights(cfg, seed=200 + seed)
    folder = dt.write_folder(str(tmp_path / "m"), cfg, w)
    reqs = dt.random_requests(cfg, [133, 2, 37], seed=seed)
    for dtype in ("float32", "bfloat16"):
        runner = runner_for(folder, dtype, max_requests=3, num_pages=60)
        for steps in (traces.whole(reqs), traces.tail_decoded(reqs, tail=20), traces.portions(reqs),
                      traces.mixed(reqs, max_live=3, seed=seed, decode_tail=9)):
            run_and_check(runner, steps, cfg, w, reqs, dtype)
