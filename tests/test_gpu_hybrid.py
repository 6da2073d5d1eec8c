"""Gugedra models on the engine against the plain restatement: prompts, decoding, portions, mixed batches, slots and pages
that are used again, generation, serving and the trace runner."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracles import gugedra as O

pytestmark = pytest.mark.gpu
TOL = 2e-5        # FP32: the worst position
BASE = O.random_config()
OTHER = O.random_config(("delta", "parallel", "delta", "delta"), vocab=150, width=72, ff=88, side=12, logit_softcap=20.0, eps=1e-4,
                        left={"heads": 6, "kv_heads": 1, "dim": 64, "vdim": 64, "mask": {"size": 150},
                              "rot": {"base": 90000.0, "dims": 64}, "softcap": 25.0, "scale": 0.125},
                        right={"heads": 2, "vdim": 24, "state": 40, "groups": 1, "conv": 2, "norm_groups": 1},
                        delta={"heads": 3, "kv_heads": 3, "dim": 16, "vdim": 24, "conv": 5}, left_scale=1.4, right_scale=0.5)
ODD = O.random_config(("parallel", "parallel", "delta"), vocab=101, width=52, ff=50, side=10,
                      left={"heads": 3, "kv_heads": 3, "dim": 10, "vdim": 13, "mask": {"size": 5}, "rot": {"base": 100.0, "dims": 2}},
                      right={"heads": 5, "vdim": 7, "state": 9, "groups": 5, "conv": 3, "norm_groups": 5},
                      delta={"heads": 4, "kv_heads": 1, "dim": 11, "vdim": 6, "conv": 1})
CONFIGS = {"base": BASE, "other": OTHER, "odd": ODD}
_cache = {}


def _model(name):
    """weights, tokens of three sequences and the restatement's logits of each."""
    if name not in _cache:
        cfg = CONFIGS[name]
        w = O.random_weights(cfg, seed=len(name))
        g = torch.Generator().manual_seed(3)
        seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (170, 61, 23)]
        _cache[name] = (cfg, w, seqs, [O.forward(cfg, w, s) for s in seqs])
    return _cache[name]


def _engine(name, precision="fp32", **kw):
    from nexus_b200.infer import EngineConfig, create_engine
    from nexus_b200.lm.hybrid import HybridWeights, check_tensors, gugedra_config
    cfg, w, _, _ = _model(name)
    hc = gugedra_config(cfg)
    check_tensors(hc, w)
    kw = {"max_seqs": 4, "max_tokens": 512, "kv_tokens": 352, "cuda_graphs": False, **kw}
    return create_engine(HybridWeights(hc, w), EngineConfig(precision=precision, **kw))


def _errors(got, want):
    """Error of every position."""
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std()


def _err(got, want):
    return _errors(got, want).max().item()


def _check(errors, precision):
    """FP32: every position.  BF16: the mean, and all positions but a few - in a random model of this size a token here and
    there sits where a norm of a nearly cancelled vector magnifies the rounding of the activations."""
    if precision == "fp32":
        assert errors.max() < TOL, errors.max()
    else:
        assert errors.mean() < 3e-2 and (errors > 6e-2).sum() <= max(2, 0.03 * errors.numel()), (errors.mean(), errors.max())


def _feed(engine, name, plan, precision):
    """plan: steps of (sequence index, token count); compares every position's logits."""
    from nexus_b200.infer import Chunk
    _, _, seqs, want = _model(name)
    V = CONFIGS[name]["vocab"]
    sid, at, errors = {}, {}, []
    for step in plan:
        chunks, refs = [], []
        for i, n in step:
            key = i
            i = i % len(seqs)
            if key not in sid:
                sid[key], at[key] = engine.add_sequence(), 0
            lo = at[key]
            n = min(n, len(seqs[i]) - lo)
            chunks.append(Chunk(sid[key], seqs[i][lo: lo + n], places=list(range(n))))
            refs.append(want[i][lo: lo + n])
            at[key] += n
        got = engine.forward(chunks)[:, :V]
        errors.append(_errors(got, torch.cat(refs)))
        for key in [k for k in at if k in sid and at[k] >= len(seqs[k % len(seqs)])]:
            engine.free_sequence(sid.pop(key))
    _check(torch.cat(errors), precision)


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("precision", ["fp32", "bf16"])
def test_prompt_decode_and_portions(name, precision):
    e = _engine(name, precision)
    _feed(e, name, [[(0, 170)]], precision)
    _feed(e, name, [[(1, 20)]] + [[(1, 1)]] * 41, precision)                                  # decoding
    _feed(e, name, [[(0, n)] for n in (2, 3, 16, 17, 1, 64, 2, 65)], precision)               # portions
    _feed(e, name, [[(2, 1)] for _ in range(23)], precision)                                  # from the first token on
    assert e.free_blocks() == e.total_blocks()


@pytest.mark.parametrize("name", ["base", "other"])
@pytest.mark.parametrize("precision", ["fp32", "bf16"])
def test_mixed_batches_with_pages_and_slots_used_again(name, precision):
    """Up to four live sequences, portions beside single tokens, some left out of a step; keys 3, 4, .. are further
    requests with the tokens of sequence key % 3, admitted into the slots and pages of finished ones."""
    e = _engine(name, precision)
    plan = [[(0, 40), (1, 7)], [(0, 1), (1, 2), (2, 5)], [(1, 1), (2, 18)], [(0, 70), (1, 50), (3, 31)], [(0, 1), (3, 1), (1, 9)],
            [(0, 60), (4, 2), (3, 100)], [(4, 59), (3, 40), (5, 23)], [(6, 100), (7, 61), (8, 1)], [(6, 1), (8, 20)], [(6, 2), (8, 2)],
            [(6, 80)]]
    _feed(e, name, plan, precision)
    assert e.free_blocks() == e.total_blocks() and e.sched.live_sequences() == 0


def test_layers_of_the_residual_stream():
    cfg, w, seqs, _ = _model("base")
    want, got = [], []
    O.forward(cfg, w, seqs[2], capture=want)
    e = _engine("base")
    e.impl_capture(got)
    from nexus_b200.infer import Chunk
    e.forward([Chunk(e.add_sequence(), seqs[2], 1)])
    assert len(got) == len(want) == len(cfg["layers"])
    for a, b in zip(got, want):
        assert ((a - b).norm() / b.norm()).item() < 1e-5


def _greedy(name, prompt, new):
    cfg, w, _, _ = _model(name)
    toks = list(prompt)
    for _ in range(new):
        toks.append(int(O.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_and_server():
    from nexus_b200.infer import SamplingParams, generate
    from nexus_b200.serve import Config, Request, Server
    e = _engine("base", "fp32")
    prompts = [[5, 17, 3], [44, 2, 9, 100, 61, 7, 33], [12]]
    want = [_greedy("base", p, 12) for p in prompts]
    assert [generate(e, p, 12) for p in prompts] == want
    greedy = SamplingParams(temperature=0.0)
    srv = Server(e, Config(max_batch_tokens=64, max_running=2))
    futs = [srv.submit(Request(p, 12, sampling=greedy)) for p in prompts * 2]
    srv.run_until_idle(400)
    assert [f.result(timeout=1).tokens for f in futs] == want * 2
    assert e.free_blocks() == e.total_blocks()


def test_server_preemption_recomputes_the_state():
    """Too few pages for the requests: a preempted one comes back as two adjacent chunks (prompt, own output) that are
    one segment of the recurrence."""
    from nexus_b200.infer import SamplingParams, generate
    from nexus_b200.serve import Config, Request, Server
    e = _engine("base", "fp32", kv_tokens=96, context=96)
    prompts = [[1, 2, 3, 4, 5, 6], [7, 8, 9, 10, 11, 12], [13, 14, 15, 16, 17, 18]]
    want = [generate(e, p, 40) for p in prompts]
    srv = Server(e, Config(max_batch_tokens=64, max_running=3))
    futs = [srv.submit(Request(p, 40, sampling=SamplingParams(temperature=0.0))) for p in prompts]
    srv.run_until_idle(800)
    got = [f.result(timeout=1) for f in futs]
    assert [r.tokens for r in got] == want and srv.metrics.preemptions > 0


@pytest.mark.parametrize("name", ["base", "other"])
def test_decode_graphs_and_pipelined_decode(name):
    """Captured decode steps give the tokens of eager ones (a captured step must advance the states exactly once), also
    when step n + 1 is launched before step n is read; long decoding past the window."""
    from nexus_b200.infer import SamplingParams, generate
    from nexus_b200.ops import _cuda as K
    from nexus_b200.serve import Config, Request, Server
    prompt = [5, 17, 3, 80, 41]
    eager = _engine(name, "bf16")
    base = generate(eager, prompt, 180)
    e = _engine(name, "bf16", cuda_graphs=True)
    assert generate(e, prompt, 180) == base and e.graphs_captured() >= 1 and e.last_step().graph
    assert generate(e, prompt, 180) == base
    outs = {}
    for graphs in (False, True):
        for pipe in (False, True):
            eng = _engine(name, "bf16", cuda_graphs=graphs)
            srv = Server(eng, Config(max_batch_tokens=128, max_running=3, pipeline_decode=pipe))
            futs = [srv.submit(Request([7 + i, 30, 2 * i + 1], 8 + 5 * i, sampling=SamplingParams(
                temperature=0.0 if i % 2 else 0.8, top_k=20, seed=i, repetition_penalty=1.1))) for i in range(5)]
            srv.run_until_idle(500)
            outs[graphs, pipe] = [f.result(timeout=1).tokens for f in futs]
            assert eng.free_blocks() == eng.total_blocks()
    assert all(v == outs[False, False] for v in outs.values())
    K.check_status()


def test_decode_logits_of_captured_steps():
    from nexus_b200.infer import Chunk
    _, _, seqs, want = _model("base")
    e = _engine("base", "bf16", cuda_graphs=True)
    a, b = e.add_sequence(), e.add_sequence()
    e.forward([Chunk(a, seqs[0][:30], 0), Chunk(b, seqs[1][:9], 0)])
    errors = []
    for t in range(50):
        got = e.forward([Chunk(a, [seqs[0][30 + t]], 1, True), Chunk(b, [seqs[1][9 + t]], 1, True)])
        assert e.last_step().graph
        errors.append(_errors(got[:, : BASE["vocab"]], torch.stack([want[0][30 + t], want[1][9 + t]])))
    _check(torch.cat(errors), "bf16")


def test_fork_truncate_and_refusals():
    from nexus_b200.infer import Chunk, EngineConfig, QuantOptions, create_engine, speculative_generate
    cfg, w, seqs, want = _model("base")
    V = cfg["vocab"]
    e = _engine("base", "fp32")
    a = e.add_sequence()
    e.forward([Chunk(a, seqs[0][:50], 1)])
    b = e.fork_sequence(a)
    for s in (a, b):                       # both branches go on alone
        got = e.forward([Chunk(s, seqs[0][50:60], 10)])
        assert _err(got[:, :V], want[0][50:60]) < TOL
    with pytest.raises(ValueError, match="recurrent state"):
        e.truncate(a, 10)
    e.truncate(a, 0)                       # starting over is possible
    assert _err(e.forward([Chunk(a, seqs[1][:5], 5)])[:, :V], want[1][:5]) < TOL
    with pytest.raises(ValueError, match="adjacent"):
        e.forward([Chunk(a, [1], 1), Chunk(b, [2], 1), Chunk(a, [3], 1)])
    assert e.length(a) == 5 and e.length(b) == 60
    got = e.forward([Chunk(a, seqs[1][5:7], 1), Chunk(a, seqs[1][7:9], 1)])      # adjacent chunks are one segment
    assert _err(got[:, :V], want[1][[6, 8]]) < TOL
    with pytest.raises(ValueError):
        speculative_generate(e, [1, 2, 3], 4, draft_layers=1, gamma=2)
    with pytest.raises(ValueError, match="quantised"):
        _engine("base", "bf16", quant=QuantOptions(weights="w8a8"))
    from nexus_b200.lm.hybrid import HybridWeights, gugedra_config
    with pytest.raises(ValueError, match="CUDA"):
        create_engine(HybridWeights(gugedra_config(cfg), w), EngineConfig(device="cpu", precision="fp32"))


def _save(tmp_path, name):
    from nexus_b200.interop.safetensors import save_file
    cfg, w, _, _ = _model(name)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))
    return str(tmp_path)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(tmp_path, dtype):
    _, _, seqs, want = _model("base")
    folder = _save(tmp_path, "base")
    out = tmp_path / "out"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": seqs[0][:70], "want": [69, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": seqs[1][:2], "want": []}, {"id": "x", "tokens": seqs[0][70:71], "want": []}],
              "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": seqs[1][2:61], "want": [0, 58]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "z", "tokens": seqs[2], "want": [22]}, {"id": "x", "tokens": seqs[0][71:170], "want": [98]}],
              "end": ["x", "z"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens",
                        "256"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600,
                       env={**os.environ, "PYTHON": sys.executable})
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (out / "1.f32").exists()
    refs = {0: want[0][[69, 3]], 2: want[1][[2, 60]], 3: torch.stack([want[2][22], want[0][169]])}
    errors = []
    for i, ref in refs.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(ref.shape))
        errors.append(_errors(got, ref))
    _check(torch.cat(errors), "fp32" if dtype == "float32" else "bf16")


def test_generate_command(tmp_path, capsys):
    from nexus_b200.tools import generate as tool
    folder = _save(tmp_path, "base")
    assert tool.main(["--model", folder, "--precision", "fp32", "--prompt", "5,17,3", "--prompt", "12", "--max-new", "6"]) == 0
    lines = capsys.readouterr().out.strip().splitlines()
    assert [json.loads(ln)["tokens"] for ln in lines] == [_greedy("base", [5, 17, 3], 6), _greedy("base", [12], 6)]
