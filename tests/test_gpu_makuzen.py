"""Makuzen models on the engine against the plain restatement: prompts, decoding, portions, mixed batches, pages used again,
generation, serving and the trace runner."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracles import makuzen as O

pytestmark = pytest.mark.gpu
TOL = 2e-5        # FP32: the worst position
L = O.random_layer
BASE = O.random_config()
# other sizes, one layer without a feed-forward, other windows, rotations and expert counts per layer
OTHER = O.random_config([L(heads=3, dim=64, rot_dim=64, vdim=96, kv_rank=144, q_rank=72, window=70, base=1e6, experts=3, top=1, ff=72),
                         L(heads=20, dim=16, rot_dim=32, vdim=16, kv_rank=64, window=33, mlp=False),
                         L(heads=4, dim=128, rot_dim=32, vdim=64, kv_rank=256, window=500, scaling=None, scale=0.08, experts=9, top=4, shared=17)],
                        vocab=150, width=120, eps=1e-6, mult=1.0, scale=1.0)
# nothing is a multiple of eight; heads too wide for the expanded form in one layer
ODD = O.random_config([L(heads=17, dim=10, rot_dim=6, vdim=13, kv_rank=37, q_rank=21, window=7, experts=5, top=3, ff=13, shared=11),
                       L(heads=2, dim=140, rot_dim=10, vdim=30, kv_rank=50, q_rank=33, window=1, experts=1, top=1, ff=5, shared=3),
                       L(heads=1, dim=3, rot_dim=2, vdim=1, kv_rank=5, q_rank=3, window=90, scale=0.9, experts=2, top=2, ff=9, shared=1)],
                      vocab=101, width=52, eps=1e-3, mult=0.7)
CONFIGS = {"base": BASE, "other": OTHER, "odd": ODD}
_cache = {}


def _model(name):
    """configuration, weights, tokens of three sequences and the restatement's logits of each."""
    if name not in _cache:
        cfg = CONFIGS[name]
        w = O.random_weights(cfg, seed=len(name))
        g = torch.Generator().manual_seed(3)
        seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (300, 61, 23)]
        _cache[name] = (cfg, w, seqs, [O.forward(cfg, w, s) for s in seqs])
    return _cache[name]


def _create(cfg, w, precision="fp32", **kw):
    from nexus_b200.infer import EngineConfig, create_engine
    from nexus_b200.lm.hybrid import HybridWeights
    from nexus_b200.lm.makuzen import check_makuzen, makuzen_config
    hc = makuzen_config(cfg)
    check_makuzen(hc, w)
    kw = {"max_seqs": 4, "max_tokens": 512, "kv_tokens": 480, "cuda_graphs": False, **kw}
    return create_engine(HybridWeights(hc, w), EngineConfig(precision=precision, **kw))


def _engine(name, precision="fp32", **kw):
    cfg, w, _, _ = _model(name)
    return _create(cfg, w, precision, **kw)


def _errors(got, want):
    """Error of every position."""
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std()


def _check(errors, precision):
    """FP32: every position.  BF16: the mean, and all positions but a few."""
    if precision == "fp32":
        assert errors.max() < TOL, errors.max()
    else:
        assert errors.mean() < 2e-2 and (errors > 5e-2).sum() <= max(2, 0.03 * errors.numel()), (errors.mean(), errors.max())


def _feed(engine, name, plan, precision):
    """plan: steps of (request, token count); request i has the tokens of sequence i % 3.  Compares every position."""
    from nexus_b200.infer import Chunk
    from nexus_b200.ops import _cuda as K
    _, _, seqs, want = _model(name)
    V = CONFIGS[name]["vocab"]
    sid, at, errors = {}, {}, []
    for step in plan:
        chunks, refs = [], []
        for key, n in step:
            i = key % len(seqs)
            if key not in sid:
                sid[key], at[key] = engine.add_sequence(), 0
            lo = at[key]
            n = min(n, len(seqs[i]) - lo)
            chunks.append(Chunk(sid[key], seqs[i][lo: lo + n], places=list(range(n))))
            refs.append(want[i][lo: lo + n])
            at[key] += n
        errors.append(_errors(engine.forward(chunks)[:, :V], torch.cat(refs)))
        for key in [k for k in at if k in sid and at[k] >= len(seqs[k % len(seqs)])]:
            engine.free_sequence(sid.pop(key))
    for s in sid.values():
        engine.free_sequence(s)
    K.check_status()
    _check(torch.cat(errors), precision)


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("precision", ["fp32", "bf16"])
def test_prompt_decode_and_portions(name, precision):
    e = _engine(name, precision)
    _feed(e, name, [[(0, 300)]], precision)
    _feed(e, name, [[(1, 20)]] + [[(1, 1)]] * 41, precision)                                          # decoding
    _feed(e, name, [[(0, n)] for n in (2, 3, 16, 17, 1, 64, 2, 65, 18, 40, 72)], precision)           # portions
    _feed(e, name, [[(2, 1)] for _ in range(23)], precision)                                          # from the first token on
    assert e.free_blocks() == e.total_blocks()


@pytest.mark.parametrize("name", ["base", "odd"])
def test_long_decoding(name):
    e = _engine(name, "bf16", cuda_graphs=True)
    _feed(e, name, [[(0, 5)]] + [[(0, 1)]] * 295, "bf16")
    assert e.graphs_captured() == 1


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("precision", ["fp32", "bf16"])
def test_mixed_batches_with_pages_used_again(name, precision):
    """Up to four live sequences, portions beside single tokens, some left out of a step; keys 3, 4, .. are further requests
    admitted into the pages of finished ones."""
    e = _engine(name, precision)
    plan = [[(0, 40), (1, 7)], [(0, 1), (1, 2), (2, 5)], [(1, 1), (2, 18)], [(0, 170), (1, 51), (4, 31)], [(0, 1), (4, 1), (5, 9)],
            [(0, 88), (7, 2), (4, 29)], [(7, 59), (5, 14), (3, 23)], [(3, 100), (10, 61), (8, 1)], [(3, 1), (8, 20)], [(3, 2), (8, 2)],
            [(3, 174), (11, 17), (13, 1)], [(13, 1), (11, 6), (14, 19)]]
    _feed(e, name, plan, precision)
    assert e.free_blocks() == e.total_blocks() and e.sched.live_sequences() == 0


@pytest.mark.parametrize("precision", ["fp32", "bf16"])
def test_pages_of_other_sizes(precision):
    e = _engine("base", precision, block_size=24, kv_tokens=504)
    _feed(e, "base", [[(0, 100), (1, 23)], [(0, 1), (1, 1)], [(0, 199), (1, 25)], [(1, 12)]], precision)
    if precision == "bf16":
        with pytest.raises(ValueError, match="multiple of 8"):
            _engine("base", precision, block_size=12)


def test_layers_of_the_residual_stream():
    from nexus_b200.infer import Chunk
    cfg, w, seqs, _ = _model("other")
    want, got = [], []
    O.forward(cfg, w, seqs[2], capture=want)
    e = _engine("other")
    e.impl_capture(got)
    e.forward([Chunk(e.add_sequence(), seqs[2], 1)])
    assert len(got) == len(want) == len(cfg["layers"])
    for a, b in zip(got, want):
        assert ((a - b).norm() / b.norm()).item() < 1e-5


@pytest.mark.parametrize("precision", ["fp32", "bf16"])
@pytest.mark.parametrize("window", [1, 16, 21, 130])
def test_what_a_window_holds(window, precision):
    """One layer: a changed token moves the logits of the positions whose window still holds it, and leaves the next ones as
    they are, bit for bit - as part of a prompt, in portions and decoded.  (A weight that is small
    beside the others may round away.)"""
    from nexus_b200.infer import Chunk
    cfg = O.random_config([L(window=window, scale=0.3)])
    w = O.random_weights(cfg, seed=5)
    e = _create(cfg, w, precision, max_tokens=512)
    g = torch.Generator().manual_seed(0)
    T, V = window + 40, cfg["vocab"]
    for key in (0, 15, 16, 30):
        toks = torch.randint(0, V, (T,), generator=g).tolist()
        other = list(toks)
        other[key] = (toks[key] + 1) % V
        for cuts in ([T], [key + window - 1, T - key - window + 1] if key + window > 1 else [T], [min(20, T)] + [1] * (T - min(20, T)), [2] * (T // 2)):
            outs = []
            for t in (toks, other):
                s, at, got = e.add_sequence(), 0, []
                for n in cuts:
                    got.append(e.forward([Chunk(s, t[at: at + n], places=list(range(n)))])[:, :V].clone())
                    at += n
                e.free_sequence(s)
                outs.append(torch.cat(got))
            same = (outs[0] == outs[1]).all(1)
            n = same.numel()
            assert same[:key].all() and same[key + window:].all(), (key, cuts)
            inside = same[key: min(n, key + window)]
            most = (0.0 if window <= 21 else 0.2) if precision == "fp32" else (0.4 if window <= 21 else 0.8)
            assert not inside[0] and inside.float().mean() <= most, (key, cuts)


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


def test_server_preemption():
    from nexus_b200.infer import SamplingParams, generate
    from nexus_b200.serve import Config, Request, Server
    e = _engine("base", "fp32", kv_tokens=96, context=96)
    prompts = [[1, 2, 3, 4, 5, 6], [7, 8, 9, 10, 11, 12], [13, 14, 15, 16, 17, 18]]
    want = [generate(e, p, 40) for p in prompts]
    srv = Server(e, Config(max_batch_tokens=64, max_running=3))
    futs = [srv.submit(Request(p, 40, sampling=SamplingParams(temperature=0.0))) for p in prompts]
    srv.run_until_idle(800)
    assert [f.result(timeout=1).tokens for f in futs] == want and srv.metrics.preemptions > 0


@pytest.mark.parametrize("name", ["base", "other"])
def test_decode_graphs_and_pipelined_decode(name):
    """Captured decode steps give the tokens of eager ones - the routing of the experts is part of the captured step - also
    when step n + 1 is launched before step n is read."""
    from nexus_b200.infer import SamplingParams, generate
    from nexus_b200.ops import _cuda as K
    from nexus_b200.serve import Config, Request, Server
    prompt = [5, 17, 3, 80, 41]
    base = generate(_engine(name, "bf16"), prompt, 120)
    e = _engine(name, "bf16", cuda_graphs=True)
    assert generate(e, prompt, 120) == base and e.graphs_captured() >= 1 and e.last_step().graph
    assert generate(e, prompt, 120) == base
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
    assert outs[True, True] == outs[True, False] and outs[False, True] == outs[False, False]
    K.check_status()


def test_fork_truncate_and_speculation():
    """No state beside the cache pages: sequences can be cut back anywhere, forked, and drafted for."""
    from nexus_b200.infer import Chunk, QuantOptions, generate, speculative_generate
    cfg, w, seqs, want = _model("base")
    V = cfg["vocab"]
    e = _engine("base", "fp32")
    a = e.add_sequence()
    e.forward([Chunk(a, seqs[0][:50], 1)])
    b = e.fork_sequence(a)
    for s in (a, b):                       # both branches go on alone
        assert _errors(e.forward([Chunk(s, seqs[0][50:60], 10)])[:, :V], want[0][50:60]).max() < TOL
    e.truncate(a, 21)
    assert _errors(e.forward([Chunk(a, seqs[0][21:40], 19)])[:, :V], want[0][21:40]).max() < TOL
    e.truncate(a, 0)
    assert _errors(e.forward([Chunk(a, seqs[1][:5], 5)])[:, :V], want[1][:5]).max() < TOL
    assert e.length(a) == 5 and e.length(b) == 60
    e.free_sequence(a)
    e.free_sequence(b)
    assert speculative_generate(e, [5, 17, 3], 16, draft_layers=1, gamma=3) == generate(e, [5, 17, 3], 16)
    with pytest.raises(ValueError, match="quantised"):
        _engine("base", "bf16", quant=QuantOptions(weights="w8a8"))


def test_many_rows_per_expert():
    """Enough rows that the experts run as a grouped GEMM, in tiles of 128 and of 256."""
    from nexus_b200.infer import Chunk
    from nexus_b200.infer.experts import alignment
    cfg = O.random_config([L(experts=2, top=1, ff=40, shared=24, window=9), L(experts=3, top=2, ff=264, window=30)], vocab=70, width=64)
    w = O.random_weights(cfg, seed=9)
    e = _create(cfg, w, "bf16", max_tokens=2048, kv_tokens=2048)
    toks = torch.randint(0, 70, (1400,), generator=torch.Generator().manual_seed(2)).tolist()
    assert [alignment(e, x.experts, 1400) for x in e.model.layers] == [256, 256] and alignment(e, e.model.layers[1].experts, 200) == 128
    want = O.forward(cfg, w, toks)
    _check(_errors(e.forward([Chunk(e.add_sequence(), toks, places=list(range(1400)))])[:, :70], want), "bf16")
    _check(_errors(e.forward([Chunk(e.add_sequence(), toks[:200], places=list(range(200)))])[:, :70], want[:200]), "bf16")


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
             {"step": 3, "entries": [{"id": "z", "tokens": seqs[2], "want": [22]}, {"id": "x", "tokens": seqs[0][71:300], "want": [228]}],
              "end": ["x", "z"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens",
                        "384"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600,
                       env={**os.environ, "PYTHON": sys.executable})
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (out / "1.f32").exists()
    refs = {0: want[0][[69, 3]], 2: want[1][[2, 60]], 3: torch.stack([want[2][22], want[0][299]])}
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
