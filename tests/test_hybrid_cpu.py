"""Host side of the hybrid decoder: configuration, weights, registry, the scheduler's segments and wanted places, and the plain
restatement's own consistency.  No GPU."""
import copy
import json

import numpy as np
import pytest
import torch

from oracles import gugedra as O


def _plan(sched, chunks, short=16, max_tokens=512):
    """chunks: (sequence, tokens, wanted places or None)."""
    return sched.plan([c[0] for c in chunks], [c[1] for c in chunks], [7] * sum(c[1] for c in chunks),
                      [1 if c[2] is None else -1 for c in chunks], [0] * len(chunks), False, max_tokens,
                      [c[2] or [] for c in chunks], short)


def _tables(sched, width):
    buf = np.zeros((10, width), dtype=np.int32)
    sched.write(buf.ctypes.data, width)
    sched.write_segments(buf[6:].ctypes.data, width)
    return buf


def test_segments_of_a_mixed_step():
    from nexus_b200 import _native
    s = _native.KvScheduler(40, 16, 4, 256)
    a, b, c, d = (s.add() for _ in range(4))
    _plan(s, [(a, 30, None), (b, 5, None)])
    p = _plan(s, [(a, 40, [39, 0]), (b, 1, [0]), (c, 2, []), (d, 1, None)])
    assert p["segments"] == [(2, 1, 2), (1, 2, 2), (1, 40, 40)] and p["logit_rows"] == 4
    t = _tables(s, 64)
    segs = [tuple(t[6:, i]) for i in range(4)]
    # one-token segments first, then the short one, then the long one; rows stay where the chunks were
    assert segs == [(40, 1, 5, b), (43, 1, 0, d), (41, 2, 0, c), (0, 40, 30, a)]
    assert (t[6:, 4:] == 0).all()
    assert t[5, :4].tolist() == [39, 0, 40, 43]                     # the wanted rows, in the order asked for
    assert p["logit_seq"] == [a, a, b, d]


def test_adjacent_chunks_are_one_segment_and_bad_places_change_nothing():
    from nexus_b200 import _native
    s = _native.KvScheduler(40, 16, 4, 256)
    a, b = s.add(), s.add()
    p = _plan(s, [(a, 10, None), (a, 20, None), (b, 3, None)])
    assert p["segments"] == [(0, 0, 0), (1, 3, 3), (1, 30, 30)]
    t = _tables(s, 33)
    assert tuple(t[6:, 1]) == (0, 30, 0, a) and tuple(t[6:, 0]) == (30, 3, 0, b)
    with pytest.raises(ValueError, match="place"):
        _plan(s, [(a, 4, [4])])
    with pytest.raises(ValueError, match="staging"):
        s.write_segments(t.ctypes.data, 1)
    assert s.length(a) == 30


def test_pages_and_slots_are_used_again():
    from nexus_b200 import _native
    s = _native.KvScheduler(8, 16, 2, 128)
    a, b = s.add(), s.add()
    _plan(s, [(a, 60, None), (b, 60, None)])
    with pytest.raises(RuntimeError):
        s.add()
    s.free(a)
    c = s.add()
    assert c == a and s.free_blocks() == 4
    p = _plan(s, [(c, 1, None), (b, 4, None)])
    assert p["segments"][0] == (1, 1, 1)
    assert _tables(s, 8)[8, 0] == 0                                  # the new owner of the slot starts at position 0


def test_config_reader():
    from nexus_b200.lm.config import ConfigError
    from nexus_b200.lm.hybrid import DeltaSpec, ParallelSpec, gugedra_config
    cfg = O.random_config(("parallel", "delta", "delta", "parallel"))
    hc = gugedra_config(cfg)
    assert [type(x.mixer) for x in hc.layers] == [ParallelSpec, DeltaSpec, DeltaSpec, ParallelSpec]
    assert [bool(x.ff) for x in hc.layers] == [True, True, False, True]
    left, right = hc.layers[0].mixer.left, hc.layers[0].mixer.right
    assert (left.window, left.rope_dims, left.softcap, left.scale) == (37, 12, 9.0, 0.21)
    assert right.channels == right.inner + 2 * right.groups * right.state
    assert (hc.layers[0].mixer.left_scale, hc.layers[0].mixer.right_scale, hc.norm_eps) == (0.7, 1.3, 1e-5)

    def broken(change):
        c = copy.deepcopy(cfg)
        change(c)
        with pytest.raises(ConfigError):
            gugedra_config(c)
    broken(lambda c: c.pop("logit_softcap"))
    broken(lambda c: c.update(surprise=1))
    broken(lambda c: c["layers"][0].update(type="other"))
    broken(lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3))
    broken(lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=13))
    broken(lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5))
    broken(lambda c: c["layers"][1]["mixer"].update(conv=0))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    broken(lambda c: c.update(layers=[]))


def test_weights_fit_the_configuration(tmp_path):
    from nexus_b200.infer import Engine, Gpt2Weights, HybridEngine, create_engine, families, load_model
    from nexus_b200.infer import EngineConfig
    from nexus_b200.interop.safetensors import save_file
    from nexus_b200.lm.config import ConfigError
    from nexus_b200.lm.hybrid import HybridWeights, gugedra_config, gugedra_tensors, random_gugedra
    cfg = O.random_config()
    w = O.random_weights(cfg)
    hc = gugedra_config(cfg)
    assert {k: tuple(v.shape) for k, v in w.items()} == gugedra_tensors(hc)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))
    got = load_model(str(tmp_path))
    assert isinstance(got, HybridWeights) and got.vocab == cfg["vocab"] and all(torch.equal(got.tensors[k], w[k]) for k in w)
    assert families()["Gugedra"].engine is HybridEngine and families()["GPT2"].engine is Engine
    assert type(create_engine(Gpt2Weights.random(1, 2, 16, 20, 32), EngineConfig(device="cpu", precision="fp32"))) is Engine
    with pytest.raises(TypeError):
        create_engine(object())
    save_file({k: v for k, v in w.items() if k != "l1.mix.b"}, str(tmp_path / "model.safetensors"))
    with pytest.raises(ConfigError, match="l1.mix.b"):
        load_model(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps({**cfg, "architecture": "Nothing"}))
    with pytest.raises(ValueError, match="unknown architecture"):
        load_model(str(tmp_path))
    r = random_gugedra(hc)
    assert {k: tuple(v.shape) for k, v in r.tensors.items()} == gugedra_tensors(hc)


def test_gpt2_wanted_places():
    """The engine the families share: logits of any places of a chunk."""
    from nexus_b200.infer import Chunk, EngineConfig, Gpt2Weights, create_engine
    w = Gpt2Weights.random(2, 2, 32, 50, 64, seed=3)
    e = create_engine(w, EngineConfig(device="cpu", precision="fp32", kv_tokens=100, block_size=16, max_seqs=2))
    assert e.total_blocks() == 7
    s, toks = e.add_sequence(), [3, 9, 27, 31, 2, 44]
    whole = e.forward([Chunk(s, toks, 6)]).clone()
    e.truncate(s, 0)
    got = e.forward([Chunk(s, toks, places=[4, 0, 5])])
    assert torch.allclose(got, whole[[4, 0, 5]], atol=1e-5)


def test_restatement_prefix_property_and_window_edge():
    """Causality of the plain model, and that its window is as wide as it says: changing the value of the first token inside
    the window moves the output, changing the one before it does not."""
    cfg = O.random_config(("parallel", "delta"))
    w = O.random_weights(cfg, seed=2)
    toks = torch.randint(0, cfg["vocab"], (50,), generator=torch.Generator().manual_seed(0)).tolist()
    full = O.forward(cfg, w, toks)
    assert torch.allclose(O.forward(cfg, w, toks[:20]), full[:20], atol=1e-9)
    q, k, v = (torch.randn(40, h, 8, dtype=torch.float64, generator=torch.Generator().manual_seed(i)) for i, h in enumerate((4, 2, 2)))
    base = O.window_attention(q, k, v, 0.4, 6.0, 11)
    for j, moved in ((29, True), (28, False)):
        v2 = v.clone()
        v2[j] += 1.0
        assert (not torch.equal(O.window_attention(q, k, v2, 0.4, 6.0, 11)[39], base[39])) == moved


def test_engine_refuses_a_cpu_device():
    from nexus_b200.infer import EngineConfig, create_engine
    from nexus_b200.lm.hybrid import HybridWeights, gugedra_config
    cfg = O.random_config()
    with pytest.raises(ValueError, match="CUDA"):
        create_engine(HybridWeights(gugedra_config(cfg), O.random_weights(cfg)), EngineConfig(device="cpu", precision="fp32"))
