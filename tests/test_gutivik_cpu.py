"""Host side of the Gutivik decoder: configuration, weights, registry, the planning of its steps, and the plain restatement's
own consistency.  No GPU."""
import copy
import json

import pytest
import torch

from oracles import gutivik as O


def _config(cfg, rank=5):
    from nexus_b200.lm.gutivik import gutivik_config
    return gutivik_config(cfg, [rank] * len(cfg["layers"]))


def test_config_reader():
    from nexus_b200.lm.config import ConfigError
    from nexus_b200.lm.hybrid import ConvAttentionSpec, GlaSpec, LatentSpec
    cfg = O.random_config()
    hc = _config(cfg)
    a, g, c, a2, g2 = (x.mixer for x in hc.layers)
    assert isinstance(a, ConvAttentionSpec) and isinstance(g, GlaSpec) and isinstance(c, LatentSpec) and hc.recurrent
    assert (hc.pre_norm, hc.post_norm, hc.norm_offset, hc.norm_eps, hc.logit_scale, hc.logit_softcap) == (True, False, 1.0, 1e-4, 1.7, 9.0)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.conv, a.window, a.keep_first, a.rope_dims, a.rope_base, a.scale) == (
        6, 2, 24, 20, 4, 21, 5, 16, 4000.0, 0.22)
    assert a.bias and a.sink and a.mix_values and a2.mix_values and hc.first_mixing == 0
    assert (g.heads, g.dim, g.vdim, g.tau, g.rank) == (3, 24, 20, 8.0, 5)
    assert (c.heads, c.dim, c.rope_dims, c.vdim, c.q_rank, c.kv_rank, c.window, c.interleaved, c.gate) == (5, 24, 16, 20, 0, 56, 17, True, False)
    f = hc.layers[0].experts
    assert (f.experts, f.top, f.ff, f.router.groups, f.router.keep) == (6, 2, 28, 3, 2)
    assert (f.glu.limit, f.glu.slope, f.glu.offset) == (0.8, 1.702, 1.0) and hc.layers[3].experts.router.groups == 1
    assert (hc.layers[1].ff, hc.layers[1].act, hc.layers[2].ff, hc.layers[2].experts) == (44, "gelu_tanh", 0, None)
    assert hc.kv_bytes_per_token(2) == 2 * (2 * 2 * 44 + 56 + 16)

    def broken(change):
        bad = copy.deepcopy(cfg)
        change(bad["layers"], bad)
        with pytest.raises(ConfigError):
            _config(bad)
    broken(lambda ls, c: c.pop("logit_scale"))
    broken(lambda ls, c: c.update(surprise=1))
    broken(lambda ls, c: c.update(layers=[]))
    broken(lambda ls, c: ls[0]["mixer"].pop("conv"))
    broken(lambda ls, c: ls[0]["mixer"].update(conv=9))
    broken(lambda ls, c: ls[0]["mixer"].update(softcap=3.0))
    broken(lambda ls, c: ls[0]["mixer"].update(kv_heads=4))
    broken(lambda ls, c: ls[0]["mixer"]["mask"].update(size=0))
    broken(lambda ls, c: ls[0]["mixer"]["mask"].update(keep_first=-1))
    broken(lambda ls, c: ls[0]["mixer"]["rot"].update(dims=7))
    broken(lambda ls, c: ls[3]["mixer"].update(vdim=24))                  # mixes values with a layer of another size
    broken(lambda ls, c: ls[1]["mixer"].update(tau=0.0))
    broken(lambda ls, c: ls[2]["mixer"]["rot"].update(dims=8))
    broken(lambda ls, c: ls[2].update(type="delta"))
    broken(lambda ls, c: ls[1]["mlp"].update(kind="gated"))
    broken(lambda ls, c: ls[0]["mlp"]["expert"].update(limit=0.0))
    broken(lambda ls, c: ls[0]["mlp"]["router"].update(top=5))            # two groups of two hold four
    broken(lambda ls, c: ls[0]["mlp"]["router"]["groups"].update(count=4))


def test_weights_fit_the_configuration(tmp_path):
    from nexus_b200.infer import EngineConfig, HybridEngine, create_engine, families, load_model
    from nexus_b200.interop.safetensors import save_file
    from nexus_b200.lm.config import ConfigError
    from nexus_b200.lm.gutivik import gutivik_tensors, random_gutivik
    cfg = O.random_config()
    w = O.random_weights(cfg, rank=7)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))
    got = load_model(str(tmp_path))
    assert got.vocab == cfg["vocab"] and all(torch.equal(got.tensors[k], w[k]) for k in w)
    assert got.config.layers[1].mixer.rank == 7 and families()["Gutivik"].engine is HybridEngine
    assert {k: tuple(v.shape) for k, v in w.items()} == gutivik_tensors(got.config)
    r = random_gutivik(got.config)
    assert {k: tuple(v.shape) for k, v in r.tensors.items()} == gutivik_tensors(got.config)
    with pytest.raises(ValueError, match="CUDA"):
        create_engine(got, EngineConfig(device="cpu", precision="fp32"))
    for name in ("l0.mix.sink", "l4.mlp.e3.gate", "l1.mix.a2.b", "l3.mix.vmix"):
        save_file({k: v for k, v in w.items() if k != name}, str(tmp_path / "model.safetensors"))
        with pytest.raises(ConfigError, match=name.replace(".", r"\.")):
            load_model(str(tmp_path))


@pytest.mark.parametrize("window,keep", [(1, 1), (40, 6), (300, 128), (64, 400), (5000, 9)])
def test_kept_keys_of_long_segments(window, keep):
    """The kv rows of the keys a row can see, in its window and among the kept first ones, are those the runs put them in."""
    from nexus_b200.infer.prompt import long_segments
    back = window - 1
    for segs in ([(0, 17, 0, 3), (17, 600, 0, 1)], [(5, 17, 900, 2), (22, 256, 0, 0), (300, 257, 31, 1), (600, 20, 4000, 3)]):
        blocks, runs, kv_rows = long_segments(segs, window, keep)
        held = {}
        for first, count, base, seq in runs:
            for k in range(count):
                assert first + k not in held
                held[first + k] = (seq, base + k)
        assert len(held) == kv_rows
        for row0, count, pos0, kv0, kept0 in blocks:
            s = next(s for s in segs if s[0] <= row0 < s[0] + s[1])
            lo = max(0, pos0 - back)
            for key in {lo, pos0, pos0 + count - 1}:
                assert (held[kv0 + key] if runs else (s[3], kv0 + key - s[0])) == (s[3], key)
            for key in {0, min(keep, lo) - 1} if min(keep, lo) > 0 else ():
                assert (held[kept0 + key] if runs else (s[3], kept0 + key - s[0])) == (s[3], key)


def _moved(cfg, w, length, j):
    """Whether the last position's logits depend on token j."""
    toks = torch.randint(0, cfg["vocab"], (length,), generator=torch.Generator().manual_seed(0)).tolist()
    other = list(toks)
    other[j] = (toks[j] + 1) % cfg["vocab"]
    return not torch.allclose(O.forward(cfg, w, other)[-1], O.forward(cfg, w, toks)[-1], atol=1e-9)


def test_restatement_views():
    """One layer each: the window's last key through the convolution's first tap, kept keys, and a state without an edge."""
    cfg = O.random_config([O.attention_layer(None, window=11, keep=3, conv=2, v_mix=False)])
    w = O.random_weights(cfg, seed=2)
    assert [_moved(cfg, w, 40, j) for j in (39, 29, 28, 27, 10, 3, 2, 0)] == [True, True, True, False, False, False, True, True]
    cfg = O.random_config([O.latent_layer(None, window=11)])
    w = O.random_weights(cfg, seed=2)
    assert [_moved(cfg, w, 40, j) for j in (39, 29, 28, 0)] == [True, True, False, False]
    cfg = O.random_config([O.gla_layer(None, tau=16.0)])
    assert _moved(cfg, O.random_weights(cfg, seed=2), 40, 0)


def test_restatement_routing():
    """The correction picks but does not weigh; a group outside the best ones is out even where all choice scores are negative."""
    z = torch.tensor([[2.0, -1.0, 0.5, 0.4, -3.0, 3.0]], dtype=torch.float64)
    corr = torch.tensor([-2.0, -2.0, -1.0, -1.0, -2.0, -1.9], dtype=torch.float64)
    s = O.sigmoid(z)[0]
    got = O.route(z, corr, {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}})[0]
    assert [e for e, _ in got] == [2, 3] and abs(got[0][1] - s[2] / (s[2] + s[3])) < 1e-12
    assert [e for e, _ in O.route(z, corr, {"experts": 6, "top": 2})[0]] == [2, 3]
    assert [e for e, _ in O.route(z, 0 * corr, {"experts": 6, "top": 2})[0]] == [5, 0]
    assert [e for e, _ in O.route(z, 0 * corr, {"experts": 6, "top": 2, "groups": {"count": 2, "keep": 1}})[0]] == [5, 3]


def test_restatement_prefix_and_first_values():
    cfg = O.random_config()
    w = O.random_weights(cfg, seed=2)
    toks = torch.randint(0, cfg["vocab"], (30,), generator=torch.Generator().manual_seed(0)).tolist()
    full = O.forward(cfg, w, toks)
    assert torch.allclose(O.forward(cfg, w, toks[:13]), full[:13], atol=1e-9)
    for name, used in (("l0.mix.vmix", False), ("l3.mix.vmix", True)):
        other = {**w, name: w[name] + 0.5}
        assert torch.allclose(O.forward(cfg, other, toks), full, atol=1e-9) != used
