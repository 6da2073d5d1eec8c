"""Host side of the Makuzen decoder: configuration, weights, registry, the planning of its steps, and the plain restatement's
own consistency.  No GPU."""
import copy
import json
import math

import pytest
import torch

from oracles import makuzen as O


def test_config_reader():
    from nexus_b200.lm.config import ConfigError
    from nexus_b200.lm.hybrid import LatentSpec
    from nexus_b200.lm.makuzen import makuzen_config
    cfg = O.random_config([O.random_layer(), O.random_layer(mlp=False, window=9), O.random_layer(scaling=None, top=1, base=50.0)])
    hc = makuzen_config(cfg)
    a, b, c = (x.mixer for x in hc.layers)
    assert all(isinstance(m, LatentSpec) for m in (a, b, c)) and hc.pre_norm is False and not hc.recurrent
    assert (hc.embed_scale, hc.residual_mult, hc.norm_eps) == (2.5, 0.45, 1e-4)
    assert (a.heads, a.dim, a.rope_dims, a.vdim, a.q_rank, a.kv_rank, a.window, b.window) == (5, 24, 16, 20, 44, 56, 19, 9)
    assert (a.rope_scaling.type, a.rope_scaling.factor, a.rope_scaling.beta_fast, a.rope_scaling.beta_slow) == ("yarn", 4.0, 8.0, 0.5)
    assert c.rope_scaling is None and c.rope_base == 50.0
    f = hc.layers[0].experts
    assert (f.experts, f.top, f.ff, f.shared) == (6, 2, 28, 36) and hc.layers[1].experts is None and hc.layers[2].experts.top == 1
    assert hc.kv_bytes_per_token(2) == 3 * (56 + 16) * 2

    def broken(change):
        bad = copy.deepcopy(cfg)
        change(bad)
        with pytest.raises(ConfigError):
            makuzen_config(bad)
    mix = ["layers", 0, "mixer"]

    def at(c, path):
        for p in path:
            c = c[p]
        return c
    broken(lambda c: c.pop("residual_mult"))
    broken(lambda c: c.update(surprise=1))
    broken(lambda c: at(c, mix).update(softcap=3.0))
    broken(lambda c: at(c, mix).pop("q_rank"))
    broken(lambda c: at(c, mix)["rot"].update(dims=8))
    broken(lambda c: at(c, mix).update(rot_dim=7) or at(c, mix)["rot"].update(dims=7))
    broken(lambda c: at(c, mix)["rot"]["scaling"].pop("slow"))
    broken(lambda c: at(c, mix)["mask"].update(size=0))
    broken(lambda c: c["layers"][0].update(type="delta"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=7))
    broken(lambda c: c.update(layers=[]))


def test_weights_fit_the_configuration(tmp_path):
    from nexus_b200.infer import HybridEngine, families, load_model
    from nexus_b200.interop.safetensors import save_file
    from nexus_b200.lm.config import ConfigError
    from nexus_b200.lm.makuzen import makuzen_config, makuzen_tensors, random_makuzen
    cfg = O.random_config([O.random_layer(), O.random_layer(mlp=False)])
    w = O.random_weights(cfg)
    hc = makuzen_config(cfg)
    assert {k: tuple(v.shape) for k, v in w.items()} == makuzen_tensors(hc)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))
    got = load_model(str(tmp_path))
    assert got.vocab == cfg["vocab"] and all(torch.equal(got.tensors[k], w[k]) for k in w)
    assert got.tensors["l0.mlp.table"].dtype == torch.int32 and families()["Makuzen"].engine is HybridEngine
    save_file({k: v for k, v in w.items() if k != "l0.mix.g"}, str(tmp_path / "model.safetensors"))
    with pytest.raises(ConfigError, match="l0.mix.g"):
        load_model(str(tmp_path))
    far = dict(w)
    far["l0.mlp.table"] = w["l0.mlp.table"].clone()
    far["l0.mlp.table"][3, 1] = 6
    save_file(far, str(tmp_path / "model.safetensors"))
    with pytest.raises(ConfigError, match="table"):
        load_model(str(tmp_path))
    r = random_makuzen(hc)
    assert {k: tuple(v.shape) for k, v in r.tensors.items()} == makuzen_tensors(hc)
    table = r.tensors["l0.mlp.table"]
    assert all(len(set(row)) == 2 for row in table.tolist())


def test_engine_refuses_what_it_does_not_have():
    from nexus_b200.infer import EngineConfig, create_engine
    from nexus_b200.lm.hybrid import HybridWeights
    from nexus_b200.lm.makuzen import makuzen_config
    cfg = O.random_config([O.random_layer()])
    with pytest.raises(ValueError, match="CUDA"):
        create_engine(HybridWeights(makuzen_config(cfg), O.random_weights(cfg)), EngineConfig(device="cpu", precision="fp32"))


def test_yarn_frequencies():
    """The engine's table against the restatement, with the ramp inside, empty, and past the last pair."""
    from nexus_b200.lm.config import RopeScaling
    from nexus_b200.lm.rope import rope_inv_freq
    for dims, base, factor, original, fast, slow in ((32, 1e4, 8.0, 512, 32.0, 1.0), (16, 50.0, 2.0, 64, 8.0, 0.5), (8, 1e6, 4.0, 4096, 2.0, 2.0),
                                                     (20, 300.0, 3.0, 6, 4.0, 2.0), (12, 9.0, 16.0, 100000, 0.25, 0.001)):
        sc = {"factor": factor, "original": original, "fast": fast, "slow": slow}
        want, mul = O.yarn_frequencies(dims, base, sc)
        got, gmul = rope_inv_freq(dims, base, RopeScaling("yarn", factor, original, beta_fast=fast, beta_slow=slow), 4096, dtype=torch.float64)
        assert torch.allclose(got, torch.tensor(want, dtype=torch.float64), rtol=1e-12) and math.isclose(mul, gmul, rel_tol=1e-12)
    plain, one = O.yarn_frequencies(8, 100.0, None)
    assert one == 1.0 and plain[0] == 1.0 and math.isclose(plain[2], 100.0 ** -0.5)


@pytest.mark.parametrize("window", [0, 1, 40, 300, 5000])
def test_blocks_and_runs_of_long_segments(window):
    """Every query row is in one block; the kv row of every key a row can see is the one the runs put it in."""
    from nexus_b200.infer.prompt import QUERY_BLOCK, long_segments
    back = window - 1 if window else 10 ** 6
    for segs in ([(0, 17, 0, 3), (17, 600, 0, 1)], [(5, 17, 900, 2), (22, 256, 0, 0), (300, 257, 31, 1)]):
        blocks, runs, kv_rows = long_segments(segs, window)
        rows = sorted(r for b in blocks for r in range(b[0], b[0] + b[1]))
        assert rows == sorted(r for s in segs for r in range(s[0], s[0] + s[1]))
        assert all(1 <= b[1] <= QUERY_BLOCK for b in blocks)
        keys = [min(b[2], back) + b[1] for b in blocks]
        assert keys == sorted(keys, reverse=True)
        held = {}
        for first, count, base, seq in runs:
            for k in range(count):
                assert first + k not in held
                held[first + k] = (seq, base + k)
        assert len(held) == kv_rows and (kv_rows > 0) == any(s[2] > 0 for s in segs)
        for row0, count, pos0, kv0, kept0 in blocks:
            s = next(s for s in segs if s[0] <= row0 < s[0] + s[1])
            assert pos0 == s[2] + row0 - s[0] and kept0 == kv0
            for pos in (pos0, pos0 + count - 1):
                for key in {max(0, pos - back), pos}:
                    if runs:
                        assert held[kv0 + key] == (s[3], key)
                    else:
                        assert kv0 + key == s[0] + key


def test_slots_bound():
    from nexus_b200.ops._experts import table_slots
    g = torch.Generator().manual_seed(0)
    for n, top, experts, align in ((1, 1, 1, 128), (7, 3, 64, 128), (64, 4, 32, 1), (300, 2, 5, 32), (1000, 8, 9, 256)):
        cap = table_slots(n * top, experts, align)
        assert cap % align == 0
        for _ in range(20):
            skew = torch.rand(experts, generator=g) ** 8
            counts = torch.multinomial(skew.expand(n, -1), min(top, experts), generator=g).flatten().bincount(minlength=experts)
            assert sum(-(-int(c) // align) * align for c in counts) <= cap


def test_restatement_window_edge_and_prefix():
    cfg = O.random_config([O.random_layer(window=11)])
    w = O.random_weights(cfg, seed=2)
    toks = torch.randint(0, cfg["vocab"], (40,), generator=torch.Generator().manual_seed(0)).tolist()
    full = O.forward(cfg, w, toks)
    assert torch.allclose(O.forward(cfg, w, toks[:20]), full[:20], atol=1e-9)
    for j, moved in ((29, True), (28, False)):         # one layer: position 39 sees 29 .. 39
        other = list(toks)
        other[j] = (toks[j] + 1) % cfg["vocab"]
        assert (not torch.allclose(O.forward(cfg, w, other)[39], full[39], atol=1e-9)) == moved
