"""Host side of the Lukopel decoder: configuration, weights, registry, the planning of its steps, and the plain restatement's own
consistency.  No GPU."""
import copy
import json
import math

import pytest
import torch

from oracles import lukopel as O


def _config(cfg, rows=12):
    from nexus_b200.lm.lukopel import lukopel_config
    return lukopel_config(cfg, [rows] * len(cfg["layers"]))


def test_config_reader():
    from nexus_b200.lm.config import ConfigError
    from nexus_b200.lm.hybrid import NormedAttentionSpec
    cfg = O.random_config()
    hc = _config(cfg)
    assert (hc.streams, hc.positions, hc.embed_scale, hc.norm_eps, hc.pre_norm, hc.post_norm, hc.recurrent) == (2, 400, 3.0, 1e-4, True, False, False)
    assert hc.order == [0, 1, 2, 1, 2, 3] and [x.mixer for x in hc.runs] == [hc.layers[i].mixer for i in hc.order]
    t, c, t1, c1 = (x.mixer for x in hc.layers)
    assert all(isinstance(m, NormedAttentionSpec) for m in (t, c, t1, c1))
    assert (t.heads, t.kv_heads, t.dim, t.vdim, t.scale, t.norm, t.bias, t.unit_values, t.head_scale, t.talk, t.gate, t.chunk) == (
        6, 3, 24, 20, 0.22, "head", False, True, False, True, True, 0)
    assert (t.distance.rows, t.distance.far, t.temperature.coef, t.temperature.every) == (12, 37, 0.4, 23)
    assert (c.heads, c.kv_heads, c.dim, c.vdim, c.scale, c.norm, c.bias, c.unit_values, c.head_scale, c.talk, c.gate, c.chunk) == (
        6, 2, 20, 24, 0.25, "all", True, False, True, False, False, 21)
    assert c.distance is None and c.temperature is None
    assert [(x.ff, x.act, x.ff_bias) for x in hc.layers[:3]] == [(52, "relu2", True), (44, "relu2", True), (0, "silu", False)]
    per = [3 * 44, 2 * 44, 1 * 44, 2 * 44]
    assert hc.kv_bytes_per_token(2) == 2 * sum(per[i] for i in hc.order)
    assert _config({k: v for k, v in cfg.items() if k != "loop"}).order == [0, 1, 2, 3]

    def broken(change):
        bad = copy.deepcopy(cfg)
        change(bad["layers"], bad)
        with pytest.raises(ConfigError):
            _config(bad)
    broken(lambda ls, c: c.pop("streams"))
    broken(lambda ls, c: c.update(surprise=1))
    broken(lambda ls, c: c.update(layers=[]))
    broken(lambda ls, c: c.update(streams=0))
    broken(lambda ls, c: c.update(streams=9))
    broken(lambda ls, c: c.update(max_positions=0))
    broken(lambda ls, c: c["loop"].update(stop=5))
    broken(lambda ls, c: c["loop"].update(start=4))
    broken(lambda ls, c: c["loop"].update(times=0))
    broken(lambda ls, c: ls[0]["mixer"].pop("q_temp"))
    broken(lambda ls, c: ls[0]["mixer"]["q_temp"].update(every=0))
    broken(lambda ls, c: ls[0]["mixer"].update(bias_max=6))              # not beyond the first half of 12 rows
    broken(lambda ls, c: ls[0]["mixer"].update(mask={"size": 4}))
    broken(lambda ls, c: ls[1]["mixer"]["mask"].update(size=0))
    broken(lambda ls, c: ls[1]["mixer"].update(kv_heads=4))
    broken(lambda ls, c: ls[1].update(type="attention_3"))
    broken(lambda ls, c: ls[1]["mlp"].update(kind="gated"))
    broken(lambda ls, c: ls[1]["mlp"].update(ff=0))


def test_weights_fit_the_configuration(tmp_path):
    from nexus_b200.infer import EngineConfig, HybridEngine, create_engine, families, load_model
    from nexus_b200.interop.safetensors import save_file
    from nexus_b200.lm.config import ConfigError
    from nexus_b200.lm.lukopel import lukopel_tensors, random_lukopel
    cfg = O.random_config()
    w = O.random_weights(cfg, bias_rows=[10, 0, 6, 0])
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))
    got = load_model(str(tmp_path))
    assert got.vocab == cfg["vocab"] and all(torch.equal(got.tensors[k], w[k]) for k in w)
    assert [x.mixer.distance.rows if x.mixer.distance else 0 for x in got.config.layers] == [10, 0, 6, 0]
    assert families()["Lukopel"].engine is HybridEngine
    assert {k: tuple(v.shape) for k, v in w.items()} == lukopel_tensors(got.config)
    r = random_lukopel(got.config)
    assert {k: tuple(v.shape) for k, v in r.tensors.items()} == lukopel_tensors(got.config)
    with pytest.raises(ValueError, match="CUDA"):
        create_engine(got, EngineConfig(device="cpu", precision="fp32"))
    # a layer without a feed-forward has no use for the second sublayer's tensors
    save_file({**w, "l2.norm2": torch.ones(88), "l2.hc2.in": torch.ones(2)}, str(tmp_path / "model.safetensors"))
    assert "l2.norm2" not in load_model(str(tmp_path)).tensors
    for name in ("l0.mix.talk", "l1.mix.temp", "l1.mix.o.b", "l2.hc1.mix", "pos", "l0.mlp.up.b"):
        save_file({k: v for k, v in w.items() if k != name}, str(tmp_path / "model.safetensors"))
        with pytest.raises(ConfigError, match=name.replace(".", r"\.")):
            load_model(str(tmp_path))


@pytest.mark.parametrize("rows,far", [(2, 2), (12, 37), (16, 1000), (32, 128), (64, 33)])
def test_buckets_of_distances(rows, far):
    from nexus_b200.lm.hybrid import DistanceBias
    b = DistanceBias(rows, far)
    got = [b.bucket(n) for n in range(2 * far + 5)]
    assert got == [O.bucket(n, rows, far) for n in range(2 * far + 5)]
    assert got[: rows // 2] == list(range(rows // 2)) and got[far:] == [rows - 1] * (far + 5)
    assert all(x <= y for x, y in zip(got, got[1:]))


def test_extended_bias_table():
    from nexus_b200.ops._mixers import BIAS_MARGIN, extended_bias
    bias = torch.randn((3, 9), generator=torch.Generator().manual_seed(0))
    ext = extended_bias(bias)
    assert ext.shape[1] % 4 == 0 and ext.shape[1] >= 9 + 2 * BIAS_MARGIN
    for n in (-BIAS_MARGIN, -1, 0, 1, 8, 9, 8 + BIAS_MARGIN):
        assert torch.allclose(ext[:, BIAS_MARGIN + n], bias[:, min(max(n, 0), 8)] * math.log2(math.e))


@pytest.mark.parametrize("chunk", [1, 40, 256, 300, 5000])
def test_long_segments_in_chunks(chunk):
    """Every key that a row can see has its place among the rows of kv, and chunks that fill a query block end one."""
    from nexus_b200.infer.prompt import QUERY_BLOCK, long_segments
    for segs in ([(0, 17, 0, 3), (17, 600, 0, 1)], [(5, 17, 900, 2), (22, 256, 0, 0), (300, 257, 31, 1), (600, 20, 4000, 3), (700, 700, chunk, 4)]):
        blocks, runs, kv_rows = long_segments(segs, 0, 0, chunk)
        held = {}
        for first, count, base, seq in runs:
            for k in range(count):
                assert first + k not in held
                held[first + k] = (seq, base + k)
        assert len(held) == kv_rows
        rows = set()
        for row0, count, pos0, kv0, _ in blocks:
            s = next(s for s in segs if s[0] <= row0 < s[0] + s[1])
            assert 0 < count <= QUERY_BLOCK and pos0 == s[2] + row0 - s[0]
            assert chunk < QUERY_BLOCK or pos0 // chunk == (pos0 + count - 1) // chunk
            rows.update(range(row0, row0 + count))
            for key in {pos0 // chunk * chunk, pos0, pos0 + count - 1}:
                assert (held[kv0 + key] if runs else (s[3], kv0 + key - s[0])) == (s[3], key)
        assert rows == {r for r0, n, _, _ in segs for r in range(r0, r0 + n)}


@pytest.mark.parametrize("most", [256, 300, 1000, 10 ** 6])
def test_slices_of_rows(most):
    from nexus_b200.infer.prompt import long_segments, row_slices
    blocks, _, _ = long_segments([(5, 17, 900, 2), (22, 256, 0, 0), (300, 700, 31, 1), (1000, 20, 4000, 3)], 0, 0, 0)
    got = row_slices(blocks, most)
    assert sorted(b for part, _, _ in got for b in part) == sorted(blocks)
    last = 0
    for part, row, rows in got:
        assert row >= last and rows <= max(most, 256)
        assert min(b[0] for b in part) == row and max(b[0] + b[1] for b in part) == row + rows
        assert [blocks.index(b) for b in part] == sorted(blocks.index(b) for b in part)
        last = row + rows


def _moved(cfg, w, length, j):
    """Whether the last position's logits depend on token j."""
    toks = torch.randint(0, cfg["vocab"], (length,), generator=torch.Generator().manual_seed(0)).tolist()
    other = list(toks)
    other[j] = (toks[j] + 1) % cfg["vocab"]
    return not torch.allclose(O.forward(cfg, w, other)[-1], O.forward(cfg, w, toks)[-1], atol=1e-9)


def test_restatement_views():
    cfg = O.random_config([O.chunked_layer(None, size=11)], loop=(0, 1, 1))
    w = O.random_weights(cfg, seed=2)
    assert [_moved(cfg, w, 33, j) for j in (32, 22, 21, 0)] == [True, True, False, False]
    assert [_moved(cfg, w, 34, j) for j in (33, 32)] == [True, False]
    cfg = O.random_config([O.talking_layer(None)], loop=(0, 1, 1))
    assert _moved(cfg, O.random_weights(cfg, seed=2), 60, 0)


def test_restatement_prefix_loop_and_streams():
    cfg = O.random_config()
    w = O.random_weights(cfg, seed=2)
    toks = torch.randint(0, cfg["vocab"], (30,), generator=torch.Generator().manual_seed(0)).tolist()
    full = O.forward(cfg, w, toks)
    assert torch.allclose(O.forward(cfg, w, toks[:13]), full[:13], atol=1e-9)
    # a loop is the same as its layers written out
    flat = copy.deepcopy(cfg)
    flat["layers"], flat["loop"] = [cfg["layers"][i] for i in O.layer_order(cfg)], {"start": 0, "stop": 0, "times": 1}
    out = {k: v for k, v in w.items() if k[0] != "l"}
    for at, i in enumerate(O.layer_order(cfg)):
        out.update({f"l{at}." + k.split(".", 1)[1]: v for k, v in w.items() if k.startswith(f"l{i}.")})
    assert torch.allclose(O.forward(flat, out, toks), full, atol=1e-9)
    # one stream with factors of one is a plain residual
    one = O.random_config([O.chunked_layer(None)], loop=(0, 1, 1), streams=1)
    w1 = {k: torch.ones_like(v) if ".hc" in k else v for k, v in O.random_weights(one, seed=4).items()}
    x = (w1["embed"][toks].double() * one["embedding"]["scale"] + w1["pos"][:30].double())
    p = {k[7:]: v.double() for k, v in w1.items() if k.startswith("l0.mix.")}
    x = x + O.chunked_attention(O.norm(x, w1["l0.norm1"].double(), 1e-4), p, one["layers"][0]["mixer"], 1e-4)
    assert torch.allclose(O.norm(x, w1["final.norm"].double(), 1e-4) @ w1["head"].double().T, O.forward(one, w1, toks), atol=1e-9)
