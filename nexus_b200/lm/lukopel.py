"""The Lukopel decoder: layers of attention on normed queries and keys, either causal with distance biases, heads that mix their
weights and an output gate, or within chunks; squared-relu feed-forwards; several residual streams; a range of layers that runs more
than once; learned positions.

:func:`lukopel_config` reads ``config.json``, :func:`load_lukopel` also ``model.safetensors``; the layers are the specs of
`lm.hybrid`, which `infer.hybrid.HybridEngine` runs."""
from __future__ import annotations

import json
import math
import os
from typing import Dict, Mapping, Optional, Sequence, Tuple

import torch

from .config import ConfigError
from .hybrid import (DistanceBias, HybridConfig, HybridLayer, HybridWeights, Loop, NormedAttentionSpec, QueryTemperature, _take,
                     check_tensors)

__all__ = ["lukopel_config", "lukopel_tensors", "load_lukopel", "random_lukopel"]


def _attention(obj: dict, where: str, bias_rows: int) -> NormedAttentionSpec:
    heads, kv, dim, vdim, scale, far, temp = _take(obj, where, ("heads", "kv_heads", "dim", "vdim", "scale", "bias_max", "q_temp"))
    coef, every = _take(temp, where + ".q_temp", ("coef", "every"))
    return NormedAttentionSpec(heads, kv, dim, vdim, float(scale), unit_values=True, temperature=QueryTemperature(float(coef), every),
                               distance=DistanceBias(bias_rows, far), talk=True, gate=True)


def _chunked(obj: dict, where: str) -> NormedAttentionSpec:
    heads, kv, dim, vdim, scale, mask = _take(obj, where, ("heads", "kv_heads", "dim", "vdim", "scale", "mask"))
    (size,) = _take(mask, where + ".mask", ("size",))
    if not isinstance(size, int) or isinstance(size, bool) or size < 1:
        raise ConfigError(f"{where}.mask: the size must be a positive integer")
    return NormedAttentionSpec(heads, kv, dim, vdim, float(scale), norm="all", bias=True, head_scale=True, chunk=size)


def _feed_forward(obj: Optional[dict], where: str) -> dict:
    """Keyword arguments of the layer."""
    if obj is None:
        return {}
    kind, ff = _take(obj, where, ("kind", "ff"))
    if kind != "dense" or not isinstance(ff, int) or ff < 1:
        raise ConfigError(f"{where}: a dense feed-forward is expected")
    return {"ff": ff, "act": "relu2", "ff_bias": True}


def lukopel_config(obj: dict, bias_rows: Sequence[int] = ()) -> HybridConfig:
    """``config.json`` of a Lukopel model.  The rows of the bias tables are stated by the tensors only: ``bias_rows`` has one entry per
    layer (used for those with a table)."""
    _, embedding, layers, loop, positions, norm, streams, vocab, width = _take(
        {"loop": None, **obj}, "config",
        ("architecture", "embedding", "layers", "loop", "max_positions", "norm", "streams", "vocab", "width"))
    (scale,) = _take(embedding, "embedding", ("scale",))
    (eps,) = _take(norm, "norm", ("eps",))
    for name, v in (("streams", streams), ("max_positions", positions)):
        if not isinstance(v, int) or isinstance(v, bool) or v < 1:
            raise ConfigError(f"{name} must be a positive integer")
    out = []
    for i, layer in enumerate(layers):
        kind, mix, mlp = _take({"mlp": None, **layer}, f"layers[{i}]", ("type", "mixer", "mlp"))
        where = f"layers[{i}].mixer"
        if kind == "attention":
            spec = _attention(mix, where, bias_rows[i] if i < len(bias_rows) else 32)
        elif kind == "attention_2":
            spec = _chunked(mix, where)
        else:
            raise ConfigError(f"layers[{i}]: unknown mixer {kind!r}")
        out.append(HybridLayer(spec, **_feed_forward(mlp, f"layers[{i}].mlp")))
    return HybridConfig(vocab, width, out, float(eps), name="Lukopel", post_norm=False, embed_scale=float(scale), streams=streams,
                        loop=None if loop is None else Loop(*_take(loop, "loop", ("start", "stop", "times"))), positions=positions)


def bias_rows(layers: int, tensors: Mapping[str, torch.Tensor]) -> list:
    """Rows of every layer's bias table (2 where there is none)."""
    return [tensors[f"l{i}.mix.rel"].shape[0] if f"l{i}.mix.rel" in tensors else 2 for i in range(layers)]


def lukopel_tensors(cfg: HybridConfig) -> Dict[str, Tuple[int, ...]]:
    """Name and shape of every tensor."""
    W, S = cfg.width, cfg.streams
    t: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, W), "pos": (cfg.positions, W), "final.norm": (W,), "head": (cfg.vocab, W)}
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        q, k, v = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
        t.update({p + "mix.q": (q, W), p + "mix.k": (k, W), p + "mix.v": (v, W), p + "mix.o": (W, m.heads * m.vdim)})
        if m.bias:
            t.update({p + "mix.q.b": (q,), p + "mix.k.b": (k,), p + "mix.v.b": (v,), p + "mix.o.b": (W,)})
        each = m.norm == "head"
        t[p + "mix.q.norm"], t[p + "mix.k.norm"] = (m.dim if each else q,), (m.dim if each else k,)
        for used, name, shape in ((m.head_scale, "temp", (m.heads,)), (m.talk, "talk", (m.heads, m.heads)), (m.gate, "g", (m.heads, W)),
                                  (m.distance, "rel", (m.distance.rows if m.distance else 0, m.heads))):
            if used:
                t[p + "mix." + name] = shape
        if layer.ff:
            t.update({p + "mlp.up": (layer.ff, W), p + "mlp.up.b": (layer.ff,), p + "mlp.down": (W, layer.ff), p + "mlp.down.b": (W,)})
        for n in ("1", "2")[: 2 if layer.ff else 1]:
            t[p + "norm" + n] = (W,)
            t.update({p + f"hc{n}.in": (S,), p + f"hc{n}.out": (S,), p + f"hc{n}.mix": (S, S)})
    return t


def check_lukopel(cfg: HybridConfig, tensors: Dict[str, torch.Tensor]) -> None:
    check_tensors(cfg, tensors, lukopel_tensors(cfg))


def load_lukopel(folder: str) -> HybridWeights:
    """A folder with ``config.json`` and ``model.safetensors``."""
    from ..interop.safetensors import load_file
    with open(os.path.join(folder, "config.json")) as f:
        obj = json.load(f)
    tensors = load_file(os.path.join(folder, "model.safetensors"))
    cfg = lukopel_config(obj, bias_rows(len(obj.get("layers", ())), tensors))
    for i, layer in enumerate(cfg.layers):      # a layer without a feed-forward has no second sublayer
        if not layer.ff:
            for name in ("norm2", "hc2.in", "hc2.out", "hc2.mix"):
                tensors.pop(f"l{i}.{name}", None)
    check_lukopel(cfg, tensors)
    return HybridWeights(cfg, tensors)


def random_lukopel(cfg: HybridConfig, seed: int = 0) -> HybridWeights:
    """Random BF16 weights of a configuration (benchmarks, examples): unit-variance activations, streams and heads that mix."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in lukopel_tensors(cfg).items():
        leaf = n.split(".", 1)[-1] if n[0] == "l" else n
        if "norm" in leaf or leaf == "mix.temp" or leaf.endswith(".out"):
            v = torch.ones(shape)
        elif leaf.startswith("hc") and leaf.endswith(".in"):
            v = torch.full(shape, 1.0 / shape[0])
        elif leaf.startswith("hc"):
            v = 0.8 * torch.eye(shape[0]) + 0.2 / shape[0]
        elif leaf == "mix.talk":
            v = 0.8 * torch.eye(shape[0]) + 0.2 * torch.randn(shape, generator=g) / math.sqrt(shape[0])
        elif leaf.endswith(".b"):
            v = 0.1 * torch.randn(shape, generator=g)
        elif leaf == "embed":
            v = torch.randn(shape, generator=g) / cfg.embed_scale
        elif leaf in ("pos", "mix.rel"):
            v = 0.5 * torch.randn(shape, generator=g)
        else:
            v = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[n] = v.to(torch.bfloat16)
    return HybridWeights(cfg, out)
