"""The Gutivik decoder: latent attention, gated linear attention and attention over convolved projections in any order, dense
gated feed-forwards and experts behind a sigmoid router, norms on the inputs of the sublayers, scaled and soft-capped logits.

:func:`gutivik_config` reads ``config.json``, :func:`load_gutivik` also ``model.safetensors``; the layers are the specs of
`lm.hybrid`, which `infer.hybrid.HybridEngine` runs."""
from __future__ import annotations

import json
import math
import os
from typing import Dict, Mapping, Optional, Sequence, Tuple

import torch

from .config import ConfigError
from .hybrid import (ClampedGlu, ConvAttentionSpec, ExpertsSpec, GlaSpec, HybridConfig, HybridLayer, HybridWeights, LatentSpec,
                     RouterSpec, _take, check_tensors)

__all__ = ["gutivik_config", "gutivik_tensors", "load_gutivik", "random_gutivik"]


def _window(mask: dict, where: str) -> int:
    size = mask.get("size")
    if not isinstance(size, int) or isinstance(size, bool) or size < 1:
        raise ConfigError(f"{where}.mask: the size must be a positive integer")
    return size


def _latent(obj: dict, where: str) -> LatentSpec:
    heads, dim, rot_dim, vdim, rank, scale, mask, rot = _take(
        obj, where, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "mask", "rot"))
    _take(mask, where + ".mask", ("size",))
    base, dims = _take(rot, where + ".rot", ("base", "dims"))
    if dims != rot_dim:
        raise ConfigError(f"{where}: rot.dims must equal rot_dim")
    return LatentSpec(heads, dim, rot_dim, vdim, 0, rank, float(scale), _window(mask, where), float(base), interleaved=True, gate=False)


def _attention(obj: dict, where: str) -> ConvAttentionSpec:
    heads, kv, dim, vdim, conv, scale, mask, rot, mix = _take(
        {"v_mix": False, **obj}, where, ("heads", "kv_heads", "dim", "vdim", "conv", "scale", "mask", "rot", "v_mix"))
    mask = {"keep_first": 0, **mask}
    _take(mask, where + ".mask", ("size", "keep_first"))
    base, dims = _take(rot, where + ".rot", ("base", "dims"))
    return ConvAttentionSpec(heads, kv, dim, vdim, float(scale), 0.0, _window(mask, where), dims, float(base), conv=conv,
                             keep_first=int(mask["keep_first"]), mix_values=bool(mix))


def _feed_forward(obj: Optional[dict], where: str) -> dict:
    """Keyword arguments of the layer."""
    if obj is None:
        return {}
    if not isinstance(obj, dict) or obj.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"{where}: a dense feed-forward or one of experts is expected")
    if obj["kind"] == "dense":
        _, ff = _take(obj, where, ("kind", "ff"))
        if not isinstance(ff, int) or ff < 1:
            raise ConfigError(f"{where}.ff must be a positive integer")
        return {"ff": ff, "act": "gelu_tanh"}
    _, expert, router = _take(obj, where, ("kind", "expert", "router"))
    ff, limit = _take(expert, where + ".expert", ("ff", "limit"))
    experts, top, groups = _take({"groups": None, **router}, where + ".router", ("experts", "top", "groups"))
    spec = RouterSpec() if groups is None else RouterSpec(*_take(groups, where + ".router.groups", ("count", "keep")))
    return {"experts": ExpertsSpec(experts, top, ff, router=spec, glu=ClampedGlu(float(limit)))}


def gutivik_config(obj: dict, decay_ranks: Sequence[int] = ()) -> HybridConfig:
    """``config.json`` of a Gutivik model.  The rank of the decay projections is stated by the tensors only: ``decay_ranks`` has
    one entry per layer (used for the gated linear ones)."""
    _, layers, scale, cap, norm, vocab, width = _take(
        obj, "config", ("architecture", "layers", "logit_scale", "logit_softcap", "norm", "vocab", "width"))
    (eps,) = _take(norm, "norm", ("eps",))
    out = []
    for i, layer in enumerate(layers):
        kind, mix, mlp = _take({"mlp": None, **layer}, f"layers[{i}]", ("type", "mixer", "mlp"))
        where = f"layers[{i}].mixer"
        if kind == "latent_attention":
            spec = _latent(mix, where)
        elif kind == "attention":
            spec = _attention(mix, where)
        elif kind == "gla":
            heads, dim, vdim, tau = _take(mix, where, ("heads", "dim", "vdim", "tau"))
            spec = GlaSpec(heads, dim, vdim, float(tau), decay_ranks[i] if i < len(decay_ranks) else 16)
        else:
            raise ConfigError(f"layers[{i}]: unknown mixer {kind!r}")
        out.append(HybridLayer(spec, **_feed_forward(mlp, f"layers[{i}].mlp")))
    return HybridConfig(vocab, width, out, float(eps), logit_softcap=float(cap), name="Gutivik", post_norm=False, norm_offset=1.0,
                        logit_scale=float(scale))


def decay_ranks(layers: int, tensors: Mapping[str, torch.Tensor]) -> list:
    """Rows of every layer's first decay projection (1 where there is none)."""
    return [tensors[f"l{i}.mix.a1"].shape[0] if f"l{i}.mix.a1" in tensors else 1 for i in range(layers)]


def gutivik_tensors(cfg: HybridConfig) -> Dict[str, Tuple[int, ...]]:
    """Name and shape of every tensor."""
    W = cfg.width
    t: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, W), "final.norm": (W,), "head": (cfg.vocab, W)}
    for i, layer in enumerate(cfg.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.experts
        t[p + "norm1"] = (W,)
        if isinstance(m, LatentSpec):
            t.update({p + "mix.q": (m.heads * (m.dim + m.rope_dims), W), p + "mix.dkv": (m.kv_rank + m.rope_dims, W),
                      p + "mix.dkv.norm": (m.kv_rank,), p + "mix.uk": (m.heads * m.dim, m.kv_rank),
                      p + "mix.uv": (m.heads * m.vdim, m.kv_rank), p + "mix.o": (W, m.heads * m.vdim)})
        elif isinstance(m, ConvAttentionSpec):
            for n, size in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                t[p + "mix." + n], t[p + f"mix.{n}.b"], t[p + f"mix.{n}.conv"] = (size, W), (size,), (size, m.conv)
            t[p + "mix.sink"], t[p + "mix.o"] = (m.heads,), (W, m.heads * m.vdim)
            if m.mix_values:
                t[p + "mix.vmix"] = ()
        else:
            qk, v = m.heads * m.dim, m.heads * m.vdim
            t.update({p + "mix.q": (qk, W), p + "mix.k": (qk, W), p + "mix.v": (v, W), p + "mix.g": (v, W), p + "mix.o": (W, v),
                      p + "mix.norm": (m.vdim,), p + "mix.a1": (m.rank, W), p + "mix.a2": (qk, m.rank), p + "mix.a2.b": (qk,)})
        if layer.ff or f is not None:
            t[p + "norm2"] = (W,)
        if layer.ff:
            t[p + "mlp.gate"] = t[p + "mlp.up"] = (layer.ff, W)
            t[p + "mlp.down"] = (W, layer.ff)
        if f is not None:
            for e in range(f.experts):
                t[p + f"mlp.e{e}.gate"] = t[p + f"mlp.e{e}.up"] = (f.ff, W)
                t[p + f"mlp.e{e}.down"] = (W, f.ff)
            t[p + "mlp.router"], t[p + "mlp.correction"] = (f.experts, W), (f.experts,)
    return t


def check_gutivik(cfg: HybridConfig, tensors: Dict[str, torch.Tensor]) -> None:
    check_tensors(cfg, tensors, gutivik_tensors(cfg))


def load_gutivik(folder: str) -> HybridWeights:
    """A folder with ``config.json`` and ``model.safetensors``."""
    from ..interop.safetensors import load_file
    with open(os.path.join(folder, "config.json")) as f:
        obj = json.load(f)
    tensors = load_file(os.path.join(folder, "model.safetensors"))
    cfg = gutivik_config(obj, decay_ranks(len(obj.get("layers", ())), tensors))
    for i, layer in enumerate(cfg.layers):      # a layer that does not mix values has no use for the factor
        if isinstance(layer.mixer, ConvAttentionSpec) and not layer.mixer.mix_values:
            tensors.pop(f"l{i}.mix.vmix", None)
    check_gutivik(cfg, tensors)
    return HybridWeights(cfg, tensors)


def random_gutivik(cfg: HybridConfig, seed: int = 0) -> HybridWeights:
    """Random BF16 weights of a configuration (benchmarks, examples): unit-variance activations, decays spread over short and
    long memories."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in gutivik_tensors(cfg).items():
        leaf = n.split(".", 2)[-1] if n[0] == "l" else n
        if leaf.endswith("dkv.norm") or leaf == "mix.norm":
            v = torch.ones(shape)
        elif "norm" in leaf or leaf.endswith(".correction") or leaf == "sink":
            v = 0.1 * torch.randn(shape, generator=g)
        elif leaf.endswith("a2.b"):
            v = torch.linspace(-2.0, 6.0, shape[0])
        elif leaf.endswith("vmix"):
            v = torch.full(shape, 0.5)
        elif leaf.endswith(".b"):
            v = 0.1 * torch.randn(shape, generator=g)
        elif leaf == "embed":
            v = torch.randn(shape, generator=g)
        else:
            v = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[n] = v.to(torch.bfloat16)
    return HybridWeights(cfg, out)
