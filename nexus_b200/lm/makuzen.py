"""The Makuzen decoder: latent attention with a sliding window and a gate per head, experts chosen by token id beside a
gated shared expert, RMS norms on the outputs of the sublayers only.

:func:`makuzen_config` reads ``config.json``, :func:`load_makuzen` also ``model.safetensors``; the layers are the specs of
`lm.hybrid`, which `infer.hybrid.HybridEngine` runs."""
from __future__ import annotations

import json
import math
import os
from typing import Dict, Optional, Tuple

import torch

from .config import ConfigError, RopeScaling
from .hybrid import ExpertsSpec, HybridConfig, HybridLayer, HybridWeights, LatentSpec, _take, check_tensors

__all__ = ["makuzen_config", "makuzen_tensors", "load_makuzen", "random_makuzen"]


def _scaling(obj: Optional[dict], where: str) -> Optional[RopeScaling]:
    if obj is None:
        return None
    factor, original, fast, slow = _take(obj, where, ("factor", "original", "fast", "slow"))
    if factor <= 0 or original <= 0 or fast <= 0 or slow <= 0:
        raise ConfigError(f"{where}: the constants must be positive")
    return RopeScaling("yarn", float(factor), original, beta_fast=float(fast), beta_slow=float(slow))


def _latent(obj: dict, where: str) -> LatentSpec:
    heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mask, rot = _take(
        obj, where, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "mask", "rot"))
    (size,) = _take(mask, where + ".mask", ("size",))
    if not isinstance(size, int) or size < 1:
        raise ConfigError(f"{where}.mask: the size must be a positive integer")
    base, dims, scaling = _take({"scaling": None, **rot}, where + ".rot", ("base", "dims", "scaling"))
    if dims != rot_dim:
        raise ConfigError(f"{where}: rot.dims must equal rot_dim")
    return LatentSpec(heads, dim, rot_dim, vdim, q_rank, kv_rank, float(scale), size, float(base),
                      _scaling(scaling, where + ".rot.scaling"))


def _experts(obj: Optional[dict], where: str) -> Optional[ExpertsSpec]:
    if obj is None:
        return None
    kind, expert, router, shared = _take({"shared": None, **obj}, where, ("kind", "expert", "router", "shared"))
    if kind != "moe":
        raise ConfigError(f"{where}: a feed-forward of experts is expected")
    (ff,) = _take(expert, where + ".expert", ("ff",))
    experts, top = _take(router, where + ".router", ("experts", "top"))
    return ExpertsSpec(experts, top, ff, 0 if shared is None else _take(shared, where + ".shared", ("ff",))[0])


def makuzen_config(obj: dict) -> HybridConfig:
    """``config.json`` of a Makuzen model."""
    _, embedding, layers, norm, mult, vocab, width = _take(
        obj, "config", ("architecture", "embedding", "layers", "norm", "residual_mult", "vocab", "width"))
    (eps,), (scale,) = _take(norm, "norm", ("eps",)), _take(embedding, "embedding", ("scale",))
    out = []
    for i, layer in enumerate(layers):
        kind, mix, mlp = _take(layer, f"layers[{i}]", ("type", "mixer", "mlp"))
        if kind != "latent_attention":
            raise ConfigError(f"layers[{i}]: unknown mixer {kind!r}")
        out.append(HybridLayer(_latent(mix, f"layers[{i}].mixer"), experts=_experts(mlp, f"layers[{i}].mlp")))
    return HybridConfig(vocab, width, out, float(eps), name="Makuzen", pre_norm=False, embed_scale=float(scale),
                        residual_mult=float(mult))


def makuzen_tensors(cfg: HybridConfig) -> Dict[str, Tuple[int, ...]]:
    """Name and shape of every tensor."""
    W = cfg.width
    t: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, W), "final.norm": (W,), "head": (cfg.vocab, W)}
    for i, layer in enumerate(cfg.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.experts
        t.update({p + "norm1": (W,), p + "mix.dq": (m.q_rank, W), p + "mix.dq.norm": (m.q_rank,),
                  p + "mix.uq": (m.heads * (m.dim + m.rope_dims), m.q_rank), p + "mix.dkv": (m.kv_rank + m.rope_dims, W),
                  p + "mix.dkv.norm": (m.kv_rank,), p + "mix.uk": (m.heads * m.dim, m.kv_rank),
                  p + "mix.uv": (m.heads * m.vdim, m.kv_rank), p + "mix.g": (m.heads, W), p + "mix.o": (W, m.heads * m.vdim)})
        if f is not None:
            t[p + "norm2"] = (W,)
            for e in range(f.experts):
                t[p + f"mlp.e{e}.up"], t[p + f"mlp.e{e}.down"] = (f.ff, W), (W, f.ff)
            t[p + "mlp.table"] = (cfg.vocab, f.top)
            if f.shared:
                t[p + "mlp.shared.up"], t[p + "mlp.shared.down"], t[p + "mlp.shared.sg"] = (f.shared, W), (W, f.shared), (1, W)
    return t


def check_makuzen(cfg: HybridConfig, tensors: Dict[str, torch.Tensor]) -> None:
    check_tensors(cfg, tensors, makuzen_tensors(cfg))
    for i, layer in enumerate(cfg.layers):
        if layer.experts is not None:
            table = tensors[f"l{i}.mlp.table"]
            if table.is_floating_point() or int(table.min()) < 0 or int(table.max()) >= layer.experts.experts:
                raise ConfigError(f"l{i}.mlp.table: entries must be integers from 0 to {layer.experts.experts - 1}")


def load_makuzen(folder: str) -> HybridWeights:
    """A folder with ``config.json`` and ``model.safetensors``."""
    from ..interop.safetensors import load_file
    with open(os.path.join(folder, "config.json")) as f:
        cfg = makuzen_config(json.load(f))
    tensors = load_file(os.path.join(folder, "model.safetensors"))
    check_makuzen(cfg, tensors)
    return HybridWeights(cfg, tensors)


def random_makuzen(cfg: HybridConfig, seed: int = 0) -> HybridWeights:
    """Random BF16 weights of a configuration (benchmarks, examples); the tables draw every token's experts uniformly."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in makuzen_tensors(cfg).items():
        leaf = n.rsplit(".", 1)[-1]
        if leaf == "table":
            f = cfg.layers[int(n[1: n.index(".")])].experts
            out[n] = torch.rand((shape[0], f.experts), generator=g).topk(f.top, -1).indices.to(torch.int32)
        elif leaf.startswith("norm"):
            out[n] = torch.ones(shape, dtype=torch.bfloat16)
        else:
            out[n] = (torch.randn(shape, generator=g) / (1.0 if leaf == "embed" else math.sqrt(shape[-1]))).to(torch.bfloat16)
    return HybridWeights(cfg, out)
