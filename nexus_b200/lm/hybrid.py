"""Decoders whose layers differ from one another: the layer list, the mixers' sizes and constants, and the weights.

A model is an ordered list of :class:`HybridLayer`; each has one mixer - :class:`AttentionSpec` and :class:`SsdSpec` side
by side (:class:`ParallelSpec`), :class:`ConvAttentionSpec`, :class:`NormedAttentionSpec`, :class:`DeltaSpec`, :class:`GlaSpec` or
:class:`LatentSpec` - and optionally a feed-forward, gated, plain or of experts (:class:`ExpertsSpec`).  A range of layers may run
several times (:class:`Loop`), and the residual may be several streams that every sublayer mixes.  The engine (`infer.hybrid.HybridEngine`) builds its cache, its state slots and its
kernels' arguments from these specs and reads no size from anywhere else, so another order of layers or another
combination of constants is another configuration, not another class.

`Gugedra` is one design that uses them: RMS norms before and after every sublayer, a sliding-window soft-capped
attention branch beside a Mamba-2 branch in some layers, the gated delta rule in the others, a per-layer token input at
the end of every layer and soft-capped logits.  :func:`gugedra_config` reads its ``config.json``, and
:func:`load_gugedra` its ``model.safetensors``.  `Makuzen` (`lm.makuzen`) and
`Gutivik` (`lm.gutivik`) and `Lukopel` (`lm.lukopel`) are others.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple, Union

import torch

from .config import ConfigError, RopeScaling

__all__ = ["AttentionSpec", "ConvAttentionSpec", "DistanceBias", "QueryTemperature", "NormedAttentionSpec", "Loop", "SsdSpec", "ParallelSpec", "DeltaSpec", "GlaSpec", "LatentSpec", "RouterSpec",
           "ClampedGlu", "ExpertsSpec", "HybridLayer", "HybridConfig", "HybridWeights", "gugedra_config", "gugedra_tensors", "load_gugedra", "random_gugedra"]


def _positive(obj, *names) -> None:
    for n in names:
        v = getattr(obj, n)
        if not isinstance(v, int) or isinstance(v, bool) or v < 1:
            raise ConfigError(f"{type(obj).__name__}.{n} must be a positive integer, not {v!r}")


@dataclass(frozen=True)
class AttentionSpec:
    """Causal softmax attention; query head h reads KV head h // (heads / kv_heads)."""
    heads: int
    kv_heads: int
    dim: int                 # query / key size of a head
    vdim: int                # value size of a head
    scale: float
    softcap: float = 0.0     # > 0: score = softcap * tanh(score / softcap)
    window: int = 0          # > 0: a token sees itself and the window - 1 tokens before it
    rope_dims: int = 0       # leading dimensions of a head that rotate (rotate-half pairing)
    rope_base: float = 10000.0

    def __post_init__(self):
        _positive(self, "heads", "kv_heads", "dim", "vdim")
        if self.heads % self.kv_heads:
            raise ConfigError("attention: heads must be a multiple of kv_heads")
        if self.rope_dims % 2 or not 0 <= self.rope_dims <= self.dim:
            raise ConfigError("attention: the rotary dimensions must be even and at most the head size")
        if self.window < 0 or self.softcap < 0:
            raise ConfigError("attention: window and softcap cannot be negative")


@dataclass(frozen=True)
class ConvAttentionSpec(AttentionSpec):
    """Attention whose projections go through a short causal convolution before the rotation (of neighbouring pairs).  The first
    ``keep_first`` keys stay visible behind a window."""
    conv: int = 1            # taps of the short convolution
    keep_first: int = 0
    bias: bool = True        # on the projections of q, k and v
    sink: bool = True        # a learned score per head that counts in the softmax denominator only
    mix_values: bool = False     # values are mixed with those of the first layer that has this set

    def __post_init__(self):
        super().__post_init__()
        _positive(self, "conv")
        if self.conv > 8:
            raise ConfigError("attention: the convolution kernel has at most 8 taps")
        if self.keep_first < 0:
            raise ConfigError("attention: keep_first cannot be negative")


@dataclass(frozen=True)
class DistanceBias:
    """A learned score per head and bucket of the distance between query and key: ``rows`` buckets, one for each distance in the
    first half, logarithmic from there to distance ``far``, the last one for everything beyond."""
    rows: int
    far: int

    def __post_init__(self):
        _positive(self, "rows", "far")
        if self.far <= self.rows // 2 or self.rows < 2:
            raise ConfigError("distance bias: at least two rows, and a largest distance beyond the first half of them")

    def bucket(self, n: int) -> int:
        half = self.rows // 2
        if n < half:
            return n
        return min(self.rows - 1, half + math.floor(math.log(n / half) / math.log(self.far / half) * (self.rows - half)))


@dataclass(frozen=True)
class QueryTemperature:
    """Queries at position p are multiplied by 1 + coef ln(floor((p + 1) / every) + 1)."""
    coef: float
    every: int

    def __post_init__(self):
        _positive(self, "every")


@dataclass(frozen=True)
class NormedAttentionSpec(AttentionSpec):
    """Attention on normed queries and keys, without a rotation."""
    norm: str = "head"       # "head": every head by itself with one shared weight; "all": the whole projection at once
    bias: bool = False       # on the projections, the output's too
    unit_values: bool = False    # every head's value is divided by its root mean square
    head_scale: bool = False     # a learned factor of the scores per head
    temperature: Optional[QueryTemperature] = None
    distance: Optional[DistanceBias] = None
    talk: bool = False       # after the softmax the heads' weights are mixed by a learned [heads, heads] matrix
    gate: bool = False       # a sigmoid per head on the output
    chunk: int = 0           # > 0: a token sees the tokens of its own chunk only (chunks count from position 0)

    def __post_init__(self):
        super().__post_init__()
        if self.norm not in ("head", "all"):
            raise ConfigError(f"attention: unknown extent {self.norm!r} of the query and key norm")
        if self.rope_dims:
            raise ConfigError("attention on normed queries and keys has no rotation")
        if self.chunk < 0:
            raise ConfigError("attention: chunk cannot be negative")


@dataclass(frozen=True)
class SsdSpec:
    """Mamba-2; head h reads group h // (heads / groups)."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                # taps of the short convolution
    norm_groups: int

    def __post_init__(self):
        _positive(self, "heads", "vdim", "state", "groups", "conv", "norm_groups")
        if self.heads % self.groups:
            raise ConfigError("ssd: heads must be a multiple of groups")
        if self.inner % self.norm_groups:
            raise ConfigError("ssd: norm_groups must divide heads * vdim")
        if self.conv > 8:
            raise ConfigError("ssd: the convolution kernel has at most 8 taps")

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class ParallelSpec:
    """left_scale * attention + right_scale * ssd, both reading the same input."""
    left: AttentionSpec
    right: SsdSpec
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule; head h reads query / key head h // (heads / kv_heads)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    unit_eps: float = 1e-6   # inside the root of the unit vectors

    def __post_init__(self):
        _positive(self, "heads", "kv_heads", "dim", "vdim", "conv")
        if self.heads % self.kv_heads:
            raise ConfigError("delta: heads must be a multiple of kv_heads")
        if self.conv > 8:
            raise ConfigError("delta: the convolution kernel has at most 8 taps")

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class GlaSpec:
    """Gated linear attention: a decay sigmoid(z)^(1 / tau) per key channel, z through ``rank`` columns."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int

    def __post_init__(self):
        _positive(self, "heads", "dim", "vdim", "rank")
        if not self.tau > 0:
            raise ConfigError("gated linear attention: tau must be positive")


@dataclass(frozen=True)
class LatentSpec:
    """Causal softmax attention whose keys and values are linear in one normed latent per token; a token's cache row is the
    latent and one rotated key part, both shared by the heads."""
    heads: int
    dim: int                 # unrotated query / key size of a head
    rope_dims: int           # rotated query / key size of a head
    vdim: int                # value size of a head
    q_rank: int              # size of the latent the queries go through, 0: none
    kv_rank: int             # size of the cached latent
    scale: float
    window: int = 0          # > 0: a token sees itself and the window - 1 tokens before it
    rope_base: float = 10000.0
    rope_scaling: Optional[RopeScaling] = None
    interleaved: bool = False    # neighbouring dimensions rotate together, else dimensions i and i + rope_dims / 2
    gate: bool = True            # a sigmoid per head on the output

    def __post_init__(self):
        _positive(self, "heads", "dim", "rope_dims", "vdim", "kv_rank")
        if self.rope_dims % 2:
            raise ConfigError("latent attention: the rotary dimensions must be even")
        if self.window < 0 or self.q_rank < 0:
            raise ConfigError("latent attention: window and q_rank cannot be negative")


@dataclass(frozen=True)
class RouterSpec:
    """Experts chosen by sigmoid scores plus a correction, weighted by the scores alone; with ``groups`` > 1 only experts of the
    ``keep`` groups whose two best corrected scores sum highest can be chosen."""
    groups: int = 1
    keep: int = 1

    def __post_init__(self):
        _positive(self, "groups", "keep")
        if self.keep > self.groups:
            raise ConfigError("router: more groups are kept than there are")


@dataclass(frozen=True)
class ClampedGlu:
    """g sigmoid(slope g) (u + offset) with the gate g = min(., limit) and the value u = clamp(., -limit, limit)."""
    limit: float
    slope: float = 1.702
    offset: float = 1.0

    def __post_init__(self):
        if not self.limit > 0:
            raise ConfigError("clamped gated unit: the limit must be positive")


@dataclass(frozen=True)
class ExpertsSpec:
    """Feed-forward of small experts of which a token uses ``top``.  Without a router a table gives every token id its experts,
    all with equal weights.  An expert is W_down act(W_up h) with act = relu squared, or with ``glu`` W_down glu(W_gate h, W_up h).
    ``shared``: width of an expert that runs for every token, times one sigmoid per token (0: none)."""
    experts: int
    top: int
    ff: int
    shared: int = 0
    router: Optional[RouterSpec] = None
    glu: Optional[ClampedGlu] = None

    def __post_init__(self):
        _positive(self, "experts", "top", "ff")
        if self.top > self.experts:
            raise ConfigError("experts: a token cannot use more experts than there are")
        if self.shared < 0:
            raise ConfigError("experts: the width of the shared expert cannot be negative")
        if self.router is not None:
            if self.experts % self.router.groups:
                raise ConfigError("experts: groups must divide the experts")
            if self.experts // self.router.groups * self.router.keep < self.top:
                raise ConfigError("experts: the groups that are kept have fewer experts than a token uses")


GLU_ACTS = ("silu", "gelu_tanh")
PLAIN_ACTS = ("relu2",)      # W_down act(W_up h): no gate


@dataclass(frozen=True)
class HybridLayer:
    mixer: Union[ParallelSpec, ConvAttentionSpec, NormedAttentionSpec, DeltaSpec, GlaSpec, LatentSpec]
    ff: int = 0              # width of the feed-forward, 0: none
    experts: Optional[ExpertsSpec] = None
    act: str = "silu"        # activation of the gate of the feed-forward, or of one without a gate
    ff_bias: bool = False    # on the projections of a feed-forward without a gate

    def __post_init__(self):
        if self.act not in GLU_ACTS + PLAIN_ACTS:
            raise ConfigError(f"unknown activation {self.act!r}")
        if self.ff_bias and self.act in GLU_ACTS:
            raise ConfigError("gated feed-forwards have no biases")


@dataclass(frozen=True)
class Loop:
    """Layers start .. stop - 1 run ``times`` times in a row, each pass with a cache of its own."""
    start: int
    stop: int
    times: int

    def __post_init__(self):
        _positive(self, "times")
        if not all(isinstance(v, int) and not isinstance(v, bool) for v in (self.start, self.stop)) or not 0 <= self.start <= self.stop:
            raise ConfigError("loop: 0 <= start <= stop is expected")


@dataclass
class HybridConfig:
    vocab: int
    width: int
    layers: List[HybridLayer] = field(default_factory=list)
    norm_eps: float = 1e-6
    token_side: int = 0      # width of the per-layer token input, 0: none
    logit_softcap: float = 0.0
    name: str = "hybrid"
    pre_norm: bool = True    # sublayers read the normed residual stream, else the stream itself
    post_norm: bool = True   # the outputs of sublayers are normed
    norm_offset: float = 0.0     # added to the stored weights of the layers' norms and the final one
    embed_scale: float = 1.0
    residual_mult: float = 1.0   # factor of every sublayer output
    logit_scale: float = 1.0     # before the soft cap
    streams: int = 0             # copies of the residual that every sublayer reads, mixes and writes (0: one plain residual)
    loop: Optional[Loop] = None
    positions: int = 0           # learned position vectors, which are the longest sequence too (0: none)

    def __post_init__(self):
        _positive(self, "vocab", "width")
        if not 0 <= self.streams <= 8 or self.positions < 0:
            raise ConfigError("streams must be 0 to 8, positions cannot be negative")
        if self.streams and (self.token_side or self.post_norm or not self.pre_norm or self.residual_mult != 1.0 or any(
                x.experts for x in self.layers)):
            raise ConfigError("residual streams: sublayers with a norm on their input only, no token side and no experts")
        if self.loop is not None and self.loop.stop > len(self.layers):
            raise ConfigError("loop: there are not as many layers")
        if self.token_side < 0:
            raise ConfigError("token_side cannot be negative")
        if not self.layers:
            raise ConfigError("a model needs at least one layer")
        if len({(m.kv_heads, m.vdim) for m in self._mixing()}) > 1:
            raise ConfigError("layers that mix values must have equal sizes of them")

    @property
    def order(self) -> List[int]:
        """The layer of every run, in order."""
        n = list(range(len(self.layers)))
        p = self.loop
        return n if p is None else n[: p.start] + n[p.start: p.stop] * p.times + n[p.stop:]

    @property
    def runs(self) -> List[HybridLayer]:
        return [self.layers[i] for i in self.order]

    def _mixing(self) -> list:
        return [x.mixer for x in self.layers if isinstance(x.mixer, ConvAttentionSpec) and x.mixer.mix_values]

    @property
    def first_mixing(self) -> int:
        """The layer run whose values later ones mix with theirs, -1: none."""
        return next((i for i, x in enumerate(self.runs) if isinstance(x.mixer, ConvAttentionSpec) and x.mixer.mix_values), -1)

    @property
    def recurrent(self) -> bool:
        """Whether a sequence owns state beside its cache pages."""
        return any(isinstance(layer.mixer, (ParallelSpec, ConvAttentionSpec, DeltaSpec, GlaSpec)) for layer in self.layers)

    def kv_bytes_per_token(self, element: int) -> int:
        n = 0
        for m in (layer.mixer for layer in self.runs):
            if isinstance(m, (ParallelSpec, ConvAttentionSpec, NormedAttentionSpec)):
                a = m.left if isinstance(m, ParallelSpec) else m
                n += a.kv_heads * (a.dim + a.vdim) * element
            elif isinstance(m, LatentSpec):
                n += (m.kv_rank + m.rope_dims) * element
        return n


@dataclass
class HybridWeights:
    """A configuration and its tensors (host memory, the design's own names)."""
    config: HybridConfig
    tensors: Dict[str, torch.Tensor]

    @property
    def vocab(self) -> int:
        return self.config.vocab

    def parameters(self) -> int:
        return sum(t.numel() for t in self.tensors.values())


# ------------------------------------------------------------------------------------------ Gugedra
def _take(obj: dict, where: str, names: Tuple[str, ...]) -> list:
    """Exactly these keys: a key nobody reads would be a constant that is silently ignored."""
    if not isinstance(obj, dict):
        raise ConfigError(f"{where}: an object is expected")
    missing, extra = [n for n in names if n not in obj], [k for k in obj if k not in names]
    if missing or extra:
        raise ConfigError(f"{where}: " + "; ".join(
            ([f"missing {', '.join(missing)}"] if missing else []) + ([f"unknown {', '.join(extra)}"] if extra else [])))
    return [obj[n] for n in names]


def _attention(obj: dict, where: str) -> AttentionSpec:
    heads, kv, dim, vdim, scale, cap, mask, rot = _take(
        obj, where, ("heads", "kv_heads", "dim", "vdim", "scale", "softcap", "mask", "rot"))
    (size,) = _take(mask, where + ".mask", ("size",))
    base, dims = _take(rot, where + ".rot", ("base", "dims"))
    return AttentionSpec(heads, kv, dim, vdim, float(scale), float(cap), int(size), int(dims), float(base))


def gugedra_config(obj: dict) -> HybridConfig:
    """``config.json`` of a Gugedra model."""
    _, layers, cap, norm, side, vocab, width = _take(
        obj, "config", ("architecture", "layers", "logit_softcap", "norm", "token_side", "vocab", "width"))
    (eps,) = _take(norm, "norm", ("eps",))
    (side_dim,) = _take(side, "token_side", ("dim",))
    if not isinstance(side_dim, int) or side_dim < 1:
        raise ConfigError("token_side.dim must be a positive integer")
    out = []
    for i, layer in enumerate(layers):
        kind, mix, mlp = _take(layer, f"layers[{i}]", ("type", "mixer", "mlp"))
        where = f"layers[{i}].mixer"
        if kind == "parallel":
            left, ls, right, rs = _take(mix, where, ("left", "left_scale", "right", "right_scale"))
            spec = ParallelSpec(_attention(left, where + ".left"),
                                SsdSpec(*_take(right, where + ".right", ("heads", "vdim", "state", "groups", "conv", "norm_groups"))),
                                float(ls), float(rs))
        elif kind == "delta":
            spec = DeltaSpec(*_take(mix, where, ("heads", "kv_heads", "dim", "vdim", "conv")))
        else:
            raise ConfigError(f"layers[{i}]: unknown mixer {kind!r}")
        ff = 0
        if mlp is not None:
            mlp_kind, ff = _take(mlp, f"layers[{i}].mlp", ("kind", "ff"))
            if mlp_kind != "dense" or ff < 1:
                raise ConfigError(f"layers[{i}].mlp: a dense feed-forward is expected")
        out.append(HybridLayer(spec, ff))
    return HybridConfig(vocab, width, out, float(eps), side_dim, float(cap), "Gugedra")


def gugedra_tensors(cfg: HybridConfig) -> Dict[str, Tuple[int, ...]]:
    """Name and shape of every tensor."""
    W = cfg.width
    t: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab, W), "side.embed": (cfg.vocab, cfg.token_side * len(cfg.layers)),
                                     "final.norm": (W,), "head": (cfg.vocab, W)}
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        t[p + "norm1"] = t[p + "norm1b"] = (W,)
        if isinstance(m, ParallelSpec):
            a, r = m.left, m.right
            t[p + "mix.left.q"], t[p + "mix.left.k"] = (a.heads * a.dim, W), (a.kv_heads * a.dim, W)
            t[p + "mix.left.v"], t[p + "mix.left.o"] = (a.kv_heads * a.vdim, W), (W, a.heads * a.vdim)
            t[p + "mix.right.in"] = (r.inner + r.channels + r.heads, W)
            t[p + "mix.right.conv"], t[p + "mix.right.conv.b"] = (r.channels, r.conv), (r.channels,)
            for n in ("dt_bias", "A_log", "D"):
                t[p + "mix.right." + n] = (r.heads,)
            t[p + "mix.right.norm"], t[p + "mix.right.o"] = (r.inner,), (W, r.inner)
        else:
            for n, size in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)):
                t[p + "mix." + n], t[p + f"mix.{n}.conv"] = (size, W), (size, m.conv)
            t[p + "mix.b"] = t[p + "mix.a"] = (m.heads, W)
            t[p + "mix.A_log"] = t[p + "mix.dt_bias"] = (m.heads,)
            t[p + "mix.norm"], t[p + "mix.g"], t[p + "mix.o"] = (m.vdim,), (m.heads * m.vdim, W), (W, m.heads * m.vdim)
        if layer.ff:
            t[p + "norm2"] = t[p + "norm2b"] = (W,)
            t[p + "mlp.gate"] = t[p + "mlp.up"] = (layer.ff, W)
            t[p + "mlp.down"] = (W, layer.ff)
        t[p + "side.gate"], t[p + "side.proj"], t[p + "side.norm"] = (cfg.token_side, W), (W, cfg.token_side), (W,)
    return t


def check_tensors(cfg: HybridConfig, tensors: Dict[str, torch.Tensor], want: Optional[Dict[str, Tuple[int, ...]]] = None) -> None:
    """``want``: names and shapes of the design's tensors (default: Gugedra's)."""
    want = gugedra_tensors(cfg) if want is None else want
    missing, extra = sorted(set(want) - set(tensors)), sorted(set(tensors) - set(want))
    if missing or extra:
        raise ConfigError(f"weights do not fit the configuration: missing {missing[:4]}, unknown {extra[:4]}")
    for n, shape in want.items():
        if tuple(tensors[n].shape) != shape:
            raise ConfigError(f"{n}: shape {tuple(tensors[n].shape)}, expected {shape}")


def load_gugedra(folder: str) -> HybridWeights:
    """A folder with ``config.json`` and ``model.safetensors``."""
    from ..interop.safetensors import load_file
    with open(os.path.join(folder, "config.json")) as f:
        cfg = gugedra_config(json.load(f))
    tensors = load_file(os.path.join(folder, "model.safetensors"))
    check_tensors(cfg, tensors)
    return HybridWeights(cfg, tensors)


def random_gugedra(cfg: HybridConfig, seed: int = 0) -> HybridWeights:
    """Random BF16 weights of a configuration (benchmarks, examples): unit-variance activations, decays spread over
    short and long memories."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, shape in gugedra_tensors(cfg).items():
        leaf = n.rsplit(".", 1)[-1]
        if leaf.startswith("norm") or leaf == "D":
            v = torch.ones(shape)
        elif leaf == "A_log":
            v = torch.linspace(-1.0, 1.5, shape[0])
        elif leaf == "dt_bias":
            v = torch.linspace(-4.0, -1.0, shape[0])
        elif leaf == "conv":
            v = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        elif leaf == "b" and len(shape) == 1:
            v = torch.zeros(shape)
        elif leaf == "embed":
            v = torch.randn(shape, generator=g)
        else:
            v = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[n] = v.to(torch.bfloat16)
    return HybridWeights(cfg, out)
