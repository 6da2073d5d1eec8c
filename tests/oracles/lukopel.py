"""Plain, slow restatement of the Lukopel decoder, one function per mechanism, for the tests.

Whole sequences in float64 (or the dtype that is passed): no cache, no batching, every score and every weight of every head
formed, every stream of the residual kept apart.  Nothing here imports the package under test."""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------------------------------------- small pieces
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def head_norm(x, w, heads, eps):
    """Every head of a projection by itself; all share one weight."""
    T = x.shape[0]
    return norm(x.view(T, heads, -1), w, eps)


def whole_norm(x, w, heads, eps):
    """The whole projection at once, then split."""
    return norm(x, w, eps).view(x.shape[0], heads, -1)


def bucket(n, rows, far):
    """Row of a bias table for distance n: one each below rows / 2, then logarithmic up to ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def distance_bias(rel, T, far):
    """[H, T, T]: entry (h, i, j) for i >= j."""
    rows = torch.tensor([bucket(n, rel.shape[0], far) for n in range(T)])
    n = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    return rel[rows[n]].permute(2, 0, 1)


def temperatures(T, coef, every, dtype):
    return torch.tensor([1 + coef * math.log((p + 1) // every + 1) for p in range(T)], dtype=dtype)


def same_chunk(T, size):
    """[T, T]: j <= i in the chunk of i."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def causal(T):
    return torch.ones(T, T).tril().bool()


def weights_of(scores, visible):
    """Softmax over the visible keys; scores [H, T, T]."""
    s = scores.masked_fill(~visible, -math.inf)
    p = torch.exp(s - s.amax(-1, keepdim=True))
    return p / p.sum(-1, keepdim=True)


def grouped(x, heads):
    """[T, G, D] -> [T, heads, D]: query head h reads head floor(h / (heads / G))."""
    return x[:, torch.arange(heads) // (heads // x.shape[1])]


# ---------------------------------------------------------------------------------------------- mixers
def talking_attention(h, p, cfg, eps):
    """Every head's weights see the biases of distance, then become mixtures of all heads' weights."""
    T, H, G = h.shape[0], cfg["heads"], cfg["kv_heads"]
    q, k = head_norm(h @ p["q"].T, p["q.norm"], H, eps), head_norm(h @ p["k"].T, p["k.norm"], G, eps)
    v = rms((h @ p["v"].T).view(T, G, cfg["vdim"]), eps)
    q = q * temperatures(T, cfg["q_temp"]["coef"], cfg["q_temp"]["every"], h.dtype)[:, None, None]
    scores = torch.einsum("ihd,jhd->hij", q, grouped(k, H)) * cfg["scale"] + distance_bias(p["rel"], T, cfg["bias_max"])
    mixed = torch.einsum("hg,gij->hij", p["talk"], weights_of(scores, causal(T)))
    o = torch.einsum("hij,jhd->ihd", mixed, grouped(v, H))
    o = o / (1 + torch.exp(-(h @ p["g"].T)))[:, :, None]
    return o.reshape(T, -1) @ p["o"].T


def chunked_attention(h, p, cfg, eps):
    T, H, G = h.shape[0], cfg["heads"], cfg["kv_heads"]
    q = whole_norm(h @ p["q"].T + p["q.b"], p["q.norm"], H, eps)
    k = whole_norm(h @ p["k"].T + p["k.b"], p["k.norm"], G, eps)
    v = (h @ p["v"].T + p["v.b"]).view(T, G, cfg["vdim"])
    scores = torch.einsum("ihd,jhd->hij", q, grouped(k, H)) * cfg["scale"] * p["temp"][:, None, None]
    o = torch.einsum("hij,jhd->ihd", weights_of(scores, same_chunk(T, cfg["mask"]["size"])), grouped(v, H))
    return o.reshape(T, -1) @ p["o"].T + p["o.b"]


def dense(h, p):
    return torch.clamp(h @ p["up"].T + p["up.b"], min=0) ** 2 @ p["down"].T + p["down.b"]


# ---------------------------------------------------------------------------------------------- the model
def hyper_step(xs, p, sublayer):
    """xs [streams, T, width]; ``sublayer``: the normed sublayer as a function of its input."""
    u = sum(p["in"][s] * xs[s] for s in range(len(xs)))
    y = sublayer(u)
    return torch.stack([sum(p["mix"][s, t] * xs[s] for s in range(len(xs))) + p["out"][t] * y for t in range(len(xs))])


def layer_order(cfg):
    loop, n = cfg["loop"], len(cfg["layers"])
    return [*range(loop["start"]), *list(range(loop["start"], loop["stop"])) * loop["times"], *range(loop["stop"], n)]


def _sub(p, prefix):
    return {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64, capture=None):
    """Logits [T, vocab] of one whole sequence; ``capture``: a list that receives the sum of the streams after each layer run."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, T = cfg["norm"]["eps"], len(tokens)
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"] + w["pos"][:T]
    xs = x.repeat(cfg["streams"], 1, 1)
    for i in layer_order(cfg):
        layer, p = cfg["layers"][i], _sub(w, f"l{i}.")
        mixer = {"attention": talking_attention, "attention_2": chunked_attention}[layer["type"]]
        xs = hyper_step(xs, _sub(p, "hc1."), lambda u: mixer(norm(u, p["norm1"], eps), _sub(p, "mix."), layer["mixer"], eps))
        if layer["mlp"] is not None:
            xs = hyper_step(xs, _sub(p, "hc2."), lambda u: dense(norm(u, p["norm2"], eps), _sub(p, "mlp.")))
        if capture is not None:
            capture.append(xs.sum(0))
    return norm(xs.sum(0), w["final.norm"], eps) @ w["head"].T


# ---------------------------------------------------------------------------------------------- random models
def talking_layer(ff=52, heads=6, kv_heads=3, dim=24, vdim=20, scale=0.22, bias_max=37, coef=0.4, every=23, bias_rows=12):
    """``bias_rows`` is a size of the tensors only."""
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"bias_max": bias_max, "dim": dim, "heads": heads, "kv_heads": kv_heads, "q_temp": {"coef": coef, "every": every},
                      "scale": scale, "vdim": vdim}}


def chunked_layer(ff=44, heads=6, kv_heads=2, dim=20, vdim=24, scale=0.25, size=21):
    return {"type": "attention_2", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": size}, "scale": scale, "vdim": vdim}}


def random_config(layers=None, vocab=181, width=88, eps=1e-4, embed_scale=3.0, loop=(1, 3, 2), streams=2, max_positions=400):
    layers = layers or [talking_layer(), chunked_layer(), talking_layer(None, kv_heads=1), chunked_layer(None, size=50)]
    return {"architecture": "Lukopel", "embedding": {"scale": embed_scale}, "layers": layers,
            "loop": dict(zip(("start", "stop", "times"), loop)), "max_positions": max_positions, "norm": {"eps": eps}, "streams": streams,
            "vocab": vocab, "width": width}


def random_weights(cfg, seed=0, bias_rows=12):
    """``bias_rows``: rows of the bias tables, one number or one per layer."""
    g = torch.Generator().manual_seed(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]

    def n(*shape, s=1.0):
        return torch.randn(*shape, generator=g) * s / math.sqrt(shape[-1])

    def around(size, mean, spread=0.3):
        return mean + spread * torch.randn(size, generator=g)
    out = {"embed": torch.randn(V, W, generator=g) / cfg["embedding"]["scale"], "pos": 0.5 * torch.randn(cfg["max_positions"], W, generator=g),
           "final.norm": around(W, 1.0), "head": n(V, W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for name, size in (("q", H * D), ("k", G * D), ("v", G * Dv)):
            out[p + "mix." + name] = n(size, W)
        out[p + "mix.o"] = n(W, H * Dv)
        if layer["type"] == "attention":
            B = bias_rows if isinstance(bias_rows, int) else bias_rows[i]
            out.update({p + "mix.q.norm": around(D, 1.3), p + "mix.k.norm": around(D, 1.3), p + "mix.rel": torch.randn(B, H, generator=g),
                        p + "mix.talk": 0.8 * torch.eye(H) + 0.4 * n(H, H), p + "mix.g": n(H, W)})
        else:
            for name, size in (("q", H * D), ("k", G * D), ("v", G * Dv), ("o", W)):
                out[p + f"mix.{name}.b"] = around(size, 0.0)
            out.update({p + "mix.q.norm": around(H * D, 1.3), p + "mix.k.norm": around(G * D, 1.3), p + "mix.temp": around(H, 1.0)})
        if f is not None:
            out.update({p + "mlp.up": n(f["ff"], W), p + "mlp.up.b": around(f["ff"], 0.0), p + "mlp.down": n(W, f["ff"]),
                        p + "mlp.down.b": around(W, 0.0)})
        for q in ("1", "2")[: 1 if f is None else 2]:
            out[p + "norm" + q] = around(W, 1.0)
            out.update({p + f"hc{q}.in": around(S, 1.0 / S), p + f"hc{q}.out": around(S, 1.0),
                        p + f"hc{q}.mix": torch.eye(S) * 0.8 + 0.2 / S + 0.1 * torch.randn(S, S, generator=g)})
    return {k: v.to(torch.bfloat16) for k, v in out.items()}
