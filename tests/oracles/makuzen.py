"""Plain, slow restatement of the Makuzen decoder, one function per mechanism, for the tests.

Whole sequences in float64 (or the dtype that is passed): no cache, no batching, every key and value of every head formed
from the latents, every token's experts one by one.  Nothing here imports the package under test."""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------------------------------------- small pieces
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def squared_relu(z):
    return torch.clamp(z, min=0) ** 2


# ---------------------------------------------------------------------------------------------- rotation
def yarn_frequencies(dims, base, scaling):
    """Frequencies of the dims / 2 pairs and the factor of cos and sin."""
    freq = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freq, 1.0

    def turns(t):      # the (fractional) pair that makes t turns over the original context
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo = max(math.floor(turns(scaling["fast"])), 0)
    hi = min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, dims]: pair (i, i + dims / 2), position = row number."""
    T, half = x.shape[0], rot["dims"] // 2
    freq, mul = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    out = x.clone()
    for i in range(half):
        ang = torch.arange(T, dtype=torch.float64) * freq[i]
        c, s = (torch.cos(ang) * mul).to(x.dtype)[:, None], (torch.sin(ang) * mul).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


# ---------------------------------------------------------------------------------------------- attention
def window_attention(q, k, v, scale, window):
    """q / k [T, H, D], v [T, H, Dv] -> [T, H, Dv]; row i sees keys i - window + 1 .. i."""
    T, H = q.shape[0], q.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        lo = max(0, i - window + 1)
        s = torch.einsum("hd,nhd->hn", q[i], k[lo: i + 1]) * scale
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hn,nhd->hd", p / p.sum(-1, keepdim=True), v[lo: i + 1])
    return out


def latents(h, p, cfg, eps):
    """The normed latent [T, kv_rank] and the rotated key part [T, rot_dim] that all heads share."""
    both = h @ p["dkv"].T
    c = rms_norm(both[:, : cfg["kv_rank"]], p["dkv.norm"], eps)
    return c, rotate(both[:, None, cfg["kv_rank"]:], cfg["rot"])[:, 0]


def latent_attention(h, p, cfg, eps):
    T, H, D, R, Dv = h.shape[0], cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"]
    q = (rms_norm(h @ p["dq"].T, p["dq.norm"], eps) @ p["uq"].T).view(T, H, D + R)
    q = torch.cat([q[:, :, :D], rotate(q[:, :, D:], cfg["rot"])], -1)
    c, kr = latents(h, p, cfg, eps)
    k = torch.cat([(c @ p["uk"].T).view(T, H, D), kr[:, None].expand(T, H, R)], -1)
    v = (c @ p["uv"].T).view(T, H, Dv)
    o = window_attention(q, k, v, cfg["scale"], cfg["mask"]["size"])
    o = o * sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(T, H * Dv) @ p["o"].T


# ---------------------------------------------------------------------------------------------- feed-forward
def expert(h, up, down):
    return squared_relu(h @ up.T) @ down.T


def table_moe(h, tokens, p, cfg):
    """Experts by token id, equal weights; the shared expert times one sigmoid per token."""
    top = cfg["router"]["top"]
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens.tolist()):
        for e in p["table"][tok].long().tolist():
            out[t] = out[t] + expert(h[t], p[f"e{e}.up"], p[f"e{e}.down"]) / top
    if cfg.get("shared") is not None:
        out = out + sigmoid(h @ p["shared.sg"].T) * expert(h, p["shared.up"], p["shared.down"])
    return out


# ---------------------------------------------------------------------------------------------- the model
def _sub(p, prefix):
    return {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64, capture=None):
    """Logits [T, vocab] of one whole sequence; ``capture``: a list that receives the residual stream after each layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = _sub(w, f"l{i}.")
        x = x + m * rms_norm(latent_attention(x, _sub(p, "mix."), layer["mixer"], eps), p["norm1"], eps)
        if layer["mlp"] is not None:
            x = x + m * rms_norm(table_moe(x, tokens, _sub(p, "mlp."), layer["mlp"]), p["norm2"], eps)
        if capture is not None:
            capture.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


# ---------------------------------------------------------------------------------------------- random models
def random_layer(heads=5, dim=24, rot_dim=16, vdim=20, kv_rank=56, q_rank=44, scale=0.19, window=19, base=7000.0, scaling="yarn",
                 experts=6, top=2, ff=28, shared=36, mlp=True):
    if scaling == "yarn":
        scaling = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}
    rot = {"base": base, "dims": rot_dim, "scaling": scaling}
    if scaling is None:
        rot.pop("scaling")
    ffn = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}
    return {"type": "latent_attention", "mlp": ffn if mlp else None,
            "mixer": {"dim": dim, "heads": heads, "kv_rank": kv_rank, "mask": {"size": window}, "q_rank": q_rank, "rot": rot,
                      "rot_dim": rot_dim, "scale": scale, "vdim": vdim}}


def random_config(layers=None, vocab=187, width=88, eps=1e-4, mult=0.45, scale=2.5):
    return {"architecture": "Makuzen", "embedding": {"scale": scale}, "layers": layers or [random_layer() for _ in range(3)],
            "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


def random_weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def n(*shape, s=1.0):
        return (torch.randn(*shape, generator=g) * s / math.sqrt(shape[-1])).to(torch.bfloat16)

    def norm(size):
        return (1 + 0.3 * torch.randn(size, generator=g)).to(torch.bfloat16)
    out = {"embed": torch.randn(cfg["vocab"], W, generator=g).to(torch.bfloat16), "final.norm": norm(W), "head": n(cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        H, D, R, Dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
        out[p + "norm1"] = norm(W)
        out.update({p + "mix.dq": n(m["q_rank"], W), p + "mix.dq.norm": norm(m["q_rank"]), p + "mix.uq": n(H * (D + R), m["q_rank"], s=1.6),
                    p + "mix.dkv": n(m["kv_rank"] + R, W), p + "mix.dkv.norm": norm(m["kv_rank"]), p + "mix.uk": n(H * D, m["kv_rank"], s=1.6),
                    p + "mix.uv": n(H * Dv, m["kv_rank"]), p + "mix.g": n(H, W), p + "mix.o": n(W, H * Dv)})
        if f is not None:
            out[p + "norm2"] = norm(W)
            E, top, F = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
            for e in range(E):
                out[p + f"mlp.e{e}.up"], out[p + f"mlp.e{e}.down"] = n(F, W), n(W, F)
            out[p + "mlp.table"] = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(cfg["vocab"])]).to(torch.int32)
            S = f["shared"]["ff"]
            out.update({p + "mlp.shared.up": n(S, W), p + "mlp.shared.down": n(W, S), p + "mlp.shared.sg": n(1, W, s=2.0)})
    return out
