"""Plain, slow restatement of the Gutivik decoder, one function per mechanism, for the tests.

Whole sequences in float64 (or the dtype that is passed): no cache, no batching, recurrences token by token, every key and
value of every head formed, every token's experts one by one.  Nothing here imports the package under test."""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------------------------------------- small pieces
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """The weight is stored around zero."""
    return rms(x, eps) * (1 + w)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def log_sigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, rot):
    """x [T, heads, >= dims]: pair (2i, 2i + 1), position = row number; further dimensions pass."""
    T = x.shape[0]
    out = x.clone()
    for i in range(rot["dims"] // 2):
        ang = torch.arange(T, dtype=torch.float64) * float(rot["base"]) ** (-2.0 * i / rot["dims"])
        c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def causal_conv(u, w):
    """u [T, channels], w [channels, taps], the last tap on the current token; zeros before the start."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], 0)
    return sum(w[:, j] * padded[j: j + u.shape[0]] for j in range(taps))


# ---------------------------------------------------------------------------------------------- attention
def window_attention(q, k, v, scale, window, keep_first=0, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv].  Row i sees the keys i - window + 1 .. i and the first
    ``keep_first`` ones up to i; ``sink`` [H]: a score without key or value in the denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        see = [j for j in range(i + 1) if i - j < window or j < keep_first]
        s = torch.einsum("hd,nhd->hn", q[i], k[see]) * scale
        m = s.max(-1, keepdim=True).values
        if sink is not None:
            m = torch.maximum(m, sink[:, None])
        p = torch.exp(s - m)
        total = p.sum(-1, keepdim=True)
        if sink is not None:
            total = total + torch.exp(sink[:, None] - m)
        out[i] = torch.einsum("hn,nhd->hd", p / total, v[see])
    return out


def conv_attention(h, p, cfg, first_values):
    """Attention over convolved projections.  ``first_values``: a list that holds the values of the first layer that mixes
    (empty: this layer is the first)."""
    T, H, G, D, Dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (causal_conv(h @ p[n].T + p[n + ".b"], p[n + ".conv"]) for n in ("q", "k", "v"))
    q, k, v = rotate(q.view(T, H, D), cfg["rot"]), rotate(k.view(T, G, D), cfg["rot"]), v.view(T, G, Dv)
    if cfg["v_mix"]:
        if first_values:
            v = (1 - p["vmix"]) * v + p["vmix"] * first_values[0]
        else:
            first_values.append(v)
    o = window_attention(q, k, v, cfg["scale"], cfg["mask"]["size"], cfg["mask"]["keep_first"], p["sink"])
    return o.reshape(T, H * Dv) @ p["o"].T


def latent_attention(h, p, cfg, eps):
    T, H, D, R, Dv = h.shape[0], cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"]
    q = (h @ p["q"].T).view(T, H, D + R)
    q = torch.cat([q[:, :, :D], rotate(q[:, :, D:], cfg["rot"])], -1)
    both = h @ p["dkv"].T
    c = rms(both[:, : cfg["kv_rank"]], eps) * p["dkv.norm"]
    kr = rotate(both[:, None, cfg["kv_rank"]:], cfg["rot"])
    k = torch.cat([(c @ p["uk"].T).view(T, H, D), kr.expand(T, H, R)], -1)
    v = (c @ p["uv"].T).view(T, H, Dv)
    o = window_attention(q, k, v, cfg["scale"], cfg["mask"]["size"])
    return o.reshape(T, H * Dv) @ p["o"].T


# ---------------------------------------------------------------------------------------------- recurrence
def decayed_outer(q, k, v, log_decay):
    """q / k / log_decay [T, H, D], v [T, H, Dv]: S = diag(e^log_decay) S + k v^T, o = S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = torch.exp(log_decay[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hd,hdv->hv", q[t], S)
    return out


def gated_linear(h, p, cfg, eps):
    T, H, D, Dv = h.shape[0], cfg["heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (h @ p["q"].T).view(T, H, D) * D ** -0.5, (h @ p["k"].T).view(T, H, D), (h @ p["v"].T).view(T, H, Dv)
    z = (h @ p["a1"].T) @ p["a2"].T + p["a2.b"]
    o = decayed_outer(q, k, v, (log_sigmoid(z) / cfg["tau"]).view(T, H, D))
    o = (rms(o, eps) * p["norm"]).reshape(T, H * Dv)
    g = h @ p["g"].T
    return (o * (g * sigmoid(g))) @ p["o"].T


# ---------------------------------------------------------------------------------------------- feed-forward
def dense(h, p):
    return (gelu_tanh(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def expert(h, gate, up, down, limit):
    g, u = torch.clamp(h @ gate.T, max=limit), torch.clamp(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(z, correction, cfg):
    """z [T, experts] -> for every token a list of (expert, weight)."""
    top, E, groups = cfg["top"], cfg["experts"], cfg.get("groups")
    out = []
    for row in sigmoid(z):
        choice = (row + correction).tolist()
        allowed = range(E)
        if groups is not None:
            n = E // groups["count"]
            score = [sum(sorted(choice[g * n: (g + 1) * n])[-2:]) for g in range(groups["count"])]
            best = sorted(range(groups["count"]), key=lambda g: (-score[g], g))[: groups["keep"]]
            allowed = [e for e in range(E) if e // n in best]
        chosen = sorted(allowed, key=lambda e: (-choice[e], e))[:top]
        total = sum(row[e] for e in chosen) + 1e-20
        out.append([(e, row[e] / total) for e in chosen])
    return out


def routed_experts(h, p, cfg):
    out = torch.zeros_like(h)
    for t, chosen in enumerate(route(h @ p["router"].T, p["correction"], cfg["router"])):
        for e, w in chosen:
            out[t] = out[t] + w * expert(h[t], p[f"e{e}.gate"], p[f"e{e}.up"], p[f"e{e}.down"], cfg["expert"]["limit"])
    return out


# ---------------------------------------------------------------------------------------------- the model
def _sub(p, prefix):
    return {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64, capture=None):
    """Logits [T, vocab] of one whole sequence; ``capture``: a list that receives the residual stream after each layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, first_values = cfg["norm"]["eps"], []
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = _sub(w, f"l{i}."), layer["mixer"], layer["mlp"]
        h, mix = offset_norm(x, p["norm1"], eps), _sub(p, "mix.")
        if layer["type"] == "attention":
            x = x + conv_attention(h, mix, m, first_values)
        elif layer["type"] == "latent_attention":
            x = x + latent_attention(h, mix, m, eps)
        else:
            x = x + gated_linear(h, mix, m, eps)
        if f is not None:
            h = offset_norm(x, p["norm2"], eps)
            x = x + (dense(h, _sub(p, "mlp.")) if f["kind"] == "dense" else routed_experts(h, _sub(p, "mlp."), f))
        if capture is not None:
            capture.append(x.clone())
    z = offset_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"]
    return cfg["logit_softcap"] * torch.tanh(z / cfg["logit_softcap"])


# ---------------------------------------------------------------------------------------------- random models
def dense_ff(ff=44):
    return {"kind": "dense", "ff": ff}


def moe_ff(experts=6, top=2, ff=28, limit=0.8, groups=(3, 2)):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router}


def attention_layer(mlp, heads=6, kv_heads=2, dim=24, vdim=20, conv=4, scale=0.22, window=21, keep=5, rot=16, base=4000.0, v_mix=True):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"keep_first": keep, "size": window},
                      "rot": {"base": base, "dims": rot}, "scale": scale, "v_mix": v_mix, "vdim": vdim}}


def latent_layer(mlp, heads=5, dim=24, rot_dim=16, vdim=20, kv_rank=56, scale=0.19, window=17, base=7000.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"dim": dim, "heads": heads, "kv_rank": kv_rank, "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim},
                      "rot_dim": rot_dim, "scale": scale, "vdim": vdim}}


def gla_layer(mlp, heads=3, dim=24, vdim=20, tau=8.0):
    return {"type": "gla", "mlp": mlp, "mixer": {"dim": dim, "heads": heads, "tau": tau, "vdim": vdim}}


def random_config(layers=None, vocab=181, width=88, eps=1e-4, scale=1.7, softcap=9.0):
    layers = layers or [attention_layer(moe_ff()), gla_layer(dense_ff()), latent_layer(None), attention_layer(moe_ff(groups=None)),
                        gla_layer(moe_ff())]
    return {"architecture": "Gutivik", "layers": layers, "logit_scale": scale, "logit_softcap": softcap, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


ROUTED = 6      # columns of the residual stream that only the embedding writes and only routers read


def random_weights(cfg, seed=0, rank=5):
    """Routers read a sign pattern that every token carries in the first columns, where no layer writes: their choices rest on no
    close call that rounding could turn."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def n(*shape, s=1.0):
        return torch.randn(*shape, generator=g) * s / math.sqrt(shape[-1])

    def reads(*shape, s=1.0):
        w = n(*shape, s=s)
        w[:, :ROUTED] = 0
        return w

    def writes(*shape):
        w = n(*shape)
        w[:ROUTED] = 0
        return w

    def norm(size, mean):
        return mean + 0.3 * torch.randn(size, generator=g)
    embed = torch.randn(V, W, generator=g)
    embed[:, :ROUTED] = torch.randint(0, 2, (V, ROUTED), generator=g) * 4.0 - 2.0
    out = {"embed": embed, "final.norm": norm(W, 0.0), "head": n(V, W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        out[p + "norm1"] = norm(W, 0.0)
        if layer["type"] == "latent_attention":
            R, C = m["rot_dim"], m["kv_rank"]
            out.update({p + "mix.q": reads(H * (D + R), W, s=1.6), p + "mix.dkv": reads(C + R, W), p + "mix.dkv.norm": norm(C, 1.0),
                        p + "mix.uk": n(H * D, C, s=1.6), p + "mix.uv": n(H * Dv, C), p + "mix.o": writes(W, H * Dv)})
        elif layer["type"] == "attention":
            G = m["kv_heads"]
            for name, size in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                out[p + "mix." + name], out[p + f"mix.{name}.b"] = reads(size, W, s=1.5), 0.4 * torch.randn(size, generator=g)
                out[p + f"mix.{name}.conv"] = n(size, m["conv"], s=1.5)
            out[p + "mix.sink"], out[p + "mix.o"] = torch.randn(H, generator=g), writes(W, H * Dv)
            if m["v_mix"]:
                out[p + "mix.vmix"] = torch.tensor(0.3 + 0.1 * i)
        else:
            out.update({p + "mix.q": reads(H * D, W), p + "mix.k": reads(H * D, W), p + "mix.v": reads(H * Dv, W), p + "mix.g": reads(H * Dv, W),
                        p + "mix.o": writes(W, H * Dv), p + "mix.norm": norm(Dv, 1.0), p + "mix.a1": reads(rank, W),
                        p + "mix.a2": n(H * D, rank, s=1.5), p + "mix.a2.b": torch.linspace(-4.0, 5.0, H * D)})
        if f is None:
            continue
        out[p + "norm2"] = norm(W, 0.0)
        if f["kind"] == "dense":
            out[p + "mlp.gate"], out[p + "mlp.up"], out[p + "mlp.down"] = reads(f["ff"], W), reads(f["ff"], W), writes(W, f["ff"])
            continue
        E, F = f["router"]["experts"], f["expert"]["ff"]
        for e in range(E):
            out[p + f"mlp.e{e}.gate"], out[p + f"mlp.e{e}.up"], out[p + f"mlp.e{e}.down"] = reads(F, W), reads(F, W), writes(W, F)
        router = torch.zeros(E, W)
        router[:, :ROUTED] = torch.randn(E, ROUTED, generator=g) * 0.6
        out[p + "mlp.router"], out[p + "mlp.correction"] = router, torch.randn(E, generator=g) * 0.4 - 0.5
    return {k: v.to(torch.bfloat16) for k, v in out.items()}
