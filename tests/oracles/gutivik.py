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
