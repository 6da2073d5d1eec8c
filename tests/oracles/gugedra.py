"""Plain, slow restatement of the Gugedra decoder, one function per mechanism, for the tests.

Everything runs on whole sequences in float64 (or the dtype that is passed), token by token where the mechanism is a
recurrence, with no cache, no batching and no chunking.  Nothing here imports the package under test."""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------------------------------------- small pieces
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_half(x, dims, base):
    """x [T, heads, D]: the first ``dims`` of D rotate, i pairs with i + dims / 2, position = row number."""
    T = x.shape[0]
    half = dims // 2
    out = x.clone()
    for i in range(half):
        ang = torch.arange(T, dtype=torch.float64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def causal_conv(x, w, b=None):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x], 0)
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + padded[j: j + T] * w[:, j]
    return y if b is None else y + b


# ---------------------------------------------------------------------------------------------- attention
def window_attention(q, k, v, scale, softcap, window):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]; row i sees keys i - window + 1 .. i."""
    T, H = q.shape[0], q.shape[1]
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        lo = max(0, i - window + 1)
        for h in range(H):
            s = (k[lo: i + 1, h // rep] @ q[i, h]) * scale
            s = softcap * torch.tanh(s / softcap)
            p = torch.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo: i + 1, h // rep]
    return out


def attention_branch(h, p, cfg):
    T = h.shape[0]
    H, G, D, Dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = (h @ p["q"].T).view(T, H, D)
    k = (h @ p["k"].T).view(T, G, D)
    v = (h @ p["v"].T).view(T, G, Dv)
    q, k = (rotate_half(t, cfg["rot"]["dims"], cfg["rot"]["base"]) for t in (q, k))
    o = window_attention(q, k, v, cfg["scale"], cfg["softcap"], cfg["mask"]["size"])
    return o.reshape(T, H * Dv) @ p["o"].T


# ---------------------------------------------------------------------------------------------- state-space branch
def ssd_recurrence(x, B, C, dt, A_log, D):
    """x [T, H, P], B / C [T, G, N], dt [T, H] (after softplus) -> y [T, H, P], final state [H, N, P]."""
    T, H, P = x.shape
    rep = H // B.shape[1]
    S = torch.zeros(H, B.shape[2], P, dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // rep
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    """y * silu(z), each of ``groups`` equal parts divided by its own root mean square, times w."""
    u = y * silu(z)
    parts = u.view(u.shape[0], groups, -1)
    parts = parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)
    return parts.reshape(u.shape) * w


def ssd_branch(h, p, cfg, eps):
    T = h.shape[0]
    H, P, N, G = cfg["heads"], cfg["vdim"], cfg["state"], cfg["groups"]
    inner = H * P
    zxbcdt = h @ p["in"].T
    z, xbc, dt = zxbcdt[:, :inner], zxbcdt[:, inner: 2 * inner + 2 * G * N], zxbcdt[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, p["conv"], p["conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner: inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    y, _ = ssd_recurrence(x, B, C, softplus(dt + p["dt_bias"]), p["A_log"], p["D"])
    return gated_group_norm(y.reshape(T, inner), z, p["norm"], cfg["norm_groups"], eps) @ p["o"].T


def parallel_mixer(h, p, cfg, eps):
    left = attention_branch(h, _sub(p, "left."), cfg["left"])
    right = ssd_branch(h, _sub(p, "right."), cfg["right"], eps)
    return cfg["left_scale"] * left + cfg["right_scale"] * right


# ---------------------------------------------------------------------------------------------- gated delta rule
def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, beta, g):
    """q / k [T, G, D] (unit vectors, q already scaled), v [T, H, Dv], beta / g [T, H] -> o [T, H, Dv], state [H, D, Dv]."""
    T, H, Dv = v.shape
    rep = H // q.shape[1]
    S = torch.zeros(H, q.shape[2], Dv, dtype=v.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // rep], q[t, h // rep]
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ kk)
            S[h] = S[h] + torch.outer(kk, u)
            o[t, h] = S[h].T @ qq
    return o, S


def delta_mixer(h, p, cfg, eps):
    T = h.shape[0]
    H, G, D, Dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (silu(causal_conv(h @ p[n].T, p[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.view(T, G, D)) * D ** -0.5
    k = unit(k.view(T, G, D))
    beta = 1 / (1 + torch.exp(-(h @ p["b"].T)))
    g = torch.exp(-torch.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))
    o, _ = delta_recurrence(q, k, v.view(T, H, Dv), beta, g)
    o = rms_norm(o, p["norm"], eps) * silu((h @ p["g"].T).view(T, H, Dv))
    return o.reshape(T, H * Dv) @ p["o"].T


# ---------------------------------------------------------------------------------------------- the model
MIXERS = {"parallel": parallel_mixer, "delta": delta_mixer}


def swiglu(h, p):
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def token_side(x, tokens, layer, table, dim, p, eps):
    e = table[tokens][:, layer * dim: (layer + 1) * dim]
    y = (gelu_tanh(x @ p["gate"].T) * e) @ p["proj"].T
    return x + rms_norm(y, p["norm"], eps)


def _sub(p, prefix):
    return {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, dtype=torch.float64, capture=None):
    """Logits [T, vocab] of one whole sequence; ``capture``: a list that receives the residual stream after each layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = w["embed"][tokens]
    for i, layer in enumerate(cfg["layers"]):
        p = _sub(w, f"l{i}.")
        m = MIXERS[layer["type"]](rms_norm(x, p["norm1"], eps), _sub(p, "mix."), layer["mixer"], eps)
        x = x + rms_norm(m, p["norm1b"], eps)
        if layer["mlp"] is not None:
            f = swiglu(rms_norm(x, p["norm2"], eps), _sub(p, "mlp."))
            x = x + rms_norm(f, p["norm2b"], eps)
        x = token_side(x, tokens, i, w["side.embed"], cfg["token_side"]["dim"], _sub(p, "side."), eps)
        if capture is not None:
            capture.append(x.clone())
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(logits / cap)


# ---------------------------------------------------------------------------------------------- random models
def random_config(layers=("parallel", "delta", "parallel"), vocab=193, width=96, ff=144, left=None, right=None, delta=None,
                  left_scale=0.7, right_scale=1.3, side=16, logit_softcap=12.0, eps=1e-5):
    left = {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 24, "scale": 0.21, "softcap": 9.0, "mask": {"size": 37},
            "rot": {"base": 5000.0, "dims": 12}, **(left or {})}
    right = {"heads": 6, "vdim": 16, "state": 24, "groups": 3, "conv": 4, "norm_groups": 2, **(right or {})}
    delta = {"heads": 6, "kv_heads": 2, "dim": 24, "vdim": 40, "conv": 3, **(delta or {})}
    out = []
    for n, kind in enumerate(layers):
        if kind == "parallel":
            out.append({"type": kind, "mixer": {"left": dict(left), "right": dict(right), "left_scale": left_scale,
                                                "right_scale": right_scale}, "mlp": {"kind": "dense", "ff": ff}})
        else:
            out.append({"type": kind, "mixer": dict(delta), "mlp": {"kind": "dense", "ff": ff} if n % 2 else None})
    return {"architecture": "Gugedra", "layers": out, "logit_softcap": logit_softcap, "norm": {"eps": eps},
            "token_side": {"dim": side}, "vocab": vocab, "width": width}


def random_weights(cfg, seed=0, spread=1.0):
    """BF16 tensors under the design's names; the decays are spread so that states live between a few and many tokens."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]

    def lin(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * (s * spread / math.sqrt(i))

    def near_one(n):
        return 1 + 0.2 * torch.randn(n, generator=g)
    w = {"embed": torch.randn(V, W, generator=g), "final.norm": near_one(W), "head": lin(V, W, 3.0),
         "side.embed": torch.randn(V, cfg["token_side"]["dim"] * len(cfg["layers"]), generator=g)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            w[p + n] = near_one(W)
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            H, G = a["heads"], a["kv_heads"]
            w[p + "mix.left.q"], w[p + "mix.left.k"] = lin(H * a["dim"], W, 1.5), lin(G * a["dim"], W, 1.5)
            w[p + "mix.left.v"], w[p + "mix.left.o"] = lin(G * a["vdim"], W), lin(W, H * a["vdim"])
            inner, gn = r["heads"] * r["vdim"], r["groups"] * r["state"]
            w[p + "mix.right.in"] = lin(2 * inner + 2 * gn + r["heads"], W)
            w[p + "mix.right.conv"] = torch.randn(inner + 2 * gn, r["conv"], generator=g) * 0.6
            w[p + "mix.right.conv.b"] = torch.randn(inner + 2 * gn, generator=g) * 0.3
            w[p + "mix.right.dt_bias"] = torch.linspace(-4.0, 0.5, r["heads"])
            w[p + "mix.right.A_log"] = torch.linspace(-1.0, 1.0, r["heads"])
            w[p + "mix.right.D"] = near_one(r["heads"])
            w[p + "mix.right.norm"], w[p + "mix.right.o"] = near_one(inner), lin(W, inner)
        else:
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, size in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                w[p + f"mix.{n}"] = lin(size, W)
                w[p + f"mix.{n}.conv"] = torch.randn(size, m["conv"], generator=g) * 0.7
            w[p + "mix.b"], w[p + "mix.a"] = lin(H, W), lin(H, W)
            w[p + "mix.A_log"], w[p + "mix.dt_bias"] = torch.linspace(-2.0, 0.5, H), torch.linspace(-3.0, 0.0, H)
            w[p + "mix.norm"], w[p + "mix.g"], w[p + "mix.o"] = near_one(Dv), lin(H * Dv, W), lin(W, H * Dv)
        if layer["mlp"]:
            F = layer["mlp"]["ff"]
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = lin(F, W), lin(F, W), lin(W, F)
        d = cfg["token_side"]["dim"]
        w[p + "side.gate"], w[p + "side.proj"], w[p + "side.norm"] = lin(d, W), lin(W, d), 0.5 * near_one(W)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
