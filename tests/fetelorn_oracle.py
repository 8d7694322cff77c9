"""Plain, slow Fetelorn: one function per mechanism, whole sequences, no cache, no batching, float64.

The oracle of the hybrid-model tests.  It shares no code with the package: weights come as a dictionary
``name -> tensor`` under the checkpoint's names, the configuration as the parsed ``config.json``.
"""
import math

import torch

F = torch.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def rotate_half(x, base, dims):
    """Rotary positions for ``x [T, heads, dim]``: channel i < dims/2 turns with channel i + dims/2."""
    T, half = x.shape[0], dims // 2
    out = x.clone()
    for i in range(half):
        a = torch.arange(T, dtype=F) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def distance_bucket(n, rows, far):
    """Bucket of the distance n >= 0: one per distance below rows/2, then logarithmic up to ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def retention_core(q, k, v, decay):
    """``q, k [T, H, dk]``, ``v [T, H, dv]``: S <- decay S + k v^T, o = S^T q, token by token."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=F)
    d = torch.as_tensor(decay, dtype=F)[:, None, None]
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def retention_mixer(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q = (h @ w[p + "q"].T).reshape(T, H, m["dim"])
    k = (h @ w[p + "k"].T).reshape(T, H, m["dim"])
    v = (h @ w[p + "v"].T).reshape(T, H, m["vdim"])
    q = rotate_half(q, m["rot"]["base"], m["rot"]["dims"])
    k = rotate_half(k, m["rot"]["base"], m["rot"]["dims"]) * m["dim"] ** -0.5
    o = rms(retention_core(q, k, v, m["decay"]), eps).reshape(T, -1)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def chunk_attention_core(q, k, v, scale, chunk, rel, far, sink):
    """``q [T, H, dk]``, ``k [T, G, dk]``, ``v [T, G, dv]``; keys of the query's own chunk only, learned distance
    bias ``rel [rows, H]``, one extra term exp(sink_h) in the denominator."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for i in range(T):
        js = torch.arange(i // chunk * chunk, i + 1)
        b = torch.tensor([distance_bucket(i - int(j), rel.shape[0], far) for j in js])
        for h in range(H):
            s = (k[js, h // per] @ q[i, h]) * scale + rel[b, h]
            top = torch.maximum(s.max(), sink[h])
            e = torch.exp(s - top)
            out[i, h] = (e[:, None] * v[js, h // per]).sum(0) / (e.sum() + torch.exp(sink[h] - top))
    return out


def left_mixer(h, w, p, m, eps):
    T = h.shape[0]
    q = rms((h @ w[p + "q"].T).reshape(T, m["heads"], m["dim"]), eps)
    k = rms((h @ w[p + "k"].T).reshape(T, m["kv_heads"], m["dim"]), eps)
    v = (h @ w[p + "v"].T).reshape(T, m["kv_heads"], m["vdim"])
    o = chunk_attention_core(q, k, v, m["scale"], m["mask"]["size"], w[p + "rel"], m["bias_max"], w[p + "sink"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].T


def short_conv(x, taps):
    """Causal convolution per channel: ``x [T, C]``, ``taps [C, K]``, the last column meets the current token."""
    T, K = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                out[t] += taps[:, j] * x[s]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_core(q, k, v, g, beta):
    """``q, k, g [T, H, dk]``, ``v [T, H, dv]``, ``beta [T, H]``: decay the rows, write the error, then read."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=F)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def delta_decay(h, w, p, H, dk):
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z).reshape(-1, H, dk))


def right_mixer(h, w, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    def proj(n):
        return silu(short_conv(h @ w[p + n].T, w[p + n + ".conv"]))
    q = unit(proj("q").reshape(T, G, m["dim"])) * m["dim"] ** -0.5
    k = unit(proj("k").reshape(T, G, m["dim"]))
    v = proj("v").reshape(T, H, m["vdim"])
    of = torch.arange(H) // (H // G)
    beta = sigmoid(h @ w[p + "b"].T)
    o = delta_core(q[:, of], k[:, of], v, delta_decay(h, w, p, H, m["dim"]), beta)
    o = rms(o, eps) * w[p + "norm"]
    o = o * sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, m["vdim"])
    return o.reshape(T, -1) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    left = left_mixer(h, w, p + "left.", m["left"], eps)
    right = right_mixer(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"])


def dense_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"retention": retention_mixer, "parallel": parallel_mixer}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers_out`` collects the residual stream after every layer."""
    w = {k: v.to(F) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        h = rms(x, eps) * w[f"l{i}.norm1"]
        y = MIXERS[layer["type"]](h, w, f"l{i}.mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + dense_ff(h, w, f"l{i}.mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T


def random_weights(cfg, seed=0, gain=1.0, rank=12, rel_rows=8):
    """Random float32 weights for a configuration, lively enough that every mechanism shows in the logits."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def lin(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * (gain * s / math.sqrt(i))

    def near_one(n):
        return 1.0 + 0.2 * torch.randn(n, generator=g)

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g), "final.norm": near_one(W)}
    for i, layer in enumerate(cfg["layers"]):
        w[f"l{i}.norm1"] = near_one(W)
        p, m = f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "retention":
            H, dk, dv = m["heads"], m["dim"], m["vdim"]
            w.update({p + "q": lin(H * dk, W), p + "k": lin(H * dk, W), p + "v": lin(H * dv, W),
                      p + "g": lin(H * dv, W), p + "o": lin(W, H * dv)})
        else:
            a, lp = m["left"], p + "left."
            H, G = a["heads"], a["kv_heads"]
            w.update({lp + "q": lin(H * a["dim"], W), lp + "k": lin(G * a["dim"], W), lp + "v": lin(G * a["vdim"], W),
                      lp + "rel": torch.randn(rel_rows, H, generator=g), lp + "sink": torch.randn(H, generator=g),
                      lp + "g": lin(H, W), lp + "o": lin(W, H * a["vdim"]), lp + "out": near_one(W)})
            b, rp = m["right"], p + "right."
            H, G, dk, dv, K = b["heads"], b["kv_heads"], b["dim"], b["vdim"], b["conv"]
            w.update({rp + "q": lin(G * dk, W), rp + "k": lin(G * dk, W), rp + "v": lin(H * dv, W),
                      rp + "q.conv": torch.randn(G * dk, K, generator=g) * 0.5,
                      rp + "k.conv": torch.randn(G * dk, K, generator=g) * 0.5,
                      rp + "v.conv": torch.randn(H * dv, K, generator=g) * 0.5,
                      rp + "b": lin(H, W), rp + "A_log": torch.rand(H, generator=g) * 2 - 1.5,
                      rp + "norm": near_one(dv), rp + "a1": lin(rank, W), rp + "a2": lin(H * dk, rank),
                      rp + "dt_bias": torch.randn(H * dk, generator=g) - 2.0,
                      rp + "g1": lin(rank + 3, W), rp + "g2": lin(H * dv, rank + 3),
                      rp + "o": lin(W, H * dv), rp + "out": near_one(W)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            w.update({f"l{i}.mlp.gate": lin(ff, W), f"l{i}.mlp.up": lin(ff, W), f"l{i}.mlp.down": lin(W, ff)})
    return w
