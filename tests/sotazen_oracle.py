"""Plain, slow Sotazen: one function per mechanism, whole sequences, no cache, no batching, float64.

The oracle of the tests of the differential / latent / lightning model.  It shares no code with the package: weights come as
a dictionary ``name -> tensor`` under the checkpoint's names, the configuration as the parsed ``config.json``.
"""
import torch

F = torch.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def relu2(z):
    return torch.clamp(z, min=0.0) ** 2


def rotate_pairs(x, base, dims):
    """Rotary positions for ``x [T, heads, dim]``: channels 2 i and 2 i + 1 turn together, i < dims / 2."""
    T = x.shape[0]
    out = x.clone()
    for i in range(dims // 2):
        a = torch.arange(T, dtype=F) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_attention(q, k, v, scale, window, cap):
    """``q [T, H, dk]``, ``k [T, G, dk]``, ``v [T, G', dv]`` (groups by integer division): softmax over the keys
    ``i - window + 1 .. i`` of scores pressed through ``cap * tanh(score / cap)``."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    pk, pv = H // k.shape[1], H // v.shape[1]
    kh, vh = k[:, torch.arange(H) // pk], v[:, torch.arange(H) // pv]
    for i in range(T):
        j0 = max(0, i - window + 1) if window else 0
        s = torch.einsum("hd,jhd->hj", q[i], kh[j0:i + 1]) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhd->hd", e, vh[j0:i + 1]) / e.sum(-1, keepdim=True)
    return out


def diff_lambda(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def differential_core(q, k, v, lam, diff, scale, window, cap, eps):
    """``q [T, H, 2, dk]``, ``k [T, G, 2, dk]``, ``v [T, G, dv]``: two attentions over the same values, subtracted, normed."""
    a1 = window_attention(q[:, :, 0], k[:, :, 0], v, scale, window, cap)
    a2 = window_attention(q[:, :, 1], k[:, :, 1], v, scale, window, cap)
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_mixer(h, w, p, m, eps):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H * 2, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G * 2, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, m["vdim"])
    q, k = rms(q, eps) * w[p + "q.norm"], rms(k, eps) * w[p + "k.norm"]
    q = rotate_pairs(q, m["rot"]["base"], m["rot"]["dims"]).reshape(T, H, 2, d)
    k = rotate_pairs(k, m["rot"]["base"], m["rot"]["dims"]).reshape(T, G, 2, d)
    lam = diff_lambda(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    o = differential_core(q, k, v, lam, m["diff"], m["scale"], m["mask"]["size"], m["softcap"], eps)
    o = o.reshape(T, -1) * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T + w[p + "o.b"]


def lightning_core(q, k, v, decay):
    """``q, k [T, H, dk]``, ``v [T, H, dv]``: S <- decay S + k v^T, o = S^T q, token by token."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=F)
    d = torch.as_tensor(decay, dtype=F)[:, None, None]
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def lightning_mixer(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k = (silu(h @ w[p + n].T).reshape(T, H, m["dim"]) for n in "qk")
    v = silu(h @ w[p + "v"].T).reshape(T, H, m["vdim"])
    o = lightning_core(q, k, v, m["decay"]).reshape(T, -1)
    return (rms(o, eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def sink_attention(q, k, v, scale, sink):
    """``q, k [T, H, dk]``, ``v [T, H, dv]``: all keys up to the query, one extra term exp(sink_h) in the denominator."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for i in range(T):
        s = torch.einsum("hd,jhd->hj", q[i], k[:i + 1]) * scale
        top = torch.maximum(s.max(-1).values, sink)[:, None]
        e = torch.exp(s - top)
        out[i] = torch.einsum("hj,jhd->hd", e, v[:i + 1]) / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None] - top))
    return out


def latent_keys(c, kr, uk, H):
    """Per head: the unrotated key from the latent, then the rotated part all heads share."""
    T = c.shape[0]
    return torch.cat([(c @ uk.T).reshape(T, H, -1), kr[:, None, :].expand(T, H, kr.shape[-1])], -1)


def latent_mixer(h, w, p, m, eps):
    T, H, d, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    q = (h @ w[p + "q"].T).reshape(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :m["kv_rank"]], eps) * w[p + "dkv.norm"]
    kr = rotate_pairs(down[:, None, m["kv_rank"]:], m["rot"]["base"], m["rot"]["dims"])[:, 0]
    q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], m["rot"]["base"], m["rot"]["dims"])], -1)
    v = (c @ w[p + "uv"].T).reshape(T, H, m["vdim"])
    o = sink_attention(q, latent_keys(c, kr, w[p + "uk"], H), v, m["scale"], w[p + "sink"])
    return o.reshape(T, -1) @ w[p + "o"].T


MIXERS = {"attention": differential_mixer, "lightning": lightning_mixer, "latent_attention": latent_mixer}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits ``[T, vocab]``; ``layers_out`` (a list) receives the residual stream after every layer."""
    w = {n: t.to(F) for n, t in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps)
        x = rms(alpha * x + y, eps) * w[p + "norm1"]
        if layer["mlp"] is not None:
            y = relu2(x @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T
            x = rms(alpha * x + y, eps) * w[p + "norm2"]
        if layers_out is not None:
            layers_out.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T


def shapes(cfg):
    W, s = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        s[p + "norm1"] = (W,)
        H = m["heads"]
        x = p + "mix."
        if layer["type"] == "lightning":
            s |= {x + "q": (H * m["dim"], W), x + "k": (H * m["dim"], W), x + "v": (H * m["vdim"], W),
                  x + "g": (H * m["vdim"], W), x + "o": (W, H * m["vdim"]), x + "norm": (H * m["vdim"],)}
        elif layer["type"] == "attention":
            G, d, v = m["kv_heads"], m["dim"], m["vdim"]
            s |= {x + "q": (2 * H * d, W), x + "q.b": (2 * H * d,), x + "k": (2 * G * d, W), x + "k.b": (2 * G * d,),
                  x + "v": (G * v, W), x + "v.b": (G * v,), x + "q.norm": (d,), x + "k.norm": (d,), x + "g": (H * v, W),
                  x + "o": (W, H * v), x + "o.b": (W,)} | {x + n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")}
        else:
            d, r, v, c = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            s |= {x + "q": (H * (d + r), W), x + "dkv": (c + r, W), x + "dkv.norm": (c,), x + "uk": (H * d, c),
                  x + "uv": (H * v, c), x + "sink": (H,), x + "o": (W, H * v)}
        if layer["mlp"] is not None:
            s[p + "norm2"] = (W,)
            s |= {p + "mlp.up": (layer["mlp"]["ff"], W), p + "mlp.down": (W, layer["mlp"]["ff"])}
    return s


def random_weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        r, last = torch.randn(shape, generator=g, dtype=torch.float32), name.rsplit(".", 1)[-1]
        if last.startswith("norm"):
            r = 1.0 + 0.2 * r
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            r = r * 0.3
        elif last == "b":
            r = r * 0.5
        elif last == "sink":
            r = 1.0 + r
        elif last == "embed":
            r = r * 0.3
        else:
            r = r * shape[-1] ** -0.5 * 1.5
        out[name] = r
    return out
