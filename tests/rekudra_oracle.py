"""Plain, slow implementation of the Rekudra decoder on whole sequences: no cache, no batching, one function per
mechanism, nothing shared with the product code. Everything runs in the dtype of `w` (the tests use float64).

Notation: T tokens, W width, H query heads, G key/value heads, d key size, e value size, s residual streams.
"""
from __future__ import annotations

import json
import math
import struct

import torch


def rms(x, eps):
    """x over the root of its mean square (plus eps under the root) along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_zero_centred(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0.0)


def causal_conv(u, w):
    """u [T, C], w [C, n]: y[t, c] = sum_j w[c, j] u[t - n + 1 + j, c], zeros before the start."""
    T, C = u.shape
    n = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(n):
            src = t - n + 1 + j
            if src >= 0:
                y[t] += w[:, j] * u[src]
    return y


def rope_frequencies(rot):
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            wavelength = 2.0 * math.pi / f
            lo, hi, orig, factor = sc["low"], sc["high"], sc["original"], sc["factor"]
            if wavelength < orig / hi:
                pass
            elif wavelength > orig / lo:
                f = f / factor
            else:
                mix = (orig / wavelength - lo) / (hi - lo)
                f = (1.0 - mix) * f / factor + mix * f
        out.append(f)
    return out


def rotate(x, rot, first_pos=0):
    """x [T, heads, d]: pairs (i, i + dims / 2) turned by position * frequency."""
    half = rot["dims"] // 2
    freq = torch.tensor(rope_frequencies(rot), dtype=torch.float64)
    ang = torch.arange(first_pos, first_pos + x.shape[0], dtype=torch.float64)[:, None] * freq[None]
    c, s = ang.cos().to(x.dtype)[:, None], ang.sin().to(x.dtype)[:, None]
    y = x.clone()
    a, b = x[..., :half], x[..., half:2 * half]
    y[..., :half] = a * c - b * s
    y[..., half:2 * half] = b * c + a * s
    return y


def attend(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, e]: ordinary causal softmax attention, head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    for h in range(H):
        sc = (q[:, h] @ k[:, h // per].T) * scale
        sc = sc.masked_fill(~mask, -math.inf)
        p = torch.exp(sc - sc.max(dim=1, keepdim=True).values)
        out[:, h] = (p / p.sum(dim=1, keepdim=True)) @ v[:, h // per]
    return out


def attention_keys_values(h, w, p, m, eps):
    """Keys (convolved, rotated, normalised) and values (convolved) of a layer with projections of its own."""
    T = h.shape[0]
    k = causal_conv(h @ w[p + "k"].T, w[p + "k.conv"]).view(T, m["kv_heads"], m["dim"])
    v = causal_conv(h @ w[p + "v"].T, w[p + "v.conv"]).view(T, m["kv_heads"], m["vdim"])
    return rms(rotate(k, m["rot"]), eps), v


def attention(h, w, p, m, eps, kv):
    T = h.shape[0]
    q = causal_conv(h @ w[p + "q"].T, w[p + "q.conv"]).view(T, m["heads"], m["dim"])
    q = rms(rotate(q, m["rot"]), eps)
    o = attend(q, kv[0], kv[1], m["scale"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].T


def delta_rule(q, k, v, g, beta, s0=None):
    """Gated delta rule with one decay per key channel. q, k, g [T, H, d], v [T, H, e], beta [T, H]; S [H, d, e]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if s0 is None else s0.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    return out, S


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_decay(h, w, p, heads, dim):
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    rate = torch.exp(w[p + "A_log"])[None, :, None]
    return torch.exp(-rate * softplus(z).view(-1, heads, dim))


def channel_delta(h, w, p, m, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(causal_conv(h @ w[p + "q"].T, w[p + "q.conv"])).view(T, G, d)
    k = silu(causal_conv(h @ w[p + "k"].T, w[p + "k.conv"])).view(T, G, d)
    v = silu(causal_conv(h @ w[p + "v"].T, w[p + "v.conv"])).view(T, H, e)
    q, k = unit(q) * d ** -0.5, unit(k)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = sigmoid(h @ w[p + "b"].T)
    o, _ = delta_rule(q, k, v, delta_decay(h, w, p, H, d), beta)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, e)
    o = rms(o, eps) * w[p + "norm"] * gate
    return o.reshape(T, -1) @ w[p + "o"].T


def feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def hyper_read(x, w, p):
    """x [s, T, W] -> the sublayer's input [T, W]."""
    return torch.einsum("s,stw->tw", w[p + "in"], x)


def hyper_write(x, w, p, y):
    """All streams at once from the old ones: mix is indexed [from, to]."""
    return torch.einsum("st,snw->tnw", w[p + "mix"], x) + w[p + "out"][:, None, None] * y[None]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence. `layers_out`, a list, receives the sum of the streams after every layer."""
    eps = cfg["norm"]["eps"]
    emb = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    x = torch.stack([emb] * cfg["streams"])
    shared = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = norm_zero_centred(hyper_read(x, w, p + "hc1."), w[p + "norm1"], eps)
        if layer["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                shared[i] = attention_keys_values(h, w, p + "mix.", m, eps)
            y = attention(h, w, p + "mix.", m, eps, shared[i if src is None else src])
        elif layer["type"] == "channel_delta":
            y = channel_delta(h, w, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = hyper_write(x, w, p + "hc1.", y)
        if layer["mlp"] is not None:
            h = norm_zero_centred(hyper_read(x, w, p + "hc2."), w[p + "norm2"], eps)
            x = hyper_write(x, w, p + "hc2.", feed_forward(h, w, p + "mlp."))
        if layers_out is not None:
            layers_out.append(x.sum(0))
    return norm_zero_centred(x.sum(0), w["final.norm"], eps) @ w["head"].T


# ------------------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------------------


def layer_attention(heads, kv_heads, dim, vdim, rot_dims, taps=4, kv_from=None, ff=None, scale=None, base=10000.0, scaling=None):
    m = {"conv": taps, "dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
         "rot": {"base": base, "dims": rot_dims}}
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


def layer_delta(heads, kv_heads, dim, vdim, taps=4, ff=None):
    return {"type": "channel_delta", "mixer": {"conv": taps, "dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim},
            "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


def config(width, vocab, streams, layers, eps=1e-5, scale=3.0):
    return {"architecture": "Rekudra", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "streams": streams,
            "vocab": vocab, "width": width}


def random_weights(cfg, seed=0, a_rank=12, g_rank=20, decay=0.0):
    """Checkpoint tensors by name, rounded to bfloat16 values (held in float32). `decay` shifts dt_bias: negative
    values make the recurrent state live longer."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std):
        return torch.randn(*shape, generator=g) * std

    W, s = cfg["width"], cfg["streams"]
    w = {"embed": rnd(cfg["vocab"], W, std=0.5), "head": rnd(cfg["vocab"], W, std=W ** -0.5), "final.norm": rnd(W, std=0.1)}

    def hyper(p):
        w[p + "in"] = 1.0 / s + rnd(s, std=0.3)
        w[p + "out"] = 1.0 + rnd(s, std=0.3)
        w[p + "mix"] = torch.eye(s) + rnd(s, s, std=0.2)

    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        w[p + "norm1"] = rnd(W, std=0.2)
        hyper(p + "hc1.")
        H, G, d, e, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]

        def proj(name, rows, taps=n):
            w[q + name] = rnd(rows, W, std=W ** -0.5)
            if taps:
                w[q + name + ".conv"] = rnd(rows, taps, std=0.6)

        if layer["type"] == "attention":
            proj("q", H * d)
            if "kv_from" not in m:
                proj("k", G * d)
                proj("v", G * e)
            proj("g", H, 0)
        else:
            proj("q", G * d)
            proj("k", G * d)
            proj("v", H * e)
            proj("b", H, 0)
            w[q + "A_log"] = rnd(H, std=0.5)
            w[q + "norm"] = 1.0 + rnd(e, std=0.2)
            w[q + "a1"], w[q + "a2"] = rnd(a_rank, W, std=W ** -0.5), rnd(H * d, a_rank, std=a_rank ** -0.5)
            w[q + "dt_bias"] = rnd(H * d, std=1.0) - 2.0 + decay
            w[q + "g1"], w[q + "g2"] = rnd(g_rank, W, std=W ** -0.5), rnd(H * e, g_rank, std=g_rank ** -0.5)
        w[q + "o"] = rnd(W, H * e, std=(H * e) ** -0.5)
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            w[p + "norm2"] = rnd(W, std=0.2)
            hyper(p + "hc2.")
            w[p + "mlp.gate"], w[p + "mlp.up"] = rnd(f, W, std=W ** -0.5), rnd(f, W, std=W ** -0.5)
            w[p + "mlp.down"] = rnd(W, f, std=f ** -0.5)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}


def as_double(w):
    return {k: v.double() for k, v in w.items()}


def write_checkpoint(path, cfg, w):
    """config.json + model.safetensors (bfloat16), written byte by byte."""
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    head, blobs, off = {}, [], 0
    for name, t in w.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(path / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))


def relative_error(got, want):
    """Per position: RMS over the vocabulary of the mean-free difference, over the RMS of the mean-free logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    c = want.double() - want.double().mean(-1, keepdim=True)
    return (d * d).mean(-1).sqrt() / (c * c).mean().sqrt()
