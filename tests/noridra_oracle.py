"""Plain, slow implementation of the Noridra decoder on whole sequences: no cache, no batching, one function per mechanism,
nothing shared with the product code. Everything runs in the dtype of `w` (the tests use float64).

Notation: T tokens, W width, H heads, G key heads, d query / key size, e value size, C channels, N states of a channel.
"""
from __future__ import annotations

import json
import math
import struct

import torch


def rms(x, eps):
    """x over the root of its mean square (plus eps under the root) along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, w, groups, eps):
    """RMS norm of each of `groups` equal runs of columns by itself, one weight per column."""
    return rms(x.reshape(*x.shape[:-1], groups, -1), eps).reshape(x.shape) * w


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def unit(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def conv(x, w):
    """x [T, C], w [C, taps]: the last tap weighs a row itself, the ones before it the rows before; zeros ahead of the first."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


def embedding(tokens, w):
    return w["embed"][torch.as_tensor(tokens, dtype=torch.long)] + w["pos"][:len(tokens)]


def delta_recurrence(q, k, v, g, beta, state=None):
    """q, k [T, H, d], v [T, H, e], g and beta [T, H]; S [H, d, e] decays, moves its answer to k towards v, answers q. Returns
    (answers, last S)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty_like(v)
    for t in range(T):
        S = S * g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None]
        o[t] = torch.einsum("hde,hd->he", S, q[t])
    return o, S


def delta(h, w, p, m, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q, k = (unit(x.view(T, G, d)).repeat_interleave(H // G, dim=1) for x in (q, k))
    beta = sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o, _ = delta_recurrence(q * d ** -0.5, k, v.view(T, H, e), g, beta)
    o = (rms(o, eps) * w[p + "norm"]).reshape(T, H * e)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def visible(T, chunk):
    """[T, T]: row i sees itself and the positions before it in its own chunk, chunks counted from position 0."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    return (j <= i) & (torch.div(i, chunk, rounding_mode="floor") == torch.div(j, chunk, rounding_mode="floor"))


def attend(q, k, v, scale, cap, r1, r2, chunk, sink=True):
    """q [T, H, d], k [T, G, d], v [T, G, e]. Scores are capped, lose r1 ln(1 + r2 distance), and share their softmax with a score
    of zero that has no value."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    gap = (torch.arange(T)[:, None] - torch.arange(T)[None]).clamp_min(0).to(q.dtype)
    seen = visible(T, chunk)
    for n in range(H):
        sc = (q[:, n] @ k[:, n // per].T) * scale
        if cap:
            sc = cap * torch.tanh(sc / cap)
        sc = sc - r1[n] * torch.log(1 + r2[n] * gap)
        p = torch.exp(sc).masked_fill(~seen, 0.0)
        out[:, n] = (p / ((1.0 if sink else 0.0) + p.sum(dim=1, keepdim=True))) @ v[:, n // per]
    return out


def attention(h, w, p, m, eps):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = (h @ w[p + "q"].T).view(T, H, d), (h @ w[p + "k"].T).view(T, G, d)
    o = attend(rms(q, eps) * w[p + "q.norm"], rms(k, eps) * w[p + "k.norm"], k, m["scale"], m["softcap"], w[p + "r1"], w[p + "r2"], m["mask"]["size"])
    return (o.reshape(T, H * d) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def scan(dt, A, x, B, C, D, state=None):
    """dt, x [T, C], A [C, N], B, C [T, N], D [C]: every channel's N states decay by exp(dt A) and take up dt x B; read by C.
    Returns (y, last S)."""
    T = x.shape[0]
    S = torch.zeros_like(A) if state is None else state.clone()
    y = torch.empty_like(x)
    for t in range(T):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def mamba1(h, w, p, m, eps):
    inner, n, r = m["inner"], m["state"], m["dt_rank"]
    xz = h @ w[p + "in"].T
    x = silu(conv(xz[:, :inner], w[p + "conv"]) + w[p + "conv.b"])
    f = x @ w[p + "x"].T
    dt = softplus(f[:, :r] @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = scan(dt, -torch.exp(w[p + "A_log"]), x, f[:, r:r + n], f[:, r + n:], w[p + "D"])
    return (y * silu(xz[:, inner:])) @ w[p + "o"].T


def expert(x, w, p):
    return (silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def mixture(h, w, p, mlp, gaps=None):
    """Every token's `top` experts of the largest sigmoid scores read the token times the score. `gaps` receives by how much of
    a logit the last choice led."""
    top, n = mlp["router"]["top"], mlp["router"]["experts"]
    z = h @ w[p + "router"].T
    order = z.sort(dim=1, descending=True)
    if gaps is not None and top < n:
        gaps.append(order.values[:, top - 1] - order.values[:, top])
    s = torch.zeros_like(z).scatter(1, order.indices[:, :top], sigmoid(order.values[:, :top]))
    y = torch.zeros_like(h)
    for j in range(n):
        used = s[:, j] != 0
        y[used] = y[used] + expert(s[used, j][:, None] * h[used], w, p + f"e{j}.")
    return y


MIXERS = {"delta": delta, "attention": attention, "mamba1": mamba1}


def layer(x, w, i, cfg, gaps=None):
    spec, p, eps, groups = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"], cfg["norm"]["groups"]
    h = x + conv(x, w[p + "canon1"])
    y = MIXERS[spec["type"]](h, w, p + "mix.", spec["mixer"], eps)
    x = group_norm(cfg["postln_alpha"] * x + w[p + "ls1"] * y, w[p + "norm1"], groups, eps)
    if spec["mlp"] is not None:
        h = x + conv(x, w[p + "canon2"])
        x = group_norm(cfg["postln_alpha"] * x + w[p + "ls2"] * mixture(h, w, p + "mlp.", spec["mlp"], gaps), w[p + "norm2"], groups, eps)
    return x


def forward(cfg, w, tokens, layers_out=None, gaps=None):
    """Logits [T, vocab] of one sequence. `layers_out`, a list, receives the residual stream after every layer."""
    x = embedding(tokens, w)
    for i in range(len(cfg["layers"])):
        x = layer(x, w, i, cfg, gaps)
        if layers_out is not None:
            layers_out.append(x)
    return group_norm(x, w["final.norm"], cfg["norm"]["groups"], cfg["norm"]["eps"]) @ w["head"].T


# ------------------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------------------


def delta_spec(heads, kv_heads, dim, vdim, taps, mlp=None):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps}}


def attention_spec(heads, kv_heads, dim, chunk, cap, mlp=None, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk}, "softcap": cap,
                      "scale": 1.2 * dim ** -0.5 if scale is None else scale}}


def mamba_spec(inner, state, dt_rank, taps, mlp=None):
    return {"type": "mamba1", "mlp": mlp, "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": taps}}


def moe_spec(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def config(width, vocab, layers, groups=1, taps=4, alpha=1.5, eps=1e-5, positions=512):
    return {"architecture": "Noridra", "canon": {"taps": taps}, "layers": layers, "max_positions": positions, "norm": {"eps": eps, "groups": groups},
            "postln_alpha": alpha, "vocab": vocab, "width": width}


def layer_tensors(spec, width, taps):
    """{name: (shape, kind)} of one layer; kind is "mat", "one" (a weight around one), "sharp" (a query norm), "conv", "scale",
    "rate", "step", "router", "bias"."""
    m, out = spec["mixer"], {"norm1": ((width,), "one"), "ls1": ((width,), "scale"), "canon1": ((width, taps), "conv")}
    if spec["type"] == "delta":
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows in (("q", G * d), ("k", G * d), ("v", H * e)):
            out.update({f"mix.{n}": ((rows, width), "mat"), f"mix.{n}.conv": ((rows, m["conv"]), "conv")})
        out.update({"mix.b": ((H, width), "mat"), "mix.A_log": ((H,), "rate"), "mix.norm": ((e,), "one"), "mix.a": ((H, width), "mat"),
                    "mix.dt_bias": ((H,), "step"), "mix.g": ((H * e, width), "mat"), "mix.o": ((width, H * e), "mat")})
    elif spec["type"] == "attention":
        H, G, d = m["heads"], m["kv_heads"], m["dim"]
        out.update({"mix.q": ((H * d, width), "mat"), "mix.k": ((G * d, width), "mat"), "mix.q.norm": ((d,), "sharp"), "mix.k.norm": ((d,), "one"),
                    "mix.r1": ((H,), "r1"), "mix.r2": ((H,), "r2"), "mix.g": ((H * d, width), "mat"), "mix.o": ((width, H * d), "mat")})
    else:
        I, n, r = m["inner"], m["state"], m["dt_rank"]
        out.update({"mix.in": ((2 * I, width), "mat"), "mix.conv": ((I, m["conv"]), "conv"), "mix.conv.b": ((I,), "bias"), "mix.x": ((r + 2 * n, I), "mat"),
                    "mix.dt": ((I, r), "mat"), "mix.dt.b": ((I,), "step"), "mix.A_log": ((I, n), "rate"), "mix.D": ((I,), "one"), "mix.o": ((width, I), "mat")})
    if spec["mlp"] is not None:
        out.update({"norm2": ((width,), "one"), "ls2": ((width,), "scale"), "canon2": ((width, taps), "conv")})
        r, f = spec["mlp"]["router"], spec["mlp"]["expert"]["ff"]
        out["mlp.router"] = ((r["experts"], width), "router")
        for j in range(r["experts"]):
            out.update({f"mlp.e{j}.gate": ((f, width), "mat"), f"mlp.e{j}.up": ((f, width), "mat"), f"mlp.e{j}.down": ((width, f), "mat")})
    return out


def random_weights(cfg, seed=0, sharp=1.0):
    """Checkpoint tensors by name, rounded to bfloat16 values (held in float32). `sharp` scales the queries, so that single
    scores stand out. Routers look at one channel per expert, where every token's embedding has the same levels in an order of
    its own and the layers add nothing: choices vary with the token and are no close calls, which rounding could decide
    either way."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0):
        return torch.randn(*shape, generator=g) * std

    W, taps = cfg["width"], cfg["canon"]["taps"]
    w = {"embed": rnd(cfg["vocab"], W), "pos": rnd(cfg["max_positions"], W, std=0.4), "head": rnd(cfg["vocab"], W), "final.norm": 1 + rnd(W, std=0.2)}
    E = max([s["mlp"]["router"]["experts"] for s in cfg["layers"] if s["mlp"]], default=0)
    assert E <= W // cfg["norm"]["groups"]        # the levels stay in one group of the norm
    if E:
        levels = torch.linspace(-1.8, 1.8, E)
        w["embed"][:, :E] = torch.stack([levels[torch.randperm(E, generator=g)] for _ in range(cfg["vocab"])])
        w["pos"][:, :E] = 0.0
    for i, spec in enumerate(cfg["layers"]):
        for name, (shape, kind) in layer_tensors(spec, W, taps).items():
            if kind in ("one", "sharp"):
                t = (1 + rnd(*shape, std=0.2)) * (sharp if kind == "sharp" else 1.0)
            elif kind == "scale":
                t = 0.8 + rnd(*shape, std=0.2)
            elif kind == "conv":
                t = rnd(*shape, std=0.5 * shape[1] ** -0.5 if name.startswith("canon") else shape[1] ** -0.5)
            elif kind == "rate":
                t = torch.rand(*shape, generator=g) * 5.0 - 4.0
            elif kind == "step":
                t = rnd(*shape) - 2.5
            elif kind == "bias":
                t = rnd(*shape, std=0.2)
            elif kind in ("r1", "r2"):
                t = torch.rand(*shape, generator=g) * (1.5 if kind == "r1" else 0.6) + 0.02
            elif kind == "router":
                t = rnd(*shape, std=0.02 * W ** -0.5)
                t[:, :shape[0]] += torch.eye(shape[0])[torch.randperm(shape[0], generator=g)] * 0.7 * max(E, 4)
            else:
                t = rnd(*shape, std=shape[-1] ** -0.5)
            if E and name in ("norm1", "norm2"):
                t[:E] = 1.0
            if E and name.startswith("canon"):
                t[:E] *= 0.02
            if E and name.startswith("ls"):
                t[:E] = 0.0
            w[f"l{i}.{name}"] = t
    if E:
        w["final.norm"][:E] = 0.02                    # the logits do not see them
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
