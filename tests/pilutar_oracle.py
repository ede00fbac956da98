"""Plain, slow implementation of the Pilutar decoder on whole sequences: no cache, no batching, one function per mechanism,
nothing shared with the product code. Everything runs in the dtype of `w` (the tests use float64).

Notation: T tokens, W width, H heads, G key / value heads, d query / key size, e value size, R size of the latent.
"""
from __future__ import annotations

import json
import math
import struct

import torch


def rms(x, eps):
    """x over the root of its mean square (plus eps under the root) along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def log_sigmoid(x):
    """-log(1 + e^-x), without overflow."""
    return -(torch.clamp(-x, min=0) + torch.log1p(torch.exp(-x.abs())))


def silu(x):
    return x * sigmoid(x)


def relu2(x):
    return x.clamp_min(0.0) ** 2


def softcap(z, cap):
    return z if cap is None else cap * torch.tanh(z / cap)


def embedding(tokens, w, cfg):
    return w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]


def angles(T, dims, base, dtype):
    """[T, dims / 2]: position times base^(-2 i / dims)."""
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    return (torch.arange(T, dtype=torch.float64)[:, None] * f[None]).to(dtype)


def rotate(x, dims, base, interleaved):
    """x [T, H, d]: the first `dims` columns turn, in neighbouring pairs (2 i, 2 i + 1) or in pairs (i, i + dims / 2)."""
    a = angles(x.shape[0], dims, base, x.dtype)[:, None]
    out = x.clone()
    u, v = (slice(0, dims, 2), slice(1, dims, 2)) if interleaved else (slice(0, dims // 2), slice(dims // 2, dims))
    out[..., u] = x[..., u] * torch.cos(a) - x[..., v] * torch.sin(a)
    out[..., v] = x[..., v] * torch.cos(a) + x[..., u] * torch.sin(a)
    return out


def visible(T, window):
    """[T, T]: row i sees itself and the window - 1 positions before it (None: all earlier ones)."""
    gap = torch.arange(T)[:, None] - torch.arange(T)[None]
    return (gap >= 0) & (gap < (window if window is not None else T))


def attend(q, k, v, scale, window=None, cap=None):
    """q [T, H, d], k [T, G, d], v [T, G, e]: softmax over the visible positions; H / G query heads share a key head."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    seen = visible(T, window)
    for h in range(H):
        sc = softcap((q[:, h] @ k[:, h // per].T) * scale, cap).masked_fill(~seen, -math.inf)
        p = torch.exp(sc - sc.max(dim=1, keepdim=True).values)
        out[:, h] = (p / p.sum(dim=1, keepdim=True)) @ v[:, h // per]
    return out


def window_of(m):
    return m["mask"]["size"] if m.get("mask") else None


def latent_attention(h, w, p, m, eps):
    """Keys and values of all heads from one latent per token, plus one rotated key part that the heads share."""
    T, H, d, r, e, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    base = m["rot"]["base"]
    q_rot, k_rot = rotate(q[..., d:], r, base, True), rotate(down[:, None, R:], r, base, True)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), k_rot.expand(T, H, r)], -1)
    o = attend(torch.cat([q[..., :d], q_rot], -1), k, (c @ w[p + "uv"].T).view(T, H, e), m["scale"], window_of(m))
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * e) @ w[p + "o"].T


def grouped_attention(h, w, p, m, eps):
    """Biased projections, one RMS norm over a whole query (key) row, rotated halves, capped scores."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + n].T + w[p + n + ".b"] for n in ("q", "k", "v"))
    q, k = rms_norm(q, w[p + "q.norm"], eps).view(T, H, d), rms_norm(k, w[p + "k.norm"], eps).view(T, G, d)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    o = attend(rotate(q, dims, base, False), rotate(k, dims, base, False), v.view(T, G, e), m["scale"], window_of(m), m.get("softcap"))
    return o.reshape(T, H * e) @ w[p + "o"].T


def decay(h, w, p, tau):
    """Logarithms of the decays, [T, H * d]: log sigmoid of a low-rank map of h, over tau."""
    return log_sigmoid((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]) / tau


def recurrence(q, k, v, log_a, state=None):
    """q, k, log_a [T, H, d], v [T, H, e]: S <- diag(a) S + k v^T, o = S^T q, token by token. Returns (o, last S)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty_like(v)
    for t in range(T):
        for n in range(H):
            S[n] = torch.exp(log_a[t, n])[:, None] * S[n] + k[t, n][:, None] * v[t, n][None]
            o[t, n] = S[n].T @ q[t, n]
    return o, S


def gated_linear_attention(h, w, p, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ w[p + n].T).view(T, H, -1) for n in ("q", "k", "v"))
    o, _ = recurrence(q * d ** -0.5, k, v, decay(h, w, p, m["tau"]).view(T, H, d))
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, H * e)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    left, right = grouped_attention(h, w, p + "left.", m["left"], eps), gated_linear_attention(h, w, p + "right.", m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def dense(h, w, p):
    return ((h @ w[p + "gate"].T).clamp_min(0.0) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p):
    return relu2(h @ w[p + "up"].T) @ w[p + "down"].T


def choice_scores(s, correction, groups, keep):
    """Scores that choose: corrected, minus infinity outside the `keep` groups of neighbours whose best score is largest."""
    c = s + correction
    best = c.view(c.shape[0], groups, -1).max(-1).values
    stays = torch.zeros_like(best, dtype=torch.bool).scatter(1, best.topk(keep, dim=1).indices, True)
    return c.masked_fill(~stays.repeat_interleave(c.shape[1] // groups, dim=1), -math.inf)


def margins(choice, s, n):
    """By how much the n-th best choice leads the next, in units of the two scores (which is what rounding disturbs)."""
    order = choice.argsort(dim=1, descending=True)
    a, b = order[:, n - 1:n], order[:, n:n + 1]
    return ((choice.gather(1, a) - choice.gather(1, b)) / (s.gather(1, a) + s.gather(1, b))).flatten()


def route(z, correction, r, gaps=None):
    """Weights [T, E + identity], zero for what a token does not use. `gaps` receives by how much every choice was made."""
    g = r.get("groups") or {"count": 1, "keep": 1}
    s = torch.exp(z - z.max(1, keepdim=True).values)
    s = s / s.sum(1, keepdim=True)
    c = choice_scores(s, correction, g["count"], g["keep"])
    if gaps is not None:
        if r["top"] < int(torch.isfinite(c[0]).sum()):
            gaps.append(margins(c, s, r["top"]))
        if g["keep"] < g["count"]:
            best = (s + correction).view(len(s), g["count"], -1).max(-1)
            gaps.append(margins(best.values, s.view(len(s), g["count"], -1).gather(2, best.indices[..., None])[..., 0], g["keep"]))
    chosen = c.topk(r["top"], dim=1).indices
    picked = s.gather(1, chosen)
    return torch.zeros_like(s).scatter(1, chosen, picked / (picked.sum(1, keepdim=True) + 1e-20))


def mixture(h, w, p, mlp, gaps=None):
    r = mlp["router"]
    weights = route(h @ w[p + "router"].T, w[p + "correction"], r, gaps)
    y = torch.zeros_like(h)
    for j in range(r["experts"]):
        y = y + weights[:, j:j + 1] * expert(h, w, p + f"e{j}.")
    y = y + weights[:, r["experts"]:].sum(1, keepdim=True) * h
    if mlp.get("shared"):
        y = y + sigmoid(h @ w[p + "shared.sg"].T) * expert(h, w, p + "shared.")
    return y


def feed_forward(h, w, p, mlp, gaps=None):
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp, gaps)


MIXERS = {"latent_attention": latent_attention, "parallel": parallel}


def layer(x, w, i, cfg, gaps=None):
    """Mixer and feed-forward read the same normalised input; both are added."""
    spec, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
    y = MIXERS[spec["type"]](h, w, p + "mix.", spec["mixer"], eps)
    if spec["mlp"] is not None:
        y = y + feed_forward(h, w, p + "mlp.", spec["mlp"], gaps)
    return x + y


def forward(cfg, w, tokens, layers_out=None, gaps=None):
    """Logits [T, vocab] of one sequence. `layers_out`, a list, receives the residual stream after every layer, `gaps` the
    margins of the routers' choices."""
    x = embedding(tokens, w, cfg)
    for i in range(len(cfg["layers"])):
        x = layer(x, w, i, cfg, gaps)
        if layers_out is not None:
            layers_out.append(x)
    return (layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"]) @ w["head"].T) * cfg["logit_scale"]


# ------------------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------------------


def latent_spec(heads, dim, rot_dim, vdim, rank, window, mlp=None, scale=None, base=10000.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}


def parallel_spec(left, right, mlp=None, scales=(0.7, 0.4)):
    """`left`: (heads, kv_heads, dim, vdim, rotated, window, softcap); `right`: (heads, dim, vdim, tau)."""
    H, G, d, e, rot, window, cap = left
    n, dr, er, tau = right
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": e, "mask": {"size": window}, "rot": {"base": 5000.0, "dims": rot},
                               "scale": 1.3 * d ** -0.5, "softcap": cap},
                      "right": {"heads": n, "dim": dr, "vdim": er, "tau": tau}, "left_scale": scales[0], "right_scale": scales[1]}}


def dense_spec(ff):
    return {"kind": "dense", "ff": ff}


def moe_spec(experts, top, ff, groups=(1, 1), identity=0, shared=None):
    out = {"kind": "moe", "router": {"experts": experts, "top": top, "groups": dict(zip(("count", "keep"), groups)), "identity": identity},
           "expert": {"ff": ff}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def config(width, vocab, layers, eps=1e-5, scale=2.0, logit_scale=0.5):
    return {"architecture": "Pilutar", "embedding": {"scale": scale}, "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}


def layer_tensors(spec, width, rank_a):
    """{name: (shape, kind)} of one layer; kind is "mat", "one" (a weight around one), "bias", "sharp" (query projections),
    "decay_bias", "router", "correction"."""
    m, out = spec["mixer"], {"norm1": ((width,), "one"), "norm1.b": ((width,), "bias")}
    if spec["type"] == "latent_attention":
        H, d, r, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        out.update({"mix.q": ((H * (d + r), width), "sharp"), "mix.dkv": ((R + r, width), "mat"), "mix.dkv.norm": ((R,), "one"), "mix.uk": ((H * d, R), "mat"),
                    "mix.uv": ((H * e, R), "mat"), "mix.g": ((H, width), "mat"), "mix.o": ((width, H * e), "mat")})
    else:
        a, b = m["left"], m["right"]
        for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
            out.update({f"mix.left.{n}": ((rows, width), "mat"), f"mix.left.{n}.b": ((rows,), "bias")})
            if n != "v":
                out[f"mix.left.{n}.norm"] = ((rows,), "two" if n == "q" else "one")
        out["mix.left.o"] = ((width, a["heads"] * a["vdim"]), "mat")
        H, d, e = b["heads"], b["dim"], b["vdim"]
        out.update({"mix.right.q": ((H * d, width), "mat"), "mix.right.k": ((H * d, width), "mat"), "mix.right.v": ((H * e, width), "mat"),
                    "mix.right.g": ((H * e, width), "mat"), "mix.right.o": ((width, H * e), "mat"), "mix.right.norm": ((e,), "one"),
                    "mix.right.a1": ((rank_a, width), "mat"), "mix.right.a2": ((H * d, rank_a), "mat"), "mix.right.a2.b": ((H * d,), "decay_bias")})
    mlp = spec["mlp"]
    if mlp is None:
        return out
    if mlp["kind"] == "dense":
        f = mlp["ff"]
        out.update({"mlp.gate": ((f, width), "mat"), "mlp.up": ((f, width), "mat"), "mlp.down": ((width, f), "mat")})
        return out
    r = mlp["router"]
    n = r["experts"] + r.get("identity", 0)
    out.update({"mlp.router": ((n, width), "router"), "mlp.correction": ((n,), "correction")})
    for q, f in [(f"mlp.e{j}", mlp["expert"]["ff"]) for j in range(r["experts"])] + ([("mlp.shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
        out.update({q + ".up": ((f, width), "mat"), q + ".down": ((width, f), "mat")})
    if mlp.get("shared"):
        out["mlp.shared.sg"] = ((1, width), "mat")
    return out


def random_weights(cfg, seed=0, sharp=1.0, rank_a=6):
    """Checkpoint tensors by name, rounded to bfloat16 values (held in float32). `sharp` scales the queries, so that single
    scores stand out. Routers mostly look at one channel per expert, where every token's embedding has the same levels in an
    order of its own and the layers add little, the other channels only differ in sign, and corrections differ by nothing or by more than scores can:
    choices vary with the token and are no close calls, which rounding could decide either way."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std):
        return torch.randn(*shape, generator=g) * std

    W = cfg["width"]
    w = {"embed": rnd(cfg["vocab"], W, std=0.5), "head": rnd(cfg["vocab"], W, std=1.0), "final.norm": 1 + rnd(W, std=0.2), "final.norm.b": rnd(W, std=0.2)}
    C = max([s["mlp"]["router"]["experts"] + s["mlp"]["router"].get("identity", 0) for s in cfg["layers"] if s["mlp"] and s["mlp"]["kind"] == "moe"], default=0)
    assert C <= W // 2
    if C > 1:
        levels = torch.linspace(-3.0, 3.0, C) / cfg["embedding"]["scale"]
        w["embed"] = w["embed"].sign() * 0.5
        w["embed"][:, :C] = torch.stack([levels[torch.randperm(C, generator=g)] for _ in range(cfg["vocab"])])
    for i, spec in enumerate(cfg["layers"]):
        for name, (shape, kind) in layer_tensors(spec, W, rank_a).items():
            full = f"l{i}.{name}"
            if kind in ("one", "two"):
                w[full] = (1 + rnd(*shape, std=0.2)) * (sharp if kind == "two" else 1.0)
            elif kind == "bias":
                w[full] = rnd(*shape, std=0.2)
            elif kind == "decay_bias":
                w[full] = rnd(*shape, std=2.0)
            elif kind == "correction":
                w[full] = torch.randint(-1, 2, shape, generator=g) * 1.5 - 0.2
            elif kind == "router":
                E = shape[0]
                w[full] = rnd(*shape, std=0.03 * W ** -0.5)
                w[full][:, :E] += torch.eye(E)[torch.randperm(E, generator=g)] * 0.2 * max(E, 4)
            else:
                w[full] = rnd(*shape, std=(sharp if kind == "sharp" else 1.0) * shape[-1] ** -0.5)
            if C > 1 and name in ("norm1", "norm1.b"):
                w[full][:C] = 1.0 if name == "norm1" else 0.0
            if C > 1 and (name.endswith(".o") or name.endswith(".down") or name in ("mix.o", "mlp.down")):
                w[full][:C] *= 0.02
    if C > 1:
        w["final.norm"][:C] = 0.02                    # the logits do not see them
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
