"""Plain, slow implementation of the Rerupel decoder on whole sequences: no cache, no batching, one function per
mechanism, nothing shared with the product code. Everything runs in the dtype of `w` (the tests use float64).

Notation: T tokens, W width, H heads, d query / key size, e value size, R size of the latent.
"""
from __future__ import annotations

import json
import math
import struct

import torch


def rms(x, eps):
    """x over the root of its mean square (plus eps under the root) along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def bigram_rows(tokens, mul_prev, mul_cur, buckets):
    """Table row of every position: a hash of the token and the one before it; the extra last row where there is none."""
    out = []
    for t, cur in enumerate(tokens):
        out.append((tokens[t - 1] * mul_prev + cur * mul_cur) % buckets if t else buckets)
    return out


def embedding(tokens, w, cfg):
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    bg = cfg["embedding"].get("bigram")
    if bg:
        x = x + w["bigram"][torch.tensor(bigram_rows(tokens, bg["mul_prev"], bg["mul_cur"], bg["buckets"]))]
    return x


def attend(q, k, v, scale):
    """q, k [T, H, d], v [T, H, e]: softmax over every earlier position and the own one."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    seen = torch.ones(T, T, dtype=torch.bool).tril()
    for h in range(H):
        sc = ((q[:, h] @ k[:, h].T) * scale).masked_fill(~seen, -math.inf)
        p = torch.exp(sc - sc.max(dim=1, keepdim=True).values)
        out[:, h] = (p / p.sum(dim=1, keepdim=True)) @ v[:, h]
    return out


def latent(h, w, p, eps):
    return norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)


def latent_attention(h, w, p, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    c = latent(h, w, p, eps)
    q = (h @ w[p + "q"].T).view(T, H, d)
    k, v = (c @ w[p + "uk"].T).view(T, H, d), (c @ w[p + "uv"].T).view(T, H, e)
    o = attend(q, k, v, m["scale"]).reshape(T, H * e)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def dense(h, w, p):
    a = (h @ w[p + "up"].T).clamp_min(0.0)
    return (a * a) @ w[p + "down"].T


def clipped_glu(g, u, limit):
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(h, w, p, limit):
    return clipped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def route(h, w_router, top, scale):
    """Weights [T, E], zero for the experts a token does not use."""
    s = sigmoid(h @ w_router.T)
    best = s.topk(top, dim=1).indices
    return torch.zeros_like(s).scatter(1, best, s.gather(1, best)) * scale


def choice_gaps(z, top):
    """How far the last chosen router logit of every row lies above the first one left out."""
    best = z.sort(dim=1, descending=True).values
    return best[:, top - 1] - best[:, top] if top < z.shape[1] else torch.full((z.shape[0],), 9.0, dtype=z.dtype)


def mixture(h, w, p, mlp, gaps=None):
    r = mlp["router"]
    if gaps is not None:
        gaps.append(choice_gaps(h @ w[p + "router"].T, r["top"]))
    weights = route(h, w[p + "router"], r["top"], r["scale"])
    y = torch.zeros_like(h)
    for e in range(r["experts"]):
        y = y + weights[:, e:e + 1] * expert(h, w, p + f"e{e}.", mlp["expert"]["limit"])
    if mlp.get("shared"):
        y = y + expert(h, w, p + "shared.", mlp["shared"]["limit"])
    return y


def feed_forward(h, w, p, mlp, gaps=None):
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp, gaps)


def layer(x, w, i, cfg, gaps=None):
    spec, p, eps, m = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"], cfg["residual_mult"]
    y = latent_attention(norm(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps)
    x = x + m * (y * w[p + "ls1"])
    if spec["mlp"] is not None:
        x = x + m * (feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp.", spec["mlp"], gaps) * w[p + "ls2"])
    return x


def layer_runs(cfg):
    """(layer, whether a pass of the loop starts ahead of it), in the order they run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    body = [(i, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return [(i, False) for i in range(lp["start"])] + body * lp["times"] + [(i, False) for i in range(lp["stop"], n)]


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def forward(cfg, w, tokens, layers_out=None, gaps=None):
    """Logits [T, vocab] of one sequence. `layers_out`, a list, receives the residual stream after every layer run, `gaps`
    the margin of every router's choice."""
    x0 = x = embedding(tokens, w, cfg)
    for i, enters in layer_runs(cfg):
        if enters:
            x = torch.cat([x, x0], dim=1) @ w["loop.in"].T
        x = layer(x, w, i, cfg, gaps)
        if layers_out is not None:
            layers_out.append(x)
    return softcap(norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T, cfg["logit_softcap"])


# ------------------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------------------


def layer_spec(heads, dim, vdim, rank, mlp=None, scale=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": dim ** -0.5 if scale is None else scale}}


def dense_spec(ff):
    return {"kind": "dense", "ff": ff}


def moe_spec(experts, top, ff, limit=2.0, scale=1.0, shared=None):
    """`shared`: (ff, limit) or None."""
    out = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff, "limit": limit}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def config(width, vocab, layers, loop=None, bigram=(97, 7, 3), eps=1e-5, scale=2.0, mult=0.7, cap=12.0):
    """`loop`: (start, stop, times); `bigram`: (buckets, mul_prev, mul_cur)."""
    out = {"architecture": "Rerupel", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult,
           "logit_softcap": cap, "vocab": vocab, "width": width}
    if bigram is not None:
        out["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


def random_weights(cfg, seed=0, sharp=1.0):
    """Checkpoint tensors by name, rounded to bfloat16 values (held in float32). `sharp` scales the query projections, so
    that single scores stand out. Routers mostly look at one channel per expert, where every token's embedding has the same
    levels in an order of its own and the layers add little: choices vary with the token and are no close calls, which
    rounding could decide either way."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std):
        return torch.randn(*shape, generator=g) * std

    W = cfg["width"]
    w = {"embed": rnd(cfg["vocab"], W, std=0.5), "final.norm": 1 + rnd(W, std=0.2)}
    if cfg["embedding"].get("bigram"):
        w["bigram"] = rnd(cfg["embedding"]["bigram"]["buckets"] + 1, W, std=0.5)
    if cfg.get("loop"):
        w["loop.in"] = torch.cat([torch.eye(W) * 0.8, torch.eye(W) * 0.3], 1) + rnd(W, 2 * W, std=0.3 * W ** -0.5)
    C = max([s["mlp"]["router"]["experts"] for s in cfg["layers"] if s["mlp"] and s["mlp"]["kind"] == "moe"], default=0)
    assert C <= W // 2
    if C > 1:
        levels = torch.linspace(-10.0, 10.0, C) / cfg["embedding"]["scale"]
        w["embed"][:, :C] = torch.stack([levels[torch.randperm(C, generator=g)] for _ in range(cfg["vocab"])])
        w["final.norm"][:C] = 0.02                    # the logits do not see them
        if "bigram" in w:
            w["bigram"][:, :C] = 0
        if "loop.in" in w:
            w["loop.in"][:C] = torch.cat([torch.eye(W) * 0.8, torch.eye(W) * 0.3], 1)[:C]
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        H, d, e, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        for name in ("norm1", "norm2") if spec["mlp"] else ("norm1",):
            w[p + name] = 1 + rnd(W, std=0.2)
            w[p + name][:C] = 1.0
        for name in ("ls1", "ls2") if spec["mlp"] else ("ls1",):
            w[p + name] = 1 + rnd(W, std=0.3)
            w[p + name][:C] = 0.02
        for name, rows, cols, std in (("q", H * d, W, sharp), ("dkv", R, W, 1), ("uk", H * d, R, 1), ("uv", H * e, R, 1), ("g", H * e, W, 1), ("o", W, H * e, 1)):
            w[p + "mix." + name] = rnd(rows, cols, std=std * cols ** -0.5)
        w[p + "mix.dkv.norm"] = 1 + rnd(R, std=0.2)
        mlp = spec["mlp"]
        if mlp is None:
            continue

        def ff(q, f, names):
            for n in names:
                w[q + n] = rnd(f, W, std=1.5 * W ** -0.5)
            w[q + "down"] = rnd(W, f, std=f ** -0.5)

        if mlp["kind"] == "dense":
            ff(p + "mlp.", mlp["ff"], ("up",))
        else:
            E = mlp["router"]["experts"]
            w[p + "mlp.router"] = rnd(E, W, std=0.03 * W ** -0.5)
            w[p + "mlp.router"][:, :E] += 1.5 * torch.eye(E)[torch.randperm(E, generator=g)]
            for j in range(E):
                ff(p + f"mlp.e{j}.", mlp["expert"]["ff"], ("gate", "up"))
            if mlp.get("shared"):
                ff(p + "mlp.shared.", mlp["shared"]["ff"], ("gate", "up"))
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
