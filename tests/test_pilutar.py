"""Pilutar against the plain implementation in `pilutar_oracle`: every mechanism alone, whole prompts, decoding, cut prompts,
mixed batches, pages and state slots used again, and greedy generation through the scheduler. The same tests run on the CPU
engine and, marked `gpu`, on the kernels in f32 and bf16."""
import io
import json

import numpy as np
import pilutar_oracle as P
import pytest
import torch

from mojo_b200 import ops
from mojo_b200.ops import reference
from mojo_b200.pipelines import LLM, PipelineConfig, SamplingParams

gpu = pytest.mark.gpu
TARGETS = [pytest.param(("cpu", "float32"), id="cpu"), pytest.param(("cuda", "float32"), id="f32", marks=gpu),
           pytest.param(("cuda", "bfloat16"), id="bf16", marks=gpu)]
BF16 = ("cuda", "bfloat16")


def model_mixed():
    """Both kinds of layers, every kind of feed-forward and none, sizes that differ from layer to layer."""
    return P.config(96, 101, [
        P.parallel_spec((6, 2, 24, 40, 16, 37, 8.0), (3, 20, 28, 4.0), P.dense_spec(72)),
        P.latent_spec(5, 20, 12, 28, 40, 51, P.moe_spec(7, 3, 40, groups=(3, 2), identity=2, shared=24)),
        P.parallel_spec((4, 4, 16, 16, 8, 64, 20.0), (2, 32, 16, 16.0), P.moe_spec(6, 2, 24, groups=(2, 1)), scales=(0.3, 1.2)),
        P.latent_spec(3, 24, 8, 40, 64, 30, None)])


def model_odd():
    """Sizes that are multiples of nothing much, more query heads per key head than an MMA tile has rows, no groups."""
    return P.config(101, 67, [
        P.latent_spec(20, 13, 6, 21, 90, 70, P.moe_spec(5, 2, 20, shared=9)),
        P.parallel_spec((34, 2, 18, 10, 10, 33, 5.0), (5, 13, 7, 1.0), P.moe_spec(3, 3, 33, identity=4, groups=(7, 3))),
        P.parallel_spec((3, 1, 70, 66, 70, 20, 30.0), (1, 70, 90, 8.0), P.dense_spec(41), scales=(1.0, 1.0))], eps=1e-3, scale=0.7, logit_scale=1.7)


def model_wide():
    """Heads that fill the tensor-core prefill kernel's columns, or only in part; latents that prompts expand."""
    return P.config(256, 200, [
        P.parallel_spec((4, 2, 128, 96, 64, 130, 15.0), (2, 128, 128, 16.0), P.dense_spec(160)),
        P.latent_spec(4, 90, 38, 128, 200, 140, P.moe_spec(8, 2, 48, groups=(2, 1), shared=112)),
        P.latent_spec(2, 64, 40, 72, 256, 200, None)])


def model_parallel_only():
    """No latents: steps with prompt chunks replay CUDA graphs."""
    return P.config(128, 90, [
        P.parallel_spec((2, 1, 128, 128, 128, 100, 25.0), (2, 64, 64, 16.0), P.moe_spec(6, 2, 32, groups=(2, 1), identity=2, shared=32)),
        P.parallel_spec((3, 3, 100, 120, 20, 128, 25.0), (4, 40, 24, 2.0), P.dense_spec(64))])


def model_single():
    """One head, one expert, one group, a window of one; no recurrence at all."""
    return P.config(64, 33, [
        P.latent_spec(1, 8, 2, 8, 16, 1, P.moe_spec(1, 1, 16, shared=16)),
        P.latent_spec(1, 16, 4, 8, 24, 1000, P.dense_spec(16))], scale=1.0, logit_scale=1.0)


MODELS = {"mixed": model_mixed, "odd": model_odd, "wide": model_wide, "parallel_only": model_parallel_only, "single": model_single}
_cache: dict = {}


def weights_of(name):
    cfg = MODELS[name]()
    return cfg, P.random_weights(cfg, seed=len(name), sharp=2.5)


def tokens_of(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def expected(name, tokens):
    """Oracle logits of one sequence in float64, once per (model, tokens). Rounding must not decide which experts run."""
    key = (name, tuple(tokens))
    if key not in _cache:
        cfg, w = weights_of(name)
        gaps = []
        _cache[key] = P.forward(cfg, P.as_double(w), tokens, gaps=gaps)
        assert min((float(x.min()) for x in gaps), default=9.0) > 0.3
    return _cache[key]


def open_llm(tmp_path, name, target, **kw):
    device, dtype = target
    cfg, w = weights_of(name)
    P.write_checkpoint(tmp_path / name, cfg, w)
    kw = {"page_size": 32, "num_pages": 24, "max_num_seqs": 4, "max_num_batched_tokens": 512, "max_model_len": 512, **kw}
    return LLM(PipelineConfig(model=str(tmp_path / name), device=device, dtype=dtype, **kw))


def run_schedule(engine, requests, steps):
    """`steps`: lists of (request, tokens to run). Every position's logits are asked for. Returns {request: [T, vocab]}."""
    ids = {name: i for i, name in enumerate(requests)}
    at = dict.fromkeys(requests, 0)
    out = {name: [] for name in requests}
    for step in steps:
        entries, end = [], []
        for name, n in step:
            entries.append((ids[name], requests[name][at[name]:at[name] + n], list(range(n))))
            at[name] += n
            if at[name] == len(requests[name]):
                end.append(ids[name])
        logits = engine.run_tokens(entries, end).float().cpu()
        row = 0
        for name, n in step:
            out[name].append(logits[row:row + n])
            row += n
    if engine.device.type == "cuda":
        ops.check_status(engine.device)
    assert engine.kv.check_invariants() == ""
    return {name: torch.cat(parts) for name, parts in out.items()}


def check(got, want, target):
    err = P.relative_error(got, want)
    worst, mean = {"float32": (1e-4, 2e-5), "bfloat16": (0.06, 0.02)}[target[1]]
    assert torch.isfinite(got).all()
    assert err.max() < worst and err.mean() < mean, f"worst {err.max():.2e} at {int(err.argmax())}, mean {err.mean():.2e}"


# ------------------------------------------------------------------------------------------------------
# whole model, through the engine
# ------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("name", sorted(MODELS))
@pytest.mark.parametrize("target", TARGETS)
def test_whole_prompts_and_token_by_token(tmp_path, target, name):
    """Requests alone, whole and token by token, one after the other through a pool that holds one of them at a time."""
    cfg, _ = weights_of(name)
    page = 128 if name in ("wide", "parallel_only") else 32
    llm = open_llm(tmp_path, name, target, page_size=page, num_pages=-(-160 // page), max_num_seqs=1)
    for n, seed in ((1, 1), (2, 2), (33, 3), (150, 4)):
        toks = tokens_of(cfg, n, seed)
        check(run_schedule(llm.engine, {"a": toks}, [[("a", n)]])["a"], expected(name, toks), target)
        if n > 1:
            check(run_schedule(llm.engine, {"a": toks}, [[("a", max(1, n - 40))]] + [[("a", 1)]] * min(40, n - 1))["a"], expected(name, toks), target)


@pytest.mark.parametrize("name", sorted(MODELS))
@pytest.mark.parametrize("target", TARGETS)
def test_portions(tmp_path, target, name):
    """Prompts cut into portions of changing size, down to two tokens and to one, across page and window borders."""
    cfg, _ = weights_of(name)
    llm = open_llm(tmp_path, name, target, page_size=128 if name in ("odd", "parallel_only") else 32)
    toks = tokens_of(cfg, 150, 4)
    for cuts in ([2] * 10 + [3] * 5 + [2, 27, 1, 31, 2, 50, 2], [31, 2, 30, 1, 1, 2, 33, 50]):
        assert sum(cuts) == 150
        check(run_schedule(llm.engine, {"a": toks}, [[("a", c)] for c in cuts])["a"], expected(name, toks), target)


@pytest.mark.parametrize("page", [8, 16, 64, 128])
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "wide", "parallel_only"])
def test_unequal_batches_with_reuse(tmp_path, target, name, page):
    """Four live requests in one batch, portions beside decoded tokens, some left out of steps; pages and state slots only fit
    the live ones, so later requests use what others gave back."""
    if name != "mixed" and target[0] == "cpu" and page != 64:
        pytest.skip("one page size is enough for the plain operations")
    cfg, _ = weights_of(name)
    lengths = {"a": 150, "b": 33, "c": 70, "d": 1, "e": 90, "f": 33}
    req = {k: tokens_of(cfg, n, {"a": 4, "b": 3}.get(k, ord(k))) for k, n in lengths.items()}
    llm = open_llm(tmp_path, name, target, page_size=page, num_pages=sum(-(-n // page) for n in (150, 90, 70, 33)), state_slots=4)
    rng = np.random.default_rng(page)
    left, steps, live, waiting = dict(lengths), [], [], list(lengths)
    while live or waiting:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        step = []
        for name_ in list(live):
            if len(live) > 1 and rng.random() < 0.2:
                continue
            n = min(left[name_], int(rng.choice([1, 1, 2, 3, 17, 40])))
            step.append((name_, n))
            left[name_] -= n
            if left[name_] == 0:
                live.remove(name_)
        if step:
            steps.append(step)
    got = run_schedule(llm.engine, req, steps)
    for k in req:
        check(got[k], expected(name, req[k]), target)
    assert llm.engine.kv.available_pages() == llm.engine.kv.num_pages
    if name == "parallel_only" and page == 128 and target == BF16:
        assert llm.engine.runner.mixed_launches > 0


@pytest.mark.parametrize("target", TARGETS)
def test_long_decoding(tmp_path, target):
    """Hundreds of decoded tokens, several windows and pages; on the GPU replayed as CUDA graphs."""
    cfg, _ = weights_of("mixed")
    toks = tokens_of(cfg, 300, 9)
    llm = open_llm(tmp_path, "mixed", target)
    check(run_schedule(llm.engine, {"a": toks}, [[("a", 4)]] + [[("a", 1)]] * 296)["a"], expected("mixed", toks), target)
    if target[0] == "cuda":
        assert llm.engine.runner.graph_launches >= 290


@gpu
def test_both_attention_forms_in_one_model(tmp_path):
    """Long portions attend over expanded keys and values, short ones and decoded tokens over the latents: the logits agree
    with the oracle either way, and the expanded form does run, also where a window leaves blocks out."""
    cfg, _ = weights_of("wide")
    toks = {"a": tokens_of(cfg, 460, 6), "b": tokens_of(cfg, 150, 4)}
    llm = open_llm(tmp_path, "wide", BF16, page_size=64)
    used, plan = [], llm.engine.model.plan_latent_prefill

    def spy(*a):
        got = plan(*a)
        used.append(None if got is None else int(got[0][:, 1].min()))
        return got

    llm.engine.model.plan_latent_prefill = spy
    steps = [[("a", 300)], [("b", 140), ("a", 1)], [("a", 150), ("b", 2)], [("b", 1), ("a", 3)]] + [[("a", 1), ("b", 1)]] * 6 + [[("b", 1)]]
    got = run_schedule(llm.engine, toks, steps)
    for k in toks:
        check(got[k], expected("wide", toks[k]), BF16)
    assert used[:2] == [0, 0] and used[3] is None


def greedy(name, prompt, n):
    cfg, w = weights_of(name)
    w = P.as_double(w)
    toks, lead = list(prompt), []
    for _ in range(n):
        top = P.forward(cfg, w, toks)[-1].topk(2)
        lead.append(float(top.values[0] - top.values[1]))
        toks.append(int(top.indices[0]))
    return toks[len(prompt):], lead


@pytest.mark.parametrize("target", TARGETS)
def test_greedy_generation_through_the_scheduler(tmp_path, target):
    """`LLM.generate` with a token budget that cuts prompts and a pool that runs out of pages (preemption and
    recomputation): the tokens of the plain implementation. The host may be a step ahead of the device."""
    cfg, _ = weights_of("mixed")
    prompts = [tokens_of(cfg, n, 20 + i) for i, n in enumerate((30, 14, 30, 1, 20))]
    want = [greedy("mixed", p, 12) for p in prompts]
    llm = open_llm(tmp_path, "mixed", target, page_size=16, num_pages=5, max_num_seqs=3, max_num_batched_tokens=24, max_model_len=96)
    outs = llm.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    for o, (toks, lead) in zip(outs, want):
        # bf16: compare up to the first step whose two best logits are closer than rounding can tell apart
        n = 12 if target[1] == "float32" else next((i for i, m in enumerate(lead) if m < 0.05), 12)
        assert o.token_ids[:n] == toks[:n]
    assert llm.engine.scheduler.total_preemptions() > 0 and llm.engine.kv.check_invariants() == ""


@pytest.mark.parametrize("target", TARGETS)
def test_pipelined_generation(tmp_path, target):
    """The host one step ahead of the device: the same tokens as step by step."""
    from mojo_b200.engine import EngineConfig, LLMEngine

    cfg, _ = weights_of("mixed")
    prompts = [tokens_of(cfg, n, 40 + n) for n in (40, 7, 23)]
    first = open_llm(tmp_path, "mixed", target, use_cuda_graphs=False)
    sp = SamplingParams(max_tokens=10, ignore_eos=True)
    want = [o.token_ids for o in first.generate(prompts, sp)]
    eng = LLMEngine(EngineConfig(model=first.model_config, device=target[0], dtype=getattr(torch, target[1]), page_size=32, num_pages=24, max_num_seqs=4,
                                 max_num_batched_tokens=512, max_model_len=512, async_scheduling=True), model=first.engine.model)
    got = eng.generate(prompts, sp)
    if target[1] == "float32":
        assert got == want
    else:       # other row counts take other kernel shapes: as many tokens
        assert [len(t) for t in got] == [10] * 3


def test_command_line_generate_and_replay(tmp_path, capsys, monkeypatch):
    """Both command-line entries on a checkpoint folder, on the CPU engine."""
    from mojo_b200 import cli

    cfg, w = weights_of("mixed")
    P.write_checkpoint(tmp_path / "m", cfg, w)
    prompt = tokens_of(cfg, 9, 5)
    cli.main(["generate", "--model", str(tmp_path / "m"), "--device", "cpu", "--token-ids", "--prompt", ",".join(map(str, prompt)), "--max-tokens", "4",
              "--max-num-seqs", "2", "--num-pages", "8", "--page-size", "16", "--max-model-len", "64"])
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["token_ids"] == greedy("mixed", prompt, 4)[0]

    lines = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:5], "want": [1, 4]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[5:7], "want": []}, {"id": "y", "tokens": prompt[:1], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "y", "tokens": prompt[:2], "want": []}, {"id": "x", "tokens": prompt[7:], "want": [1]}], "end": ["x", "y"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    with pytest.raises(SystemExit) as done:
        cli.main(["replay", "--model", str(tmp_path / "m"), "--dtype", "float32", "--device", "cpu", "--out", str(tmp_path / "o"), "--max-tokens", "128"])
    assert done.value.code == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = expected("mixed", prompt)
    got = [torch.from_numpy(np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"]) for i in range(3)]
    check(torch.cat(got), torch.stack([want[1], want[4], want[0], want[8]]), ("cpu", "float32"))


# ------------------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------------------


def close(got, want, target, f32=2e-5, bf16=0.012):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    tol = f32 if target[1] == "float32" else bf16
    err = (got - want).abs().max() / want.abs().max().clamp_min(1e-6)
    assert err < tol, f"{err:.2e}"


def dev(t, target, dtype=None):
    return t.to(device=target[0], dtype=dtype or getattr(torch, target[1])).contiguous()


def f32(t, target):
    return dev(t, target, torch.float32)


def rounded(t, target):
    """float64 values that `target`'s element type holds exactly."""
    return t.to(getattr(torch, target[1])).double()


def sync(target):
    if target[0] == "cuda":
        ops.check_status()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("width,pad,top", [(64, 64, 1), (20, 24, 3), (1000, 1000, 2), (101, 104, 9)])
def test_residual_and_layer_norm(target, width, pad, top):
    """A stream far from zero mean takes up a sublayer's rows, expert rows of which some are the token's own input, a row behind
    a gate, or all of them; layer-normalised, with padded columns that count for nothing."""
    g = torch.Generator().manual_seed(width)

    def rnd(*s):
        t = torch.zeros(*s[:-1], pad, dtype=torch.float64)
        t[..., :width] = rounded(torch.randn(*s, generator=g), target)
        return t

    T, dtype = 6, getattr(torch, target[1])
    table, ids = rnd(11, width), torch.tensor([4, 0, 10, 4, 7, 7])
    table[:, :width] += 3.0
    table = rounded(table, target)
    w, b = rnd(width).float(), rnd(width).float()
    x = torch.full((T, pad), float("nan"), device=target[0])
    kw = dict(eps=1e-2, dtype=dtype, mean_width=width, bias=f32(b, target))
    norm = lambda t: P.layer_norm(t[:, :width], w[:width].double(), b[:width].double(), 1e-2)  # noqa: E731
    h = ops.residual_norm(x, f32(w, target), start=ops.StreamStart(ids.to(target[0]), dev(table, target), 2.5), **kw)
    want = table[ids] * 2.5
    close(x, want, (target[0], "float32"))
    close(h[:, :width], norm(want), target)
    assert float(h[:, width:].abs().sum()) == 0
    y, own, gated, rows, z = rnd(T, width), rnd(T, width), rnd(T, width), rnd(T * top, width), torch.randn(T, 3, generator=g) * 2
    wts, slot = torch.rand(T, top, generator=g), torch.randperm(T * top, generator=g).view(T, top)
    slot[1, 0] = slot[4, top - 1] = -1
    picked = torch.where((slot < 0)[..., None], own[:, None], rows[slot.clamp_min(0)])
    mixed = torch.einsum("tk,tkw->tw", wts.double(), picked)
    experts = ops.ExpertRows(dev(rows, target), dev(slot, target, torch.int32), f32(wts, target), dev(own, target))
    behind = P.sigmoid(z[:, 1].double())[:, None] * gated
    zs = f32(z, target)
    for done, add in ((ops.Finished(None, dev(y, target)), y), (ops.Finished(None, None, experts), mixed),
                      (ops.Finished(None, dev(y, target), experts, dev(gated, target), zs[:, 1]), y + mixed + behind)):
        want = x.double().cpu() + add
        kept = x.clone()
        close(ops.residual_norm(x, f32(w, target), done=done, rows=torch.tensor([3, 0, 5], device=target[0]), store=False, **kw)[:, :width],
              norm(want)[[3, 0, 5]], target)
        assert torch.equal(x, kept)
        close(ops.residual_norm(x, f32(w, target), done=done, **kw)[:, :width], norm(want), target)
        close(x, want, (target[0], "float32"))
    sync(target)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,T", [(1, 1, 8, 8, 8, 5), (6, 2, 24, 40, 12, 5), (8, 1, 64, 64, 32, 5), (5, 5, 13, 7, 6, 5), (4, 2, 128, 96, 0, 5),
                                                       (34, 2, 18, 10, 10, 5), (3, 1, 128, 128, 64, 700), (2, 1, 256, 256, 256, 650), (9, 3, 32, 32, 16, 1000),
                                                       (40, 4, 128, 128, 128, 600)])
def test_projection_norms_and_rotation(target, heads, kv, dim, vdim, rot, T):
    """Biases, one norm over all query (key) columns of a row, rotated halves, keys and values in their cache rows."""
    g = torch.Generator().manual_seed(heads + dim)
    page, n = 4, heads * dim + kv * (dim + vdim)
    pad = next(x for x in (64, 128, 256) if x >= max(dim, vdim)) if target[1] == "bfloat16" else None
    proj = rounded(torch.randn(T, n + 24, generator=g), target)
    proj[2] *= 30.0                                                          # the norm of a row is its own
    bias, qw, kw = (torch.randn(s, generator=g) for s in (n, heads * dim, kv * dim))
    pos, slots = torch.tensor([0, 1, 70, 500, 3]), torch.tensor([7, -1, 0, 19, 12])
    if T > 5:                                                                # many rows: another kernel, rows in a random order
        pos, slots = torch.randint(0, 600, (T,), generator=g), torch.randperm(4 * T, generator=g)[:T]
        slots[3] = -1
    table = reference.rope_table(600, rot, 5000.0)
    kc, vc = (dev(torch.zeros(5 if T == 5 else T, kv, page, pad or s), target) for s in (dim, vdim))
    q = ops.norm_qkv(dev(proj, target), ops.QkvNorm(*(f32(t, target) for t in (bias, qw, kw))), table.to(target[0]), dev(pos, target, torch.int32),
                     slots.to(target[0]), kc, vc, heads, kv, dim, vdim, pad or dim, 1e-2)
    sync(target)
    u = proj[:, :n] + bias.double()


    def turned(z, m):      # row i at position pos[i]
        if not rot:
            return z
        ang, out = P.angles(600, rot, 5000.0, torch.float64)[pos][:, None], z.clone()
        a, b = z[..., :rot // 2], z[..., rot // 2:rot]
        out[..., :rot // 2], out[..., rot // 2:rot] = a * torch.cos(ang) - b * torch.sin(ang), b * torch.cos(ang) + a * torch.sin(ang)
        return out

    wq = turned(P.rms_norm(u[:, :heads * dim], qw.double(), 1e-2).view(T, heads, dim), heads)
    wk = turned(P.rms_norm(u[:, heads * dim:(heads + kv) * dim], kw.double(), 1e-2).view(T, kv, dim), kv)
    got = q.view(T, heads, -1)
    close(got[..., :dim], wq, target)
    assert float(got[..., dim:].abs().sum()) == 0
    kept = slots >= 0
    at = slots[kept].to(target[0])
    close(kc.transpose(1, 2).flatten(0, 1)[at][..., :dim], wk[kept], target)
    close(vc.transpose(1, 2).flatten(0, 1)[at][..., :vdim], u[:, (heads + kv) * dim:].view(T, kv, vdim)[kept], target)
    empty = torch.ones(len(kc) * page, dtype=torch.bool)
    empty[slots[kept]] = False
    assert float(kc[..., dim:].abs().sum()) == 0 and float(vc.transpose(1, 2).flatten(0, 1)[empty.to(target[0])].abs().sum()) == 0


def edge_batch(target, ctx, page, q_len, heads, kv, dim, vdim, window, cap, seed):
    """Sequences of `ctx` keys in scattered pages: decode rows and chunks of `q_len` rows. Every query strongly asks for one key:
    the oldest that its window holds, the one before that, its own, the sequence's first."""
    g = torch.Generator().manual_seed(seed)
    n_dec, n = 4, 6
    lens = [1] * n_dec + [q_len] * (n - n_dec)
    k = rounded(torch.randn(n, ctx, kv, dim, generator=g), target)
    v = rounded(torch.randn(n, ctx, kv, vdim, generator=g), target)
    qs, want = [], []
    for b in range(n):
        q = torch.randn(lens[b], heads, dim, generator=g).double() * 0.2
        for i in range(lens[b]):
            p = ctx - lens[b] + i
            spot = [p - window + 1, p - window, p, 0][(b + i) % 4]
            if spot >= 0:
                key = k[b, spot].repeat_interleave(heads // kv, dim=0)
                q[i] = key * 12.0 / key.pow(2).sum(-1, keepdim=True)
        q = rounded(q, target)
        qs.append(q)
        full = torch.cat([torch.zeros(ctx - lens[b], heads, dim).double(), q])
        want.append(P.attend(full, k[b], v[b], 1.0, window, cap)[-lens[b]:])
    pages = -(-ctx // page)
    table = torch.randperm(n * pages, generator=g).view(n, pages).int()
    pad = next(x for x in (64, 128, 256) if x >= max(dim, vdim)) if target[1] == "bfloat16" else None
    kc, vc = (torch.zeros(n * pages, kv, page, pad or s, dtype=torch.float64) for s in (dim, vdim))
    for b in range(n):
        for t in range(ctx):
            kc[table[b, t // page], :, t % page, :dim], vc[table[b, t // page], :, t % page, :vdim] = k[b, t], v[b, t]
    ends = np.cumsum(lens)
    cu = torch.from_numpy(np.concatenate([[0], ends]).astype(np.int32)).to(target[0])
    rows = torch.tensor([[e - m, e] for m, e in zip(lens, ends)], dtype=torch.int32)
    seq = ops.SeqRows(torch.repeat_interleave(torch.arange(n, dtype=torch.int32), torch.tensor(lens)).to(target[0]), rows.to(target[0]), rows.to(target[0]),
                      n_dec, n_dec, n - n_dec)
    pos = torch.tensor([ctx - m + i for m in lens for i in range(m)], dtype=torch.int32, device=target[0])
    meta = ops.AttnMeta(cu, torch.full((n,), ctx, dtype=torch.int32, device=target[0]), table.to(target[0]), n_dec, q_len, ctx, seq=seq)
    return torch.cat(qs), dev(kc, target), dev(vc, target), meta, pos, torch.cat(want), pad


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("window", [1, 2, 31, 33, 64, 127, 128, 129, 299, 300, 5000])
@pytest.mark.parametrize("heads,kv,dim,vdim,page", [(6, 2, 24, 40, 16), (4, 1, 128, 128, 128), (3, 3, 200, 130, 64), (20, 1, 64, 48, 32), (2, 2, 100, 128, 8)])
def test_windows_and_capped_scores(target, window, heads, kv, dim, vdim, page):
    """Keys just inside and just outside a window, own and first ones, for decode rows and chunks, on every attention kernel."""
    if target[0] == "cpu" and window not in (1, 33, 300):
        pytest.skip("three windows are enough for the plain operations")
    cap = 25.0
    q, kc, vc, meta, pos, want, pad = edge_batch(target, 300, page, 140, heads, kv, dim, vdim, window, cap, window + dim)
    T, e = q.shape[0], pad or vdim
    qs = torch.zeros(T, heads, pad or dim, dtype=torch.float64)
    qs[..., :dim] = q
    out = torch.zeros(T, heads * e + 16, dtype=getattr(torch, target[1]), device=target[0])
    got = ops.paged_attention(dev(qs.view(T, -1), target), kc, vc, meta, 1.0, pad or dim, out=out[:, 16:], positions=pos, mods=ops.ScoreMods(window, cap, 0.6))
    sync(target)
    assert got.data_ptr() == out[:, 16:].data_ptr()
    close(got.view(T, heads, e)[..., :vdim], want * 0.6, target, f32=5e-5, bf16=0.03)
    assert float(out[:, :16].abs().sum()) == 0
    if window >= 300:                                                        # nothing is left out: the plain kernels agree
        plain = ops.paged_attention(dev(qs.view(T, -1), target), kc, vc, meta, 0.3, pad or dim, positions=pos)
        capped = ops.paged_attention(dev(qs.view(T, -1), target), kc, vc, meta, 0.3, pad or dim, positions=pos, mods=ops.ScoreMods(window, 0.0, 1.0))
        close(capped, plain.double().cpu(), target, f32=1e-6, bf16=0.01)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("window", [1, 32, 100, 128, 129, 300])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,page", [(1, 16, 8, 24, 64, 16), (5, 20, 12, 40, 90, 8), (16, 64, 64, 64, 512, 128), (20, 40, 96, 24, 100, 48),
                                                          (2, 90, 38, 128, 200, 64), (3, 24, 64, 40, 1000, 32)])
def test_latent_attention_with_a_rotated_part(monkeypatch, target, window, heads, dim, rot, vdim, rank, page):
    """Writing (latent norm, rotated shared key, rotated queries) and attending, decode rows and chunks, absorbed and, where its
    kernel fits, expanded. Queries ask for keys at the window's edge by the rotated part alone."""
    if target[0] == "cpu" and window not in (1, 100):
        pytest.skip("two windows are enough for the plain operations")
    g = torch.Generator().manual_seed(heads + window)
    bf16 = target[1] == "bfloat16"
    dq, e = (-(-(dim + rot) // 64) * 64, -(-vdim // 64) * 64) if bf16 else (dim + rot, vdim)
    R, Q = (next(x for x in (64, 128, 256, 512, 1024) if x >= rank), next(x for x in (64, 128) if x >= rot)) if bf16 else (rank, rot)
    ctx, lens = 300, [1, 1, 1, 130, 130]
    n, pages, base = len(lens), -(-ctx // page), 700.0
    table = reference.rope_table(ctx, rot, base).to(target[0])
    lat_w = 1 + 0.2 * torch.randn(rank, generator=g)
    uk, uv = (rounded(torch.randn(heads, s, rank, generator=g) * rank ** -0.5, target) for s in (dim, vdim))
    c, kr = rounded(torch.randn(n, ctx, rank, generator=g), target), rounded(torch.randn(n, ctx, rot, generator=g), target)
    cl = P.rms_norm(c, lat_w.double(), 1e-3)
    kr_t = torch.stack([P.rotate(kr[b][:, None], rot, base, True)[:, 0] for b in range(n)])
    bt = torch.randperm(n * pages, generator=g).view(n, pages).int()
    cache = dev(torch.full((n * pages, page, R + Q), 3.0), target)           # nothing of what was there must stay in a written row
    slot_of = lambda b, t: int(bt[b, t // page]) * page + t % page  # noqa: E731
    # every position's latent and rotated part, and the last rows' queries
    q_raw, want, gate = [], [], rounded(torch.randn(sum(lens), heads, generator=g), target)
    for b, m in enumerate(lens):
        q = torch.randn(m, heads, dim + rot, generator=g).double() * 0.3
        for i in range(m):
            p = ctx - m + i
            spot = [p - window + 1, p - window, p, 0][(b + i) % 4]
            if spot >= 0:      # turned back by the query's own angle, so that it meets the key's rotated part
                ang = P.angles(p + 1, rot, base, torch.float64)[-1]
                t = kr_t[b, spot] * 14.0 / kr_t[b, spot].pow(2).sum()
                u, v = t[0::2], t[1::2]
                q[i, :, dim::2], q[i, :, dim + 1::2] = u * torch.cos(ang) + v * torch.sin(ang), v * torch.cos(ang) - u * torch.sin(ang)
        q = rounded(q, target)
        q_raw.append(q)
        q_turned = P.rotate(torch.cat([torch.zeros(ctx - m, heads, rot).double(), q[..., dim:]]), rot, base, True)
        full = torch.cat([torch.cat([torch.zeros(ctx - m, heads, dim).double(), q[..., :dim]]), q_turned], -1)
        k = torch.cat([torch.einsum("tr,hdr->thd", cl[b], uk), kr_t[b][:, None].expand(ctx, heads, rot)], -1)
        want.append(P.attend(full, k, torch.einsum("tr,her->the", cl[b], uv), 1.0, window)[-m:])
    want = torch.cat(want) * P.sigmoid(gate)[..., None]
    T, q_raw = sum(lens), torch.cat(q_raw)
    # the earlier positions go in first, through the same kernel
    old = [(b, t) for b, m in enumerate(lens) for t in range(ctx - m)]
    new = [(b, t) for b, m in enumerate(lens) for t in range(ctx - m, ctx)]
    off = heads * dq
    for rows, q in ((old, None), (new, q_raw)):
        proj = torch.zeros(len(rows), off + rank + rot + (-(rank + rot)) % 8, dtype=torch.float64)
        if q is not None:
            proj[:, :off].view(len(rows), heads, dq)[..., :dim + rot] = q
        proj[:, off:off + rank], proj[:, off + rank:off + rank + rot] = torch.stack([c[b, t] for b, t in rows]), torch.stack([kr[b, t] for b, t in rows])
        proj = dev(proj, target)
        pos = torch.tensor([t for _, t in rows], dtype=torch.int32, device=target[0])
        rope = ops.SharedRope(proj[:, off + rank:off + rank + rot], proj[:, :off], heads, dim, R, table, pos)
        ops.latent_write(proj[:, off:off + rank], f32(lat_w, target), 1e-3, torch.tensor([slot_of(b, t) for b, t in rows], device=target[0]), cache, rope)
    sync(target)
    flat = cache.view(n * pages * page, -1)
    at = torch.tensor([slot_of(*r) for r in new], device=target[0])
    close(flat[at, :rank], torch.stack([cl[r] for r in new]), target)
    close(flat[at, R:R + rot], torch.stack([kr_t[r] for r in new]), target)
    if bf16:
        assert float(flat[at, rank:R].abs().sum() + flat[at, R + rot:].abs().sum()) == 0
    # attention
    key = torch.zeros(heads, dq, R + Q, dtype=torch.float64)
    key[:, :dim, :rank], key[:, dim:dim + rot, R:R + rot] = uk, torch.eye(rot, dtype=torch.float64)
    val = torch.zeros(heads, e, R + Q, dtype=torch.float64)
    val[:, :vdim, :rank] = uv
    w_qk = dev(key.transpose(1, 2).reshape(heads * (R + Q), dq), target)
    w_kv = dev(torch.cat([key.view(heads * dq, -1), val.view(heads * e, -1)]), target)
    ends = np.cumsum(lens)
    cu = torch.from_numpy(np.concatenate([[0], ends]).astype(np.int32)).to(target[0])
    meta = ops.AttnMeta(cu, torch.full((n,), ctx, dtype=torch.int32, device=target[0]), bt.to(target[0]), 3, 130, ctx)
    rows = ops.token_rows(meta, T, torch.device(target[0]))
    q, gs = proj[:, :off], dev(gate, target)
    q_lat = ops.head_linear(q, w_qk, heads)
    o_lat = ops.latent_attend(q_lat, cache, meta, rows, heads, 1.0, pos, R, window)
    o = ops.head_linear(o_lat, w_kv[heads * dq:, :R], heads, gate=gs)
    sync(target)
    close(o.view(T, heads, e)[..., :vdim], want, target, f32=5e-5, bf16=0.04)
    if bf16 and (dq, e) == (128, 128):
        monkeypatch.setattr(ops.latent, "ABSORBED_RATE", 1e-3)               # the expanded form however narrow the window
        host = cu.cpu().numpy(), np.full(n, ctx)
        plan = ops.plan_latent_prefill(*host, 3, 1024, heads, 128, 128, window)
        first = max(0, ctx - 130 - window + 1) // 128
        assert plan[0][:, 1].min() == first and len(plan[0]) == 2 * (3 - first)
        meta.expand = tuple(torch.from_numpy(t).cuda() for t in plan)
        meta.work = torch.from_numpy(ops.prefill_work_items(*host, 3)).cuda()
        meta.n_items = meta.work.shape[0]
        out = torch.full((T, heads * 128), 7.0, dtype=torch.bfloat16, device="cuda")
        ops.latent_prefill(q, cache, w_kv, meta, heads, 1.0, gs, out, window)
        sync(target)
        assert bool((out[:3] == 7).all())
        close(out[3:].view(-1, heads, 128)[..., :vdim], want[3:], target, bf16=0.04)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,dim,vdim,tau", [(1, 8, 8, 1.0), (2, 48, 32, 16.0), (3, 13, 7, 4.0), (4, 128, 128, 16.0), (2, 70, 90, 8.0), (1, 256, 200, 2.0)])
@pytest.mark.parametrize("lens", [(1, 1, 1, 37, 2, 5, 130), (1, 1, 1, 700, 16, 531, 2), (1, 1, 1, 1100, 33)], ids=lambda x: f"{sum(x)}rows")
def test_recurrence(target, heads, dim, vdim, tau, lens):
    """Decode rows beside chunks of several lengths, fresh sequences and ones with history, decays from almost none to almost
    total; states land in their slots, other slots stay as they are, and a fresh sequence ignores what its slot held. Few long
    chunks are cut into segments that run side by side."""
    if sum(lens) > 200 and target[0] == "cpu" and dim != 13:
        pytest.skip("one size is enough for the plain operations")
    g = torch.Generator().manual_seed(dim + heads)
    fresh, slots = [False, True, False, True, False, False, False][:len(lens)], [5, 0, 7, 2, 3, 8, 1][:len(lens)]
    T, nk, nv, n = sum(lens), heads * dim, heads * vdim, len(lens)
    proj = rounded(torch.randn(T, 2 * (nk + nv), generator=g), target)
    z, bias, w = torch.randn(T, nk + 3, generator=g) * 3, torch.randn(nk, generator=g) * 4, 1 + 0.2 * torch.randn(vdim, generator=g)
    state = torch.randn(10, heads, dim, vdim, generator=g)
    ends = np.cumsum(lens)
    rows = torch.tensor([[e - m, e] for m, e in zip(lens, ends)], dtype=torch.int32)
    banks = torch.tensor([[-1 if f else 2 * s, 2 * s + 1] for f, s in zip(fresh, slots)], dtype=torch.int32)
    seq = ops.SeqRows(torch.repeat_interleave(torch.arange(n, dtype=torch.int32), torch.tensor(lens)).to(target[0]), rows.to(target[0]), banks.to(target[0]), 3, 3, n - 3)
    log_a = (P.log_sigmoid(z[:, :nk].double() + bias.double()) / tau).view(T, heads, dim)
    assert float(log_a.min()) < -8.0 / tau and float(log_a.max()) > -1e-2
    want, last = torch.zeros(T, heads, vdim, dtype=torch.float64), state.double()
    q, k, v = proj[:, :nk].view(T, heads, dim) * dim ** -0.5, proj[:, nk:2 * nk].view(T, heads, dim), proj[:, 2 * nk:2 * nk + nv].view(T, heads, vdim)
    for (b, e), f, s in zip(rows.tolist(), fresh, slots):
        want[b:e], last[s] = P.recurrence(q[b:e], k[b:e], v[b:e], log_a[b:e], None if f else last[s])
    want = P.rms_norm(want, w.double(), 1e-4).reshape(T, nv) * P.silu(proj[:, 2 * nk + nv:]) * 0.5
    out = torch.full((T, nv + 8), 7.0, dtype=getattr(torch, target[1]), device=target[0])
    st = f32(state, target)
    ops.gated_linear(dev(proj, target), f32(z, target), ops.GatedLinearParams(f32(bias, target), f32(w, target), tau), st, seq, heads, dim, vdim, 1e-4,
                     out[:, :nv], 0.5)
    sync(target)
    close(out[:, :nv], want, target)
    close(st, last, (target[0], "float32"))
    assert bool((out[:, nv:] == 7).all())
    for s in set(range(10)) - set(slots):
        assert torch.equal(st[s].cpu(), state[s])


@pytest.mark.parametrize("target", TARGETS)
def test_recurrence_does_not_depend_on_the_cuts(target):
    """Long prompts in one piece, in portions and token by token: the same outputs and state."""
    g = torch.Generator().manual_seed(1)
    T, H, d, e = 200, 2, 40, 24
    proj, z = dev(torch.randn(T, 2 * H * (d + e), generator=g), target), f32(torch.randn(T, H * d, generator=g) * 2, target)
    p = ops.GatedLinearParams(f32(torch.zeros(H * d) + 3.0, target), f32(torch.ones(e), target), 16.0)

    def run(cuts):
        st, out = torch.full((2, H, d, e), 9.0, device=target[0]), torch.zeros(T, H * e, dtype=proj.dtype, device=target[0])
        a = 0
        for i, n in enumerate(cuts):
            one = n == 1
            i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=target[0])  # noqa: E731
            seq = ops.SeqRows(i32([0] * n), i32([[0, n]]), i32([[-1 if i == 0 else 2 + (i + 1) % 2, 2 + i % 2]]), int(one), int(one), int(not one))
            ops.gated_linear(proj[a:a + n], z[a:a + n], p, st, seq, H, d, e, 1e-5, out[a:a + n])
            a += n
        sync(target)
        return out.float().cpu(), st[1].cpu()

    whole = run([T])
    for cuts in ([2] * 100, [1] * T, [64, 1, 3, 1, 60, 71], [199, 1]):
        got = run(cuts)
        close(got[0], whole[0].double(), target, f32=1e-5)
        close(got[1], whole[1].double(), (target[0], "float32"))


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("experts,identity,top,groups,rows", [(1, 0, 1, (1, 1), 3), (7, 2, 3, (3, 2), 40), (6, 2, 4, (2, 1), 300), (64, 0, 6, (8, 3), 200), (62, 2, 6, (8, 4), 130),
                                                              (300, 20, 5, (40, 7), 300), (3, 5, 8, (1, 1), 20), (5, 0, 5, (5, 5), 10), (12, 4, 2, (16, 3), 700)])
def test_mixture_with_groups_and_identity(target, experts, identity, top, groups, rows):
    """Corrected choices group by group, weights from the uncorrected scores, squared-ReLU experts and ones that return their
    input. Corrections push choice scores below zero, so that a group left out must not count as zero."""
    g = torch.Generator().manual_seed(experts + rows)
    W, f, n = 72, 32, experts + identity
    h = rounded(torch.randn(rows, W, generator=g), target)
    router = rounded(torch.randn(n, W, generator=g) * 2.0 * W ** -0.5, target)
    corr = torch.randn(n, generator=g) * 0.3 - 1.0
    up, down = rounded(torch.randn(experts, f, W, generator=g) * 2 * W ** -0.5, target), rounded(torch.randn(experts, W, f, generator=g) * f ** -0.5, target)
    r = {"experts": experts, "top": top, "identity": identity, "groups": dict(zip(("count", "keep"), groups))}
    gaps = []
    wt = P.route(h @ router.T, corr.double(), r, gaps)
    want = wt[:, experts:].sum(1, keepdim=True) * h
    for e in range(experts):
        want = want + wt[:, e:e + 1] * (P.relu2(h @ up[e].T) @ down[e].T)
    if n > 2 * top and groups[0] > groups[1]:
        plain = (h @ router.T).topk(top, 1).indices                          # what is chosen differs from the plain choice
        assert bool((wt.gather(1, plain) == 0).any())
    p = ops.MoeWeights(dev(torch.cat([router, torch.zeros(-n % 8, W).double()]), target), dev(up, target), dev(down, target), experts, top, "softmax", True, 1.0, None,
                       f32(corr, target), *groups, identity)
    sure = torch.stack([(x > 1e-4) for x in gaps]).all(0) if gaps else torch.ones(rows, dtype=torch.bool)
    assert sure.float().mean() > 0.9
    hd = dev(h, target)
    for _ in range(2):                                                       # the counters are clean again afterwards
        ex = ops.moe_experts(hd, p)
        slot = ex.slot.long().cpu()
        assert (ex.own is None) == (identity == 0)
        got = ex.rows.double().cpu()[slot.clamp_min(0)]
        if identity:
            got = torch.where((slot < 0)[..., None], ex.own.double().cpu()[:, None], got)
        got = torch.where(ex.weights.cpu()[..., None] > 0, got, torch.zeros_like(got))
        close(torch.einsum("tk,tkw->tw", ex.weights.double().cpu(), got)[sure], want[sure], target, bf16=0.02)
    used = slot[slot >= 0]
    assert used.unique().numel() == used.numel() and (used < rows * top).all()
    sync(target)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("rows", [1, 37, 300])
def test_relu_gated_unit(target, rows):
    """max(g, 0) u behind a matrix product, into columns of a wider matrix; zeros stay zeros."""
    g = torch.Generator().manual_seed(rows)
    K, F = 104, 144
    x, wg, wu = (rounded(torch.randn(*s, generator=g) * c, target) for s, c in (((rows, K), 1.0), ((F, K), 3 * K ** -0.5), ((F, K), 3 * K ** -0.5)))
    x[0] = 0.0
    out = torch.full((rows, F + 32), 7.0, dtype=getattr(torch, target[1]), device=target[0])
    ops.linear_swiglu(dev(x, target), dev(reference.interleave_gate_up(wg.float(), wu.float()), target), out=out[:, 32:], glu=ops.REGLU)
    sync(target)
    close(out[:, 32:], (x @ wg.T).clamp_min(0) * (x @ wu.T), target)
    assert bool((out[:, :32] == 7).all()) and float(out[0, 32:].abs().sum()) == 0


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,n,k", [(1, 64, 64), (5, 128, 192), (16, 128, 512)])
def test_one_gate_per_head(target, heads, n, k):
    g = torch.Generator().manual_seed(n + k)
    T = 130
    x, w = rounded(torch.randn(T, heads * k, generator=g), target), rounded(torch.randn(heads * n, k + 64, generator=g) * k ** -0.5, target)
    z = rounded(torch.randn(T, heads + 3, generator=g), target)
    want = torch.cat([x[:, h * k:(h + 1) * k] @ w[h * n:(h + 1) * n, :k].T * P.sigmoid(z[:, 1 + h:2 + h]) for h in range(heads)], dim=1)
    out = torch.zeros(T, heads * n + 8, dtype=getattr(torch, target[1]), device=target[0])
    ops.head_linear(dev(x, target), dev(w, target)[:, :k], heads, gate=dev(z, target)[:, 1:1 + heads], out=out[:, :heads * n])
    sync(target)
    close(out[:, :heads * n], want, target)


# ------------------------------------------------------------------------------------------------------
# configuration and bookkeeping
# ------------------------------------------------------------------------------------------------------


def test_plan_of_the_expanded_form_with_a_window():
    """Blocks that no row of a sequence sees are not expanded; the tables still count blocks from a sequence's start."""
    plan = lambda cu, ctx, nd, w: ops.plan_latent_prefill(cu, ctx, nd, 512, 16, 128, 128, w)  # noqa: E731
    pages, tables = plan([0, 1, 501, 901], [70, 500, 1400], 1, 200)
    assert pages.tolist() == [[0, b] for b in range(4)] + [[1, b] for b in range(6, 11)]
    assert tables[0, :4].tolist() == [0, 1, 2, 3] and tables[1, 6:11].tolist() == [4, 5, 6, 7, 8]
    assert 0 <= tables.min() and tables.max() < len(pages)
    assert plan([0, 30], [4000], 0, 0) is not None and plan([0, 30], [4000], 0, 16) is None      # a narrow window is cheap to attend over
    assert (plan([0, 900], [900], 0, 5000)[0] == plan([0, 900], [900], 0, 0)[0]).all()


def test_config_reading_and_refusals(tmp_path):
    from mojo_b200.models import build_model, get_config

    cfg, w = weights_of("mixed")
    P.write_checkpoint(tmp_path / "m", cfg, w)
    mc = get_config(str(tmp_path / "m"))
    assert (mc.architecture, mc.num_layers, mc.hidden_size, mc.vocab_size, mc.logit_scale) == ("pilutar", 4, 96, 101, 0.5)
    left, right = mc.layers[0].parts
    assert (left.window, left.softcap, left.rot.dims, left.rot.interleaved, right.tau) == (37, 8.0, 16, False, 4.0)
    assert mc.layers[2].part_scales == [0.3, 1.2] and mc.layers[3].moe is None and mc.layers[3].ffn == 0 and mc.layers[1].rot.interleaved
    moe = mc.layers[1].moe
    assert (moe.experts, moe.identity, moe.groups, moe.keep, moe.top, moe.shared.ffn) == (7, 2, 3, 2, 3, 24) and mc.layers[2].moe.shared is None
    model = build_model(mc)
    assert model.recurrent_state and model.kv_bytes_per_page(16) == (2 * (24 + 40) + 40 + 12 + 4 * 32 + 64 + 8) * 16 * 4
    assert model.state_bytes_per_slot() == (3 * 20 * 28 + 2 * 32 * 16) * 4
    assert not build_model(P_config(tmp_path, model_single())).recurrent_state

    def broken(i, edit):
        bad = json.loads(json.dumps(cfg))
        edit(bad["layers"][i])
        (tmp_path / "m" / "config.json").write_text(json.dumps(bad))
        return lambda: get_config(str(tmp_path / "m"))

    for i, edit, match in ((0, lambda s: s.update(type="other"), "mixer"), (0, lambda s: s["mixer"]["left"].update(kv_heads=4), "key heads"),
                           (1, lambda s: s["mlp"]["router"].update(top=7), "experts"), (1, lambda s: s["mlp"]["router"]["groups"].update(count=2), "groups"),
                           (1, lambda s: s["mixer"].update(rot_dim=11), "rotary"), (0, lambda s: s["mixer"]["left"]["rot"].update(dims=26), "rotary"),
                           (1, lambda s: s["mlp"].update(kind="other"), "feed-forward")):
        with pytest.raises(ValueError, match=match):
            broken(i, edit)()
    for name in ("l1.mix.uk", "head", "l1.mlp.e6.down", "l0.mix.right.a2.b", "l1.mlp.correction"):
        P.write_checkpoint(tmp_path / "bad", cfg, {**w, name: w[name][:-1]})
        with pytest.raises(ValueError, match=name.split(".", 1)[-1]):
            LLM(PipelineConfig(model=str(tmp_path / "bad"), device="cpu"))


def P_config(tmp_path, cfg):
    from mojo_b200.models import get_config

    (tmp_path / "c").mkdir(exist_ok=True)
    (tmp_path / "c" / "config.json").write_text(json.dumps(cfg))
    return get_config(str(tmp_path / "c"))


def test_presets_generate():
    from mojo_b200.models import build_model, get_config

    assert 20e9 > get_config("pilutar-lite").num_params() > 5e9
    mc = get_config("tiny-pilutar")
    model = build_model(mc)
    n = sum(int(np.prod(s)) for s in model.global_shapes().values())
    n += sum(int(np.prod([16 if x == -1 else x for x in s])) for spec in mc.layers for s in model.tensor_shapes(spec, mc.hidden_size).values())
    assert abs(n - mc.num_params()) < 0.01 * n
    llm = LLM(PipelineConfig(model="tiny-pilutar", device="cpu", random_init=True, page_size=16, num_pages=16, max_num_seqs=2, max_model_len=64))
    assert len(llm.generate([[1, 2, 3]], SamplingParams(max_tokens=3))[0].token_ids) == 3
