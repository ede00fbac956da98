"""Rerupel against the plain implementation in `rerupel_oracle`: every mechanism alone, whole prompts, decoding, cut
prompts, mixed batches, pages used again, and greedy generation through the scheduler. The same tests run on the CPU
engine and, marked `gpu`, on the kernels in f32 and bf16."""
import json

import numpy as np
import pytest
import rerupel_oracle as R
import torch

from mojo_b200 import ops
from mojo_b200.ops import reference
from mojo_b200.pipelines import LLM, PipelineConfig, SamplingParams

gpu = pytest.mark.gpu
TARGETS = [pytest.param(("cpu", "float32"), id="cpu"), pytest.param(("cuda", "float32"), id="f32", marks=gpu),
           pytest.param(("cuda", "bfloat16"), id="bf16", marks=gpu)]
BF16 = ("cuda", "bfloat16")


def model_looped():
    """Every kind of feed-forward, layers of different sizes, a loop over the middle ones, a narrow bigram table."""
    return R.config(96, 101, [
        R.layer_spec(6, 24, 40, 48, R.dense_spec(72)),
        R.layer_spec(3, 48, 16, 64, R.moe_spec(7, 2, 40, limit=1.0, scale=1.7, shared=(24, 0.5))),
        R.layer_spec(4, 32, 32, 80, None),
        R.layer_spec(6, 24, 40, 48, R.moe_spec(12, 3, 24))], loop=(1, 3, 3), bigram=(53, 11, 5))


def model_odd():
    """Sizes that are multiples of nothing much, more heads than an MMA tile has rows, every expert used, loop to the end."""
    return R.config(101, 67, [
        R.layer_spec(2, 70, 90, 150, R.moe_spec(5, 5, 20, limit=0.8, scale=0.5, shared=(9, 3.0))),
        R.layer_spec(20, 13, 21, 90, R.moe_spec(9, 1, 33, limit=1.5))], loop=(1, 2, 2), eps=1e-3, mult=1.3, cap=5.0)


def model_wide_heads():
    """Heads that fill the prefill kernel's 128 columns only in part; the loop starts at the first layer."""
    return R.config(256, 200, [
        R.layer_spec(4, 96, 128, 256, R.moe_spec(8, 2, 48, shared=(112, 2.5))),
        R.layer_spec(2, 128, 72, 200, R.dense_spec(160))], loop=(0, 2, 2), bigram=(401, 3, 1))


def model_single():
    """One head, one expert, one pass; no loop, no bigram table."""
    return R.config(64, 33, [
        R.layer_spec(1, 16, 8, 16, R.moe_spec(1, 1, 16, limit=1.0, shared=(16, 1.0))),
        R.layer_spec(1, 8, 16, 24, R.dense_spec(16))], bigram=None, mult=1.0, scale=1.0)


MODELS = {"looped": model_looped, "odd": model_odd, "wide_heads": model_wide_heads, "single": model_single}
_cache: dict = {}


def weights_of(name):
    cfg = MODELS[name]()
    return cfg, R.random_weights(cfg, seed=len(name), sharp=2.0)


def tokens_of(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def expected(name, tokens):
    """Oracle logits of one sequence in float64, once per (model, tokens). Rounding must not decide which experts run."""
    key = (name, tuple(tokens))
    if key not in _cache:
        cfg, w = weights_of(name)
        gaps = []
        _cache[key] = R.forward(cfg, R.as_double(w), tokens, gaps=gaps)
        assert min((float(x.min()) for x in gaps), default=9.0) > 0.2
    return _cache[key]


def open_llm(tmp_path, name, target, **kw):
    device, dtype = target
    cfg, w = weights_of(name)
    R.write_checkpoint(tmp_path / name, cfg, w)
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
    err = R.relative_error(got, want)
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
    page = 128 if name == "wide_heads" else 32
    llm = open_llm(tmp_path, name, target, page_size=page, num_pages=-(-160 // page), max_num_seqs=1)
    for n, seed in ((1, 1), (2, 2), (33, 3), (150, 4)):
        toks = tokens_of(cfg, n, seed)
        check(run_schedule(llm.engine, {"a": toks}, [[("a", n)]])["a"], expected(name, toks), target)
        if n > 1:
            check(run_schedule(llm.engine, {"a": toks}, [[("a", max(1, n - 40))]] + [[("a", 1)]] * min(40, n - 1))["a"], expected(name, toks), target)


@pytest.mark.parametrize("name", sorted(MODELS))
@pytest.mark.parametrize("target", TARGETS)
def test_portions(tmp_path, target, name):
    """Prompts cut into portions of changing size, down to two tokens and to one, across page borders."""
    cfg, _ = weights_of(name)
    llm = open_llm(tmp_path, name, target, page_size=128 if name == "odd" else 32)
    toks = tokens_of(cfg, 150, 4)
    for cuts in ([2] * 10 + [3] * 5 + [2, 27, 1, 31, 2, 50, 2], [31, 2, 30, 1, 1, 2, 33, 50]):
        assert sum(cuts) == 150
        check(run_schedule(llm.engine, {"a": toks}, [[("a", c)] for c in cuts])["a"], expected(name, toks), target)


@pytest.mark.parametrize("page", [8, 16, 64, 128])
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["looped", "wide_heads"])
def test_unequal_batches_with_reuse(tmp_path, target, name, page):
    """Four live requests in one batch, portions beside decoded tokens, some left out of steps; the pool only fits the live
    ones, so later requests use pages that others gave back."""
    cfg, _ = weights_of(name)
    lengths = {"a": 150, "b": 33, "c": 70, "d": 1, "e": 90, "f": 33}
    req = {k: tokens_of(cfg, n, {"a": 4, "b": 3}.get(k, ord(k))) for k, n in lengths.items()}
    llm = open_llm(tmp_path, name, target, page_size=page, num_pages=sum(-(-n // page) for n in (150, 90, 70, 33)))
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


@pytest.mark.parametrize("target", TARGETS)
def test_long_decoding(tmp_path, target):
    """Hundreds of decoded tokens, several pages; on the GPU replayed as CUDA graphs."""
    cfg, _ = weights_of("looped")
    toks = tokens_of(cfg, 300, 9)
    llm = open_llm(tmp_path, "looped", target)
    check(run_schedule(llm.engine, {"a": toks}, [[("a", 4)]] + [[("a", 1)]] * 296)["a"], expected("looped", toks), target)
    if target[0] == "cuda":
        assert llm.engine.runner.graph_launches >= 290


@gpu
def test_both_attention_forms_in_one_model(tmp_path):
    """Long portions attend over expanded keys and values, short ones and decoded tokens over the latents: the logits agree
    with the oracle either way, and the expanded form does run."""
    cfg, _ = weights_of("wide_heads")
    toks = {"a": tokens_of(cfg, 460, 6), "b": tokens_of(cfg, 150, 4)}
    llm = open_llm(tmp_path, "wide_heads", BF16, page_size=64)
    used, plan = [], llm.engine.model.plan_latent_prefill
    llm.engine.model.plan_latent_prefill = lambda *a: used.append(plan(*a) is not None) or plan(*a)
    steps = [[("a", 300)], [("b", 140), ("a", 1)], [("a", 150), ("b", 2)], [("b", 1), ("a", 3)]] + [[("a", 1), ("b", 1)]] * 6 + [[("b", 1)]]
    got = run_schedule(llm.engine, toks, steps)
    for k in toks:
        check(got[k], expected("wide_heads", toks[k]), BF16)
    assert used[:3] == [True, True, True] and used[3] is False


def greedy(name, prompt, n):
    cfg, w = weights_of(name)
    w = R.as_double(w)
    toks, margins = list(prompt), []
    for _ in range(n):
        top = R.forward(cfg, w, toks)[-1].topk(2)
        margins.append(float(top.values[0] - top.values[1]))
        toks.append(int(top.indices[0]))
    return toks[len(prompt):], margins


@pytest.mark.parametrize("target", TARGETS)
def test_greedy_generation_through_the_scheduler(tmp_path, target):
    """`LLM.generate` with a token budget that cuts prompts and a pool that runs out of pages (preemption and
    recomputation): the tokens of the plain implementation."""
    cfg, _ = weights_of("looped")
    prompts = [tokens_of(cfg, n, 20 + i) for i, n in enumerate((30, 14, 30, 1, 20))]
    want = [greedy("looped", p, 12) for p in prompts]
    llm = open_llm(tmp_path, "looped", target, page_size=16, num_pages=5, max_num_seqs=3, max_num_batched_tokens=24, max_model_len=96)
    outs = llm.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    for o, (toks, margins) in zip(outs, want):
        # bf16: compare up to the first step whose two best logits are closer than rounding can tell apart
        n = 12 if target[1] == "float32" else next((i for i, m in enumerate(margins) if m < 0.1), 12)
        assert o.token_ids[:n] == toks[:n]
    assert llm.engine.scheduler.total_preemptions() > 0 and llm.engine.kv.check_invariants() == ""


@pytest.mark.parametrize("target", TARGETS)
def test_pipelined_and_prefix_cached_generation(tmp_path, target):
    """The host one step ahead of the device (the newest token of a sequence is still on the device when its next row is
    planned), and prompts that continue from cached pages: the same tokens as step by step."""
    from mojo_b200.engine import EngineConfig, LLMEngine

    cfg, _ = weights_of("looped")
    shared = tokens_of(cfg, 64, 50)
    prompts = [shared + tokens_of(cfg, n, 40 + n) for n in (20, 7, 13)]
    first = open_llm(tmp_path, "looped", target, use_cuda_graphs=False)
    sp = SamplingParams(max_tokens=10, ignore_eos=True)
    want = [o.token_ids for o in first.generate(prompts, sp)]
    for kw in ({"async_scheduling": True}, {"enable_prefix_cache": True}):
        ecfg = EngineConfig(model=first.model_config, device=target[0], dtype=getattr(torch, target[1]), page_size=32, num_pages=24, max_num_seqs=4,
                            max_num_batched_tokens=512, max_model_len=512, **kw)
        eng = LLMEngine(ecfg, model=first.engine.model)
        if target[1] == "float32":
            assert eng.generate(prompts, sp) == want
            assert eng.generate(prompts, sp) == want                # the second time the prompts' pages are in the cache
            assert "enable_prefix_cache" not in kw or eng.kv.stats().prefix_hits >= 6
        else:       # other row counts take other kernel shapes: the same tokens as itself
            assert [len(t) for t in eng.generate(prompts, sp)] == [10] * 3


def test_command_line_generate_and_replay(tmp_path, capsys, monkeypatch):
    """Both command-line entries on a checkpoint folder, on the CPU engine."""
    import io

    from mojo_b200 import cli

    cfg, w = weights_of("looped")
    R.write_checkpoint(tmp_path / "m", cfg, w)
    prompt = tokens_of(cfg, 9, 5)
    cli.main(["generate", "--model", str(tmp_path / "m"), "--device", "cpu", "--token-ids", "--prompt", ",".join(map(str, prompt)), "--max-tokens", "4",
              "--max-num-seqs", "2", "--num-pages", "8", "--page-size", "16", "--max-model-len", "64"])
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["token_ids"] == greedy("looped", prompt, 4)[0]

    lines = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:5], "want": [1, 4]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[5:7], "want": []}, {"id": "y", "tokens": prompt[:1], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "y", "tokens": prompt[:2], "want": []}, {"id": "x", "tokens": prompt[7:], "want": [1]}], "end": ["x", "y"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    with pytest.raises(SystemExit) as done:
        cli.main(["replay", "--model", str(tmp_path / "m"), "--dtype", "float32", "--device", "cpu", "--out", str(tmp_path / "o"), "--max-tokens", "128"])
    assert done.value.code == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = expected("looped", prompt)
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


def rounded(t, target):
    """float64 values that `target`'s element type holds exactly."""
    return t.to(getattr(torch, target[1])).double()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("width,top", [(64, 1), (20, 3), (1000, 2), (2048, 6), (101, 9)])
def test_residual(target, width, top):
    """The stream starts from both tables, takes up a sublayer's rows, a token's expert rows, or both; normalised, plain, and
    for chosen rows."""
    g = torch.Generator().manual_seed(width)

    def rnd(*s):
        return rounded(torch.randn(*s, generator=g), target)

    T, f32 = 6, (target[0], "float32")
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": 13, "mul_prev": 123456789012, "mul_cur": 17}}}
    tokens = [4, 0, 10, 4, 7, 7]
    w = {"embed": rnd(11, width), "bigram": rnd(14, width)}
    x0 = R.embedding(tokens, w, cfg)
    dtype = getattr(torch, target[1])
    ids = torch.tensor(tokens, device=target[0])
    prev = torch.tensor([-1] + tokens[:-1], dtype=torch.int32, device=target[0])
    both = torch.zeros(T, 2 * width + 8, dtype=dtype, device=target[0])
    start = ops.StreamStart(ids, dev(w["embed"], target), 2.5, prev, dev(w["bigram"], target), 123456789012, 17, both[:, width:2 * width])
    x = torch.full((T, width), float("nan"), device=target[0])
    weight, scale = torch.randn(width, generator=g), torch.randn(width, generator=g)
    h = ops.residual_norm(x, dev(weight, f32), 1e-2, dtype, start=start)
    close(x, x0, f32)                                                   # the stream stays f32 in both forms
    close(both[:, width:2 * width], x0, target)
    close(h, R.norm(x0, weight.double(), 1e-2), target)
    # without a bigram table
    y = torch.empty(T, width, device=target[0])
    ops.residual_norm(y, dev(weight, f32), 1e-2, dtype, start=ops.StreamStart(ids, start.embed, 0.5))
    close(y, w["embed"][tokens] * 0.5, f32)
    # sublayer rows, expert rows, both
    out, rows, wts = rnd(T, width), rnd(T * top, width), torch.rand(T, top, generator=g)
    slot = torch.randperm(T * top, generator=g).view(T, top)
    mixed = torch.einsum("tk,tkw->tw", wts.double(), rows[slot])
    experts = ops.ExpertRows(dev(rows, target), dev(slot, target, torch.int32), dev(wts, f32))
    for y_, ex, add in ((out, None, out), (None, experts, mixed), (out, experts, out + mixed)):
        want = x.double().cpu() + scale.double() * add
        done = ops.Finished(dev(scale, f32), None if y_ is None else dev(y_, target), ex)
        kept = x.clone()
        pick = torch.tensor([3, 0, 5], device=target[0])
        close(ops.residual_norm(x, dev(weight, f32), 1e-2, dtype, done, rows=pick, store=False), R.norm(want, weight.double(), 1e-2)[[3, 0, 5]], target)
        assert torch.equal(x, kept)
        ops.residual_norm(x, None, 1e-2, dtype, done, out=both[:, :width], store=False)
        close(both[:, :width], want, target)
        assert torch.equal(x, kept)
        close(ops.residual_norm(x, dev(weight, f32), 1e-2, dtype, done), R.norm(want, weight.double(), 1e-2), target)
        close(x, want, f32)
    if target[0] == "cuda":
        ops.check_status()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("rank,pad", [(64, 64), (48, 64), (90, 128), (512, 512), (1000, 1024), (7, 7)])
def test_latents_into_pages(target, rank, pad):
    g = torch.Generator().manual_seed(rank)
    T, page = 9, 4
    proj = rounded(torch.randn(T, rank + 24, generator=g), target)
    w = torch.randn(rank, generator=g)
    cache = dev(torch.ones(5, page, pad), target)
    slots = torch.tensor([7, -1, 0, 19, 3, 4, 11, -1, 12], device=target[0])
    ops.latent_write(dev(proj, target)[:, 16:16 + rank], dev(w, target, torch.float32), 1e-2, slots, cache)
    if target[0] == "cuda":
        ops.check_status()
    want = R.norm(proj[:, 16:16 + rank], w.double(), 1e-2)
    flat = cache.view(-1, pad)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            close(flat[s, :rank], want[t], target)
    if pad > rank and target[0] == "cuda":
        assert float(flat[slots[slots >= 0], rank:].abs().sum()) == 0
    untouched = [s for s in range(20) if s not in slots.tolist()]
    assert bool((flat[untouched] == 1).all())


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,n,k", [(1, 64, 64), (5, 128, 64), (3, 64, 192), (16, 512, 128), (16, 128, 512), (2, 1024, 64)])
@pytest.mark.parametrize("rows", [1, 130])
def test_one_matrix_per_head(target, heads, n, k, rows):
    g = torch.Generator().manual_seed(n + k)
    x, w = rounded(torch.randn(rows, heads * k + 8, generator=g), target), rounded(torch.randn(heads * n, k, generator=g) * k ** -0.5, target)
    z = rounded(torch.randn(rows, heads * n + 16, generator=g), target)
    want = torch.cat([x[:, h * k:(h + 1) * k] @ w[h * n:(h + 1) * n].T for h in range(heads)], dim=1)
    xs, ws, zs = dev(x, target)[:, :heads * k], dev(w, target), dev(z, target)[:, 8:8 + heads * n]
    close(ops.head_linear(xs, ws, heads), want, target)
    out = torch.zeros(rows + 1, heads * n, dtype=xs.dtype, device=target[0])
    ops.head_linear(xs, ws, heads, gate=zs, out=out[:rows])
    close(out[:rows], want * R.sigmoid(z[:, 8:8 + heads * n]), target)
    assert float(out[rows:].abs().sum()) == 0
    if target[0] == "cuda":
        ops.check_status()


def planted_batch(target, ctx, page, q_len, heads, dim, vdim, rank, seed):
    """Sequences of `ctx` latents in scattered pages, each with one latent whose key the last query of the sequence asks for.
    Returns (inputs, oracle outputs per row, planted values)."""
    g = torch.Generator().manual_seed(seed)
    spots = sorted({s for s in (0, 1, page - 1, page, page + 1, 2 * page - 1, 31, 32, 127, 128, 255, ctx - 2, ctx - 1) if s < ctx})
    B, pages = len(spots), -(-ctx // page)
    lens = [1] * B + [q_len] * B
    n = 2 * B
    uk, uv = (rounded(torch.randn(heads, s, rank, generator=g) * rank ** -0.5, target) for s in (dim, vdim))
    lat = torch.randn(n, ctx, rank, generator=g)
    ends = np.cumsum(lens)
    q = torch.randn(sum(lens), heads, dim, generator=g) * 0.3
    for b in range(n):
        c = lat[b, spots[b % B]] = torch.randn(rank, generator=g) * 4.0
        k = torch.einsum("hdr,r->hd", uk.float(), c)                  # every head asks for the planted latent's own key
        q[ends[b] - 1] = k * 14.0 / k.pow(2).sum(-1, keepdim=True)
    lat, q = rounded(lat, target), rounded(q, target)
    want, planted = [], []
    for b in range(n):
        k, v = torch.einsum("tr,hdr->thd", lat[b], uk), torch.einsum("tr,her->the", lat[b], uv)
        rows = q[ends[b] - lens[b]:ends[b]]
        o = R.attend(torch.cat([torch.zeros(ctx - lens[b], heads, dim).double(), rows]), k, v, 1.0)[-lens[b]:]
        want.append(o)
        planted.append(v[spots[b % B]])
        assert (o[-1] - planted[-1]).abs().max() < 0.1 * planted[-1].abs().max()     # it carries nearly all of the weight
    table = torch.randperm(n * pages, generator=g).view(n, pages).int()
    cache = torch.full((n * pages, page, rank), float("nan"), dtype=torch.float64)      # stale rows must not matter
    for b in range(n):
        for t in range(ctx):
            cache[table[b, t // page], t % page] = lat[b, t]
    cu = torch.from_numpy(np.concatenate([[0], ends]).astype(np.int32)).to(target[0])
    pos = torch.tensor([ctx - m + i for m in lens for i in range(m)], dtype=torch.int32, device=target[0])
    meta = ops.AttnMeta(cu, torch.full((n,), ctx, dtype=torch.int32, device=target[0]), table.to(target[0]), B, q_len, ctx)
    return dict(q=q, uk=uk, uv=uv, cache=cache, meta=meta, pos=pos, ends=ends), torch.cat(want), planted


def widened(t, size, dim):
    out = torch.zeros(*t.shape[:dim], size, *t.shape[dim + 1:], dtype=t.dtype)
    out.narrow(dim, 0, t.shape[dim]).copy_(t)
    return out


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("page", [8, 16, 48, 64, 128])
@pytest.mark.parametrize("heads,dim,vdim,rank", [(1, 16, 24, 64), (4, 32, 48, 128), (16, 64, 64, 512), (20, 40, 24, 96), (3, 64, 128, 1024)])
def test_latent_attention_finds_one_key(target, page, heads, dim, vdim, rank):
    """One latent's key matches the last query far better than all others: wherever it lies (first token, page borders, far
    back, the query's own place), decode rows and portions return its value."""
    a, want, planted = planted_batch(target, 300, page, 5, heads, dim, vdim, rank, page + heads)
    bf16 = target[1] == "bfloat16"
    d, e, r = (-(-dim // 64) * 64, -(-vdim // 64) * 64, next(n for n in (64, 128, 256, 512, 1024) if n >= rank)) if bf16 else (dim, vdim, rank)
    uk, uv, q = widened(widened(a["uk"], d, 1), r, 2), widened(widened(a["uv"], e, 1), r, 2), widened(a["q"], d, 2)
    cache = dev(widened(a["cache"], r, 2), target)
    rows = ops.token_rows(a["meta"], q.shape[0], torch.device(target[0]))
    q_lat = ops.head_linear(dev(q.reshape(q.shape[0], -1), target), dev(uk.transpose(1, 2).reshape(heads * r, d), target), heads)
    o_lat = ops.latent_attend(q_lat, cache, a["meta"], rows, heads, 1.0, a["pos"])
    o = ops.head_linear(o_lat, dev(uv.reshape(heads * e, r), target), heads)
    if target[0] == "cuda":
        ops.check_status()
    close(o.view(-1, heads, e)[..., :vdim], want, target, f32=5e-5, bf16=0.04)


@gpu
@pytest.mark.parametrize("page,ctx,q_len", [(16, 300, 5), (128, 300, 290), (64, 257, 129), (32, 128, 128)])
@pytest.mark.parametrize("heads,dim,vdim,rank", [(2, 128, 128, 512), (5, 100, 72, 90)])
def test_expanded_attention_finds_one_key(page, ctx, q_len, heads, dim, vdim, rank):
    """The prefill sequences of the same batches in the expanded form, gated; decode rows are left alone."""
    a, want, planted = planted_batch(BF16, ctx, page, q_len, heads, dim, vdim, rank, ctx)
    r, meta, n = next(x for x in (64, 128, 256, 512) if x >= rank), a["meta"], a["q"].shape[0]
    uk, uv, q = widened(widened(a["uk"], 128, 1), r, 2), widened(widened(a["uv"], 128, 1), r, 2), widened(a["q"], 128, 2)
    w_kv = dev(torch.cat([uk.reshape(heads * 128, r), uv.reshape(heads * 128, r)]), BF16)
    cu, ctx_lens = meta.cu_q.cpu().numpy(), meta.ctx_lens.cpu().numpy()
    blocks = -(-ctx // 128)
    S = len(ctx_lens) - meta.num_decode
    meta.expand = (torch.tensor([[s, b] for s in range(S) for b in range(blocks)], dtype=torch.int32, device="cuda"),
                   torch.arange(S * blocks, dtype=torch.int32, device="cuda").view(S, blocks))
    gate = rounded(torch.randn(n, heads * 128, generator=torch.Generator().manual_seed(1)), BF16)
    for listed in (False, True):
        if listed:
            meta.work = torch.from_numpy(ops.prefill_work_items(cu, ctx_lens, meta.num_decode)).cuda()
            meta.n_items = meta.work.shape[0]
        out = torch.full((n, heads * 128), 7.0, dtype=torch.bfloat16, device="cuda")
        ops.latent_prefill(dev(q.reshape(n, -1), BF16), dev(widened(a["cache"], r, 2), BF16), w_kv, meta, heads, 1.0, dev(gate, BF16), out)
        ops.check_status()
        nd = meta.num_decode
        assert bool((out[:nd] == 7).all())
        close(out[nd:].view(-1, heads, 128)[..., :vdim], want[nd:] * R.sigmoid(gate).view(n, heads, 128)[nd:, :, :vdim], BF16, bf16=0.04)


def test_plan_of_the_expanded_form():
    """Long portions expand, short ones do not; the pages cover every context in blocks of 128."""
    plan = lambda cu, ctx, nd, **kw: ops.plan_latent_prefill(cu, ctx, nd, **{"latent": 512, "heads": 16, "dim": 128, "vdim": 128, **kw})  # noqa: E731
    assert plan([0, 1, 2], [50, 60], 2) is None                                           # decode rows only
    assert plan([0, 8], [1000], 0) is None and plan([0, 2], [2000], 0) is None
    assert plan([0, 64], [1000], 0) is not None
    pages, tables = plan([0, 1, 501, 901], [70, 500, 700], 1)
    assert pages.tolist() == [[0, b] for b in range(4)] + [[1, b] for b in range(6)]
    assert tables[0, :4].tolist() == [0, 1, 2, 3] and tables[1].tolist() == [4, 5, 6, 7, 8, 9] and tables.max() < len(pages)
    assert plan([0, 4096], [1 << 20], 0, heads=128) is None                               # scratch would be too large
    assert plan([0, 24], [2000], 0) is not None and plan([0, 24], [2000], 0, latent=256) is None    # narrow latents are cheap to attend over


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("experts,top,rows", [(1, 1, 3), (7, 3, 1), (16, 2, 40), (64, 6, 200), (300, 4, 700), (5, 5, 300), (8, 1, 1100)])
@pytest.mark.parametrize("scoring,norm_top", [("sigmoid", False), ("softmax", True)])
def test_mixture_of_experts(target, experts, top, rows, scoring, norm_top):
    """Rows through their experts, with clamps that bite; one expert far more popular than the rest."""
    if scoring == "softmax" and experts == 300:
        pytest.skip("one scoring is enough at this size")
    g = torch.Generator().manual_seed(experts + rows)
    W, f, limit, scale = 72, 32, 0.9, 1.6
    h = rounded(torch.randn(rows, W, generator=g), target)
    router = rounded(torch.randn(experts, W, generator=g) * W ** -0.5, target)
    h[:, 0] = 2.0
    router[experts // 2, 0] = 1.5 if rows > 100 else 0.0                # most rows choose this one
    gate, up = (rounded(torch.randn(experts, f, W, generator=g) * 2 * W ** -0.5, target) for _ in range(2))
    down = rounded(torch.randn(experts, W, f, generator=g) * f ** -0.5, target)
    z = h @ router.T
    s = R.sigmoid(z) if scoring == "sigmoid" else torch.softmax(z, 1)
    best = s.topk(top, 1)
    wt = best.values / best.values.sum(1, keepdim=True) if norm_top else best.values
    want = torch.zeros(rows, W, dtype=torch.float64)
    for e in range(experts):
        share = (wt * (best.indices == e)).sum(1, keepdim=True) * scale
        want += share * (R.clipped_glu(h @ gate[e].T, h @ up[e].T, limit) @ down[e].T)
    assert bool(((h @ gate[0].T) > limit).any()) and bool(((h @ up[0].T).abs() > limit).any())
    pad = torch.zeros(-experts % 8, W, dtype=torch.float64)
    p = ops.MoeWeights(dev(torch.cat([router, pad]), target), torch.stack([dev(reference.interleave_gate_up(gate[e], up[e]), target) for e in range(experts)]),
                       dev(down, target), experts, top, scoring, norm_top, scale, ops.Glu(limit, 1.702, 1.0))
    gap = z.topk(min(top + 1, experts), 1).values
    sure = (gap[:, -2] - gap[:, -1] > 1e-4) if experts > top else torch.ones(rows, dtype=torch.bool)    # f32 scores tell these apart
    for _ in range(2):                                                   # the counters are clean again afterwards
        ex = ops.moe_experts(dev(h, target), p)
        got = torch.einsum("tk,tkw->tw", ex.weights.double().cpu(), ex.rows.double().cpu()[ex.slot.long().cpu()])
        close(got[sure], want[sure], target, bf16=0.02)
    assert sorted(ex.slot.flatten().tolist()) == list(range(rows * top))
    if target[0] == "cuda":
        ops.check_status()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("rows", [1, 37, 130, 300])
def test_epilogues(target, rows):
    """Squared ReLU, soft cap, clamped gated unit and f32 results behind a matrix product; on the GPU also on CTA pairs."""
    g = torch.Generator().manual_seed(rows)
    K, N = 104, 288
    x, w = rounded(torch.randn(rows, K, generator=g), target), rounded(torch.randn(N, K, generator=g) * 3 * K ** -0.5, target)
    xs, ws, z = dev(x, target), dev(w, target), x @ w.T
    close(ops.linear_relu2(xs, ws), z.clamp_min(0) ** 2, target)
    close(ops.linear_softcap(xs, ws, 4.0), R.softcap(z, 4.0), target)
    f = ops.linear_f32(xs, ws)
    assert f.dtype == torch.float32
    close(f, z, (target[0], "float32"))                                  # nothing is rounded to 16 bits
    gu = dev(reference.interleave_gate_up(w[:N // 2].float(), w[N // 2:].float()), target)
    glu = ops.Glu(1.25, 1.702, 1.0)
    want = R.clipped_glu(z[:, :N // 2], z[:, N // 2:], 1.25)
    close(ops.linear_swiglu(xs, gu, glu=glu), want, target)
    close(ops.linear_swiglu(xs, gu), R.sigmoid(z[:, :N // 2]) * z[:, :N // 2] * z[:, N // 2:], target)
    if target == BF16:
        out = torch.empty(rows, N, dtype=torch.bfloat16, device="cuda")
        C, st = ops._ext.require(), ops._state.get(out.device)
        C.gemm_bf16_pair(xs, ws, out, ops.EPI_RELU2, 128, st.status)
        close(out, z.clamp_min(0) ** 2, target)
        close(ops.linear_swiglu(xs, gu, config=ops.PAIR_CONFIG | 128, glu=glu), want, target)
        ops.check_status()


# ------------------------------------------------------------------------------------------------------
# configuration and bookkeeping
# ------------------------------------------------------------------------------------------------------


def test_previous_tokens_follow_the_sequences(tmp_path):
    """Portions, decode rows and requests left out of steps: each row's predecessor, -1 for a first token."""
    from mojo_b200 import _ext

    C = _ext.require()
    kv, sc = C.KVCacheManager(16, 8, False), C.SchedulerConfig()
    sc.max_num_seqs, sc.max_num_batched_tokens, sc.max_model_len = 4, 64, 64
    s = C.Scheduler(sc, kv)
    rows = lambda b: sorted(zip(b.token_ids.tolist(), b.prev_tokens.tolist()))  # noqa: E731
    assert rows(s.run_tokens([(0, [5, 6, 7]), (1, [9])])) == [(5, -1), (6, 5), (7, 6), (9, -1)]
    assert rows(s.run_tokens([(0, [8]), (2, [1, 2])])) == [(1, -1), (2, 1), (8, 7)]
    assert rows(s.run_tokens([(1, [3, 4])])) == [(3, 9), (4, 3)]
    s.append_token(1, -1)                                                # sampled, still on the device
    s.append_token(1, 6)
    assert -2 in s.step().prev_tokens.tolist()


def test_config_reading_and_refusals(tmp_path):
    from mojo_b200.models import build_model, get_config

    cfg, w = weights_of("looped")
    R.write_checkpoint(tmp_path / "m", cfg, w)
    mc = get_config(str(tmp_path / "m"))
    assert (mc.architecture, mc.num_layers, mc.hidden_size, mc.vocab_size) == ("rerupel", 4, 96, 101)
    assert [i for i, _ in mc.layer_runs()] == [0, 1, 2, 1, 2, 1, 2, 3] and [e for _, e in mc.layer_runs()] == [False, True, False, True, False, True, False, False]
    assert mc.layers[1].moe.shared.limit == 0.5 and mc.layers[3].moe.shared is None and mc.layers[2].moe is None and mc.layers[2].ffn == 0
    assert (mc.bigram.buckets, mc.bigram.mul_prev, mc.bigram.mul_cur, mc.residual_mult, mc.logit_softcap) == (53, 11, 5, 0.7, 12.0)
    model = build_model(mc)
    assert model.kv_bytes_per_page(16) == (48 + 3 * (64 + 80) + 48) * 16 * 4 and len(model.allocate_kv_cache(3, 16)) == 8

    def broken(**change):
        bad = json.loads(json.dumps(cfg))
        bad.update(change)
        (tmp_path / "m" / "config.json").write_text(json.dumps(bad))
        return lambda: get_config(str(tmp_path / "m"))

    layers = json.loads(json.dumps(cfg["layers"]))
    layers[1]["mlp"]["router"]["top"] = 8
    for change, match in (({"loop": {"start": 2, "stop": 2, "times": 1}}, "loop"), ({"loop": {"start": 0, "stop": 5, "times": 1}}, "loop"),
                          ({"layers": layers}, "experts"), ({"layers": [{**cfg["layers"][0], "type": "other"}]}, "mixer")):
        with pytest.raises(ValueError, match=match):
            broken(**change)()
    for name in ("l1.mix.uk", "bigram", "l3.mlp.e11.down"):
        R.write_checkpoint(tmp_path / "bad", cfg, {**w, name: w[name][:-1]})
        with pytest.raises(ValueError, match=name.split(".", 1)[-1]):
            LLM(PipelineConfig(model=str(tmp_path / "bad"), device="cpu"))


def test_presets_generate():
    from mojo_b200.models import get_config

    assert 15e9 > get_config("rerupel-lite").num_params() > 5e9
    llm = LLM(PipelineConfig(model="tiny-rerupel", device="cpu", random_init=True, page_size=16, num_pages=16, max_num_seqs=2, max_model_len=64))
    n = sum(t.numel() for lw in llm.engine.model.layers for t in (lw.w_in, lw.wo))
    assert n > 0 and len(llm.generate([[1, 2, 3]], SamplingParams(max_tokens=3))[0].token_ids) == 3
