"""Noridra against the plain implementation in `noridra_oracle`: every mechanism alone, whole prompts, decoding, cut prompts, mixed
batches, pages and state slots used again, and greedy generation through the scheduler. The same tests run on the CPU engine and,
marked `gpu`, on the kernels in f32 and bf16."""
import io
import json
import math

import noridra_oracle as N
import numpy as np
import pytest
import torch

from mojo_b200 import ops
from mojo_b200.pipelines import LLM, PipelineConfig, SamplingParams

gpu = pytest.mark.gpu
TARGETS = [pytest.param(("cpu", "float32"), id="cpu"), pytest.param(("cuda", "float32"), id="f32", marks=gpu),
           pytest.param(("cuda", "bfloat16"), id="bf16", marks=gpu)]
BF16 = ("cuda", "bfloat16")


def model_mixed():
    """Every kind of layer, with and without experts, sizes that differ from layer to layer."""
    return N.config(96, 101, [
        N.delta_spec(6, 2, 24, 40, 3, N.moe_spec(7, 3, 40)), N.attention_spec(6, 2, 24, 37, 8.0, N.moe_spec(6, 2, 24)),
        N.mamba_spec(80, 12, 7, 4), N.attention_spec(4, 4, 16, 64, 20.0), N.delta_spec(2, 2, 32, 16, 4),
        N.mamba_spec(48, 16, 16, 2, N.moe_spec(5, 1, 16))], groups=3)


def model_odd():
    """Sizes that are multiples of nothing much, more query heads per key head than an MMA tile has rows, one group of columns."""
    return N.config(101, 67, [
        N.attention_spec(34, 2, 18, 20, 5.0, N.moe_spec(5, 3, 20)), N.mamba_spec(37, 5, 3, 2, N.moe_spec(3, 3, 9)),
        N.delta_spec(3, 1, 13, 7, 2), N.attention_spec(3, 1, 70, 33, 30.0, N.moe_spec(5, 2, 33))], taps=3, alpha=1.2, eps=1e-3)


def model_wide():
    """Heads that fill the tensor-core prefill kernel's columns, or only in part: steps with prompt chunks replay CUDA graphs."""
    return N.config(256, 120, [
        N.attention_spec(4, 2, 128, 130, 15.0, N.moe_spec(8, 2, 48)), N.delta_spec(2, 2, 128, 128, 4), N.mamba_spec(256, 32, 20, 4, N.moe_spec(6, 2, 32)),
        N.attention_spec(3, 3, 100, 90, 15.0)], groups=2)


def model_taps():
    """Convolutions longer and shorter than usual, a head size of its own, groups of few columns."""
    return N.config(65, 50, [
        N.delta_spec(2, 1, 16, 24, 1, N.moe_spec(4, 1, 16)), N.mamba_spec(24, 3, 5, 1), N.attention_spec(2, 1, 200, 100, 12.0), N.mamba_spec(16, 40, 2, 6),
        N.delta_spec(4, 2, 8, 8, 5)], groups=5, taps=6, alpha=3.0)


def model_single():
    """One head, one expert, chunks of one position, no memory ahead of a sublayer; no recurrence at all."""
    return N.config(64, 33, [N.attention_spec(1, 1, 8, 1, 9.0, N.moe_spec(1, 1, 16)), N.attention_spec(1, 1, 16, 1000, 20.0)], groups=8, taps=1, alpha=1.0)


MODELS = {"mixed": model_mixed, "odd": model_odd, "wide": model_wide, "taps": model_taps, "single": model_single}
_cache: dict = {}


def weights_of(name):
    cfg = MODELS[name]()
    return cfg, N.random_weights(cfg, seed=len(name), sharp=2.5)


def tokens_of(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def expected(name, tokens):
    """Oracle logits of one sequence in float64, once per (model, tokens). Rounding must not decide which experts run."""
    key = (name, tuple(tokens))
    if key not in _cache:
        cfg, w = weights_of(name)
        gaps = []
        _cache[key] = N.forward(cfg, N.as_double(w), tokens, gaps=gaps)
        assert min((float(x.min()) for x in gaps), default=9.0) > 0.2
    return _cache[key]


def open_llm(tmp_path, name, target, **kw):
    device, dtype = target
    cfg, w = weights_of(name)
    N.write_checkpoint(tmp_path / name, cfg, w)
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
    err = N.relative_error(got, want)
    worst, mean = {"float32": (1e-4, 2e-5), "bfloat16": (0.08, 0.025)}[target[1]]
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
    page = 128 if name == "wide" else 32
    llm = open_llm(tmp_path, name, target, page_size=page, num_pages=-(-160 // page), max_num_seqs=1)
    for n, seed in ((1, 1), (2, 2), (33, 3), (150, 4)):
        toks = tokens_of(cfg, n, seed)
        check(run_schedule(llm.engine, {"a": toks}, [[("a", n)]])["a"], expected(name, toks), target)
        if n > 1:
            check(run_schedule(llm.engine, {"a": toks}, [[("a", max(1, n - 40))]] + [[("a", 1)]] * min(40, n - 1))["a"], expected(name, toks), target)


@pytest.mark.parametrize("target", TARGETS)
def test_stream_after_every_layer(tmp_path, target):
    """The residual that a model cut off behind each layer hands to its final norm."""
    cfg, w = weights_of("mixed")
    toks, streams = tokens_of(cfg, 45, 8), []
    N.forward(cfg, N.as_double(w), toks, streams)
    for n in range(1, len(cfg["layers"]) + 1):
        part = {**cfg, "layers": cfg["layers"][:n], "vocab": 96}
        pw = {k: v for k, v in w.items() if not k.startswith("l") or int(k[1:k.index(".")]) < n}
        pw.update(embed=w["embed"][:96], head=torch.eye(96), **{"final.norm": torch.ones(96)})
        N.write_checkpoint(tmp_path / "p", part, pw)
        llm = LLM(PipelineConfig(model=str(tmp_path / "p"), device=target[0], dtype=target[1], page_size=16, num_pages=4, max_num_seqs=1,
                                 max_num_batched_tokens=64, max_model_len=64))
        small = [t for t in toks if t < 96]
        if len(small) == len(toks):
            got = run_schedule(llm.engine, {"a": toks}, [[("a", 20)], [("a", 2)], [("a", 23)]])["a"]
            check(got, N.group_norm(streams[n - 1], 1.0, 3, 1e-5), target)
        else:
            out = []
            N.forward(cfg, N.as_double(w), small, out)
            got = run_schedule(llm.engine, {"a": small}, [[("a", 20)], [("a", 2)], [("a", len(small) - 22)]])["a"]
            check(got, N.group_norm(out[n - 1], 1.0, 3, 1e-5), target)


@pytest.mark.parametrize("name", sorted(MODELS))
@pytest.mark.parametrize("target", TARGETS)
def test_portions(tmp_path, target, name):
    """Prompts cut into portions of changing size, down to two tokens and to one, across page and chunk borders."""
    cfg, _ = weights_of(name)
    llm = open_llm(tmp_path, name, target, page_size=128 if name in ("odd", "wide") else 32)
    toks = tokens_of(cfg, 150, 4)
    for cuts in ([2] * 10 + [3] * 5 + [2, 27, 1, 31, 2, 50, 2], [31, 2, 30, 1, 1, 2, 33, 50]):
        assert sum(cuts) == 150
        check(run_schedule(llm.engine, {"a": toks}, [[("a", c)] for c in cuts])["a"], expected(name, toks), target)


@pytest.mark.parametrize("page", [8, 16, 64, 128])
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "wide", "taps"])
def test_unequal_batches_with_reuse(tmp_path, target, name, page):
    """Four live requests in one batch, portions beside decoded tokens, some left out of steps; pages and state slots only fit
    the live ones, so later requests use what others gave back."""
    if name != "mixed" and target[0] == "cpu" and page != 64:
        pytest.skip("one page size is enough for the plain operations")
    cfg, _ = weights_of(name)
    lengths = {"a": 150, "b": 33, "c": 70, "d": 1, "e": 90, "f": 33}
    req = {k: tokens_of(cfg, n, {"a": 4, "b": 3}.get(k, ord(k))) for k, n in lengths.items()}
    if name == "taps" and page == 8:
        page = 32                                        # heads of 256 columns in pages that the TMA boxes fit
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
    if name == "wide" and page == 128 and target == BF16:
        assert llm.engine.runner.mixed_launches > 0


@pytest.mark.parametrize("target", TARGETS)
def test_long_decoding(tmp_path, target):
    """Hundreds of decoded tokens, several chunks and pages; on the GPU replayed as CUDA graphs."""
    cfg, _ = weights_of("mixed")
    toks = tokens_of(cfg, 300, 9)
    llm = open_llm(tmp_path, "mixed", target)
    check(run_schedule(llm.engine, {"a": toks}, [[("a", 4)]] + [[("a", 1)]] * 296)["a"], expected("mixed", toks), target)
    if target[0] == "cuda":
        assert llm.engine.runner.graph_launches >= 290


def greedy(name, prompt, n):
    cfg, w = weights_of(name)
    w = N.as_double(w)
    toks, lead = list(prompt), []
    for _ in range(n):
        top = N.forward(cfg, w, toks)[-1].topk(2)
        lead.append(float(top.values[0] - top.values[1]))
        toks.append(int(top.indices[0]))
    return toks[len(prompt):], lead


@pytest.mark.parametrize("target", TARGETS)
def test_greedy_generation_through_the_scheduler(tmp_path, target):
    """`LLM.generate` with a token budget that cuts prompts and a pool that runs out of pages (preemption and
    recomputation): the tokens of the plain implementation."""
    cfg, _ = weights_of("mixed")
    prompts = [tokens_of(cfg, n, 20 + i) for i, n in enumerate((30, 14, 30, 1, 20))]
    want = [greedy("mixed", p, 12) for p in prompts]
    llm = open_llm(tmp_path, "mixed", target, page_size=16, num_pages=5, max_num_seqs=3, max_num_batched_tokens=24, max_model_len=96)
    outs = llm.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    for o, (toks, lead) in zip(outs, want):
        # bf16: compare up to the first step whose two best logits are closer than rounding can tell apart
        n = 12 if target[1] == "float32" else next((i for i, m in enumerate(lead) if m < 0.3), 12)
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
    N.write_checkpoint(tmp_path / "m", cfg, w)
    prompt = tokens_of(cfg, 9, 5)
    cli.main(["generate", "--model", str(tmp_path / "m"), "--device", "cpu", "--token-ids", "--prompt", ",".join(map(str, prompt)), "--max-tokens", "4",
              "--max-num-seqs", "2", "--num-pages", "8", "--page-size", "16", "--max-model-len", "64"])
    assert json.loads(capsys.readouterr().out.strip().splitlines()[-1])["token_ids"] == greedy("mixed", prompt, 4)[0]

    lines = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:5], "want": [1, 4]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[5:7], "want": []}, {"id": "y", "tokens": prompt[:1], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "y", "tokens": prompt[:2], "want": []}, {"id": "x", "tokens": prompt[7:], "want": [1]}], "end": ["x", "y"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    with pytest.raises(SystemExit) as done:
        cli.main(["replay", "--model", str(tmp_path / "m"), "--dtype", "float32", "--device", "cpu", "--out", str(tmp_path / "o"), "--max-tokens", "1024"])
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
    return t.to(device=target[0], dtype=dtype or getattr(torch, target[1])).contiguous().clone()


def f32(t, target):
    return dev(t, target, torch.float32)


def rounded(t, target):
    """float64 values that `target`'s element type holds exactly."""
    return t.to(getattr(torch, target[1])).double()


def sync(target):
    if target[0] == "cuda":
        ops.check_status()


def seq_rows(lengths, banks, target, pad=0):
    """SeqRows of sequences with these row counts, the first ones of one row being the decode rows, and `pad` rows of no sequence
    behind them. banks: [(read, write)]."""
    ends = np.cumsum(lengths)
    rows = np.stack([ends - lengths, ends], axis=1).astype(np.int32)
    n_dec = next((i for i, n in enumerate(lengths) if n != 1), len(lengths))
    of = np.concatenate([np.repeat(np.arange(len(lengths)), lengths), np.full(pad, -1)]).astype(np.int32)
    return ops.SeqRows(torch.from_numpy(of).to(target[0]), torch.from_numpy(rows).to(target[0]), torch.tensor(banks, dtype=torch.int32, device=target[0]),
                       n_dec, n_dec, len(lengths) - n_dec)


def history(x, taps):
    """The last taps - 1 rows of x, zeros ahead of its first."""
    return torch.cat([torch.zeros(taps, x.shape[1], dtype=x.dtype), x])[-(taps - 1):] if taps > 1 else None


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("width,pad,groups,taps,top", [(96, 96, 3, 4, 2), (101, 104, 1, 3, 9), (65, 72, 5, 6, 1), (64, 64, 64, 1, 3), (2048, 2048, 4, 4, 6),
                                                       (4096, 4096, 1, 4, 1), (1024, 1024, 8, 16, 4), (8192, 8192, 1, 2, 2), (1030, 1032, 2, 4, 5), (1111, 1112, 1, 5, 2)])
def test_norm_after_the_sum_and_input_convolution(target, width, pad, groups, taps, top):
    """A stream takes up rows of a product or of experts (weighted and not), is normalised group by group and convolved: decode
    rows, portions shorter and longer than the history and than a tile, fresh sequences, unused entries, rows of no sequence. A far
    larger group must not disturb its neighbours, and only the last rows are remembered."""
    if target[0] == "cpu" and width > 2000:
        pytest.skip("sizes of the kernels' variants")
    g = torch.Generator().manual_seed(width)
    dtype, eps, alpha = getattr(torch, target[1]), 1e-2, 1.7
    lens, extra = [1, 1, 1, 2, 75, 5], 3
    T, n = sum(lens) + extra, len(lens)
    banks = [(0, 1), (-1, 3), (-1, -1), (5, 4), (7, 6), (-1, 8)]             # the third entry is unused
    seq = seq_rows(lens, banks, target, extra)

    def rnd(*s):
        t = torch.zeros(*s[:-1], pad, dtype=torch.float64)
        t[..., :width] = rounded(torch.randn(*s, generator=g), target)
        return t

    x, y, rows = rnd(T, width), rnd(T, width), rnd(T * top, width)
    x = x.float().double()
    if groups > 1:
        x[:, :width // groups] *= 50.0
    scale, weight, then = (rnd(width).float() + 1.0 for _ in range(3))
    w = torch.zeros(taps, pad)
    w[:, :width] = torch.randn(taps, width, generator=g) * 0.5
    slot, wts = torch.randperm(T * top, generator=g).view(T, top), torch.rand(T, top, generator=g)
    picked = rows[slot]
    norm = ops.GroupNorm(groups, eps, width)
    real = lambda t: t[..., :width].double()  # noqa: E731
    for kind in ("rows", "experts", "weighted", "start"):
        bank = torch.randn(10, max(taps - 1, 1), pad, generator=g)           # stale contents everywhere
        past = [torch.randn(7, width, generator=g).double() if rd >= 0 else torch.zeros(0, width, dtype=torch.float64) for rd, _ in banks]
        for p, (rd, _) in zip(past, banks):
            if rd >= 0 and taps > 1:
                bank[rd] = 0
                bank[rd, :, :width] = history(p, taps).float()
        past = [p.float().double() for p in past]
        state = f32(bank, target) if taps > 1 else None
        conv = ops.InputConv(f32(w, target), state)
        if kind == "start":
            table, pos_table = rnd(11, width), rnd(40, width)
            ids, pos = torch.randint(0, 11, (T,), generator=g), torch.randint(0, 40, (T,), generator=g)
            start = ops.StreamStart(ids.to(target[0]), dev(table, target), pos_table=dev(pos_table, target), positions=dev(pos, target, torch.int32))
            h, new = ops.post_norm(None, norm, dtype, seq, start=start, conv=conv)
            want = real(table[ids] + pos_table[pos])
        else:
            if kind == "rows":
                done, add = ops.Finished(f32(scale, target), dev(y, target)), real(scale) * real(y)
            elif kind == "experts":
                done, add = ops.Finished(None, None, ops.ExpertRows(dev(rows, target), dev(slot, target, torch.int32), None)), real(picked).sum(1)
            else:
                done = ops.Finished(f32(scale, target), dev(y, target), ops.ExpertRows(dev(rows, target), dev(slot, target, torch.int32), f32(wts, target)))
                add = real(scale) * (real(y) + torch.einsum("tk,tkw->tw", wts.double(), real(picked)))
            kw = dict(done=done, weight=f32(weight, target), alpha=alpha)
            old = f32(x, target)
            h, new = ops.post_norm(old, norm, dtype, seq, conv=conv, **kw)
            assert torch.equal(old.cpu(), x.float())
            want = N.group_norm(alpha * real(x) + add, real(weight), groups, eps)
            pick = torch.tensor([T - 1, 3, 0, 40], device=target[0])
            last, none = ops.post_norm(old, norm, dtype, seq, then=f32(then, target), rows=pick, **kw)
            close(last[:, :width], N.group_norm(want, real(then), groups, eps)[pick.cpu()], target)
            assert none is None and float(last[:, width:].abs().sum()) == 0
        sync(target)
        row = 0
        for i, (m, p, (rd, wr)) in enumerate(zip(lens, past, banks)):
            a, b = row, row + m
            row = b
            if wr < 0:
                assert float(h[a:b].abs().sum()) == 0 and float(new[a:b].abs().sum()) == 0
                continue
            full = torch.cat([p, want[a:b]])
            close(new[a:b, :width], want[a:b], (target[0], "float32"), f32=1e-5)
            close(h[a:b, :width], (full + N.conv(full, w[:, :width].t().double()))[len(p):], target)
            if taps > 1:
                close(state[wr, :, :width], history(full, taps), (target[0], "float32"), f32=1e-5)
        assert float(h[row:].abs().sum()) == 0 and float(new[row:].abs().sum()) == 0
        assert float(h[:, width:].abs().sum()) == 0 and float(new[:, width:].abs().sum()) == 0
        if taps > 1:
            for b in set(range(10)) - {wr for _, wr in banks}:
                assert torch.equal(state[b].cpu(), bank[b])


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,kv,dim,T", [(1, 1, 8, 5), (6, 2, 24, 5), (8, 1, 64, 300), (5, 5, 13, 5), (4, 2, 128, 700), (34, 2, 18, 5), (3, 1, 200, 40), (40, 4, 128, 600),
                                            (2, 1, 256, 5)])
def test_head_norms_and_values_that_are_keys(target, heads, kv, dim, T):
    """Every head has a norm of its own; keys in the cache are normalised, values are the keys as projected."""
    g = torch.Generator().manual_seed(heads + dim)
    page, nq, nk = 4, heads * dim, kv * dim
    pad = next(x for x in (64, 128, 256) if x >= dim) if target[1] == "bfloat16" else dim
    proj = rounded(torch.randn(T, nq + nk + 24, generator=g), target)
    proj[:, :dim] *= 30.0                                                    # the norm of a head is its own
    qw, kw = torch.randn(dim, generator=g), torch.randn(dim, generator=g)
    slots = torch.randperm(4 * T, generator=g)[:T]
    slots[1] = -1
    kc, vc = (dev(torch.zeros(T, kv, page, pad), target) for _ in range(2))
    q = ops.head_norm_qkv(dev(proj, target), f32(qw, target), f32(kw, target), slots.to(target[0]), kc, vc, heads, kv, dim, nq, pad, 1e-2)
    sync(target)
    k = proj[:, nq:nq + nk].view(T, kv, dim)
    got = q.view(T, heads, -1)
    close(got[..., :dim], N.rms(proj[:, :nq].view(T, heads, dim), 1e-2) * qw.double(), target)
    assert float(got[..., dim:].abs().sum()) == 0
    kept = slots >= 0
    at = slots[kept].to(target[0])
    flat = lambda c: c.transpose(1, 2).flatten(0, 1)  # noqa: E731
    close(flat(kc)[at][..., :dim], (N.rms(k, 1e-2) * kw.double())[kept], target)
    assert torch.equal(flat(vc)[at][..., :dim].double().cpu(), k[kept])
    empty = torch.ones(T * page, dtype=torch.bool)
    empty[slots[kept]] = False
    for c in (kc, vc):
        assert float(c[..., dim:].abs().sum()) == 0 and float(flat(c)[empty.to(target[0])].abs().sum()) == 0


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("chunk", [1, 2, 31, 64, 100, 127, 128, 129, 299, 300, 5000])
@pytest.mark.parametrize("heads,kv,dim,page", [(6, 2, 24, 16), (4, 1, 128, 128), (3, 3, 200, 64), (20, 1, 64, 32), (2, 2, 100, 8)])
def test_chunks_distance_bias_sink_and_gate(target, chunk, heads, kv, dim, page):
    """Keys on both sides of a chunk's border, own and far ones, for decode rows and portions at several places of a chunk, on every
    attention kernel. Every query strongly asks for one key, against the bias, or for none, so that the sink takes most."""
    if target[0] == "cpu" and chunk not in (1, 100, 300):
        pytest.skip("three chunks are enough for the plain operations")
    g = torch.Generator().manual_seed(chunk + dim)
    ctxs, lens, cap = [300, 257, 128, 1, 300, 229, 140], [1, 1, 1, 1, 140, 2, 140], 25.0
    n, n_dec, per = len(lens), 4, heads // kv
    r1, r2 = torch.rand(heads, generator=g) * 2 + 0.1, torch.rand(heads, generator=g) * 0.7 + 0.05
    k = [rounded(torch.randn(c, kv, dim, generator=g), target) for c in ctxs]
    v = [rounded(torch.randn(c, kv, dim, generator=g), target) for c in ctxs]
    qs, want = [], []
    for b, (c, m) in enumerate(zip(ctxs, lens)):
        q = torch.randn(m, heads, dim, generator=g).double() * 0.2
        for i in range(m):
            p = c - m + i
            spot = [p - p % chunk, p - p % chunk - 1, p, 0, None][(b + i) % 5]
            if spot is None:
                q[i] = 0.0
            elif spot >= 0:
                key = k[b][spot].repeat_interleave(per, dim=0)
                q[i] = key * 16.0 / key.pow(2).sum(-1, keepdim=True)
        q = rounded(q, target)
        qs.append(q)
        full = torch.cat([torch.zeros(c - m, heads, dim).double(), q])
        want.append(N.attend(full, k[b], v[b], 1.0, cap, r1.double(), r2.double(), chunk)[-m:])
    T, gate = sum(lens), rounded(torch.randn(sum(lens), heads * dim, generator=g), target)
    want = torch.cat(want) * N.sigmoid(gate).view(T, heads, dim)
    pages = -(-300 // page)
    table = torch.randperm(n * pages, generator=g).view(n, pages).int()
    pad = next(x for x in (64, 128, 256) if x >= dim) if target[1] == "bfloat16" else dim
    kc, vc = (torch.zeros(n * pages, kv, page, pad, dtype=torch.float64) for _ in range(2))
    for b, c in enumerate(ctxs):
        for t in range(c):
            kc[table[b, t // page], :, t % page, :dim], vc[table[b, t // page], :, t % page, :dim] = k[b][t], v[b][t]
    seq = seq_rows(lens, [(0, 0)] * n, target)
    cu = torch.from_numpy(np.concatenate([[0], np.cumsum(lens)]).astype(np.int32)).to(target[0])
    pos = torch.tensor([c - m + i for c, m in zip(ctxs, lens) for i in range(m)], dtype=torch.int32, device=target[0])
    meta = ops.AttnMeta(cu, torch.tensor(ctxs, dtype=torch.int32, device=target[0]), table.to(target[0]), n_dec, 140, 300, seq=seq)

    def wide(t):
        out = torch.zeros(T, heads, pad, dtype=torch.float64)
        out[..., :dim] = t.view(T, heads, dim)
        return dev(out.view(T, -1), target)

    mods = ops.ScoreMods(softcap=cap, chunk=chunk, sink=True, distance=f32(torch.stack([r1, r2]), target))
    out = torch.zeros(T, heads * pad + 16, dtype=getattr(torch, target[1]), device=target[0])
    ops.paged_attention(wide(torch.cat(qs)), dev(kc, target), dev(vc, target), meta, 1.0, pad, out=out[:, 16:], gate=wide(gate), positions=pos, mods=mods)
    sync(target)
    close(out[:, 16:].view(T, heads, pad)[..., :dim], want, target, f32=5e-5, bf16=0.03)
    assert float(out[:, :16].abs().sum()) == 0


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,kv,dim,vdim,taps", [(4, 2, 32, 48, 4), (2, 2, 128, 128, 4), (3, 1, 20, 13, 2), (2, 1, 200, 256, 3), (1, 1, 8, 64, 1), (6, 3, 64, 20, 4), (2, 2, 1, 4, 4)])
def test_delta_rule_with_decays_per_head(target, heads, kv, dim, vdim, taps):
    """Decode rows and portions continued from given matrices and banks, decays from almost none to almost total, silu gates."""
    g = torch.Generator().manual_seed(dim + vdim)
    past, now, slots = [9, 40, 2, 0], [1, 1, 21, 37], [3, 0, 4, 1]
    ck, nv = kv * dim, heads * vdim
    C, b_off = 2 * ck + nv, 2 * ck + nv + 3
    a_off, g_off = b_off + heads + 2, -(-(b_off + 2 * heads + 2) // 8) * 8
    full = [rounded(torch.randn(p + n, g_off + nv, generator=g), target) for p, n in zip(past, now)]
    w, a_log = torch.randn(C, taps, generator=g).double() * 0.7, torch.linspace(-4.0, 1.5, heads).double()
    bias, norm = torch.randn(heads, generator=g).double() - 1.0, 1 + torch.randn(vdim, generator=g).double() * 0.2

    def oracle(f):
        u, T = N.silu(N.conv(f[:, :C], w)), f.shape[0]
        q, k = (N.unit(u[:, o:o + ck].reshape(T, kv, dim)).repeat_interleave(heads // kv, 1) for o in (0, ck))
        decay = torch.exp(-torch.exp(a_log) * N.softplus(f[:, a_off:a_off + heads] + bias))
        return (q * dim ** -0.5, k, u[:, 2 * ck:].reshape(T, heads, vdim), decay, N.sigmoid(f[:, b_off:b_off + heads])), N.silu(f[:, g_off:])

    state, bank = torch.randn(5, heads, dim, vdim, generator=g), torch.randn(10, max(taps - 1, 1), C, generator=g)
    want_o, want_s = [], []
    for f, p, slot in zip(full, past, slots):
        args, gate = oracle(f)
        _, s0 = N.delta_recurrence(*(a[:p] for a in args))
        o, s1 = N.delta_recurrence(*(a[p:] for a in args), s0)
        want_o.append((N.rms(o, 1e-4) * norm).reshape(-1, nv) * gate[p:])
        want_s.append(s1)
        if p:
            state[slot] = s0.float()
            if taps > 1:
                bank[2 * slot + 1] = history(f[:p, :C], taps).float()
    st, bk = f32(state, target), dev(bank, target) if taps > 1 else None
    seq = seq_rows(now, [(2 * s + 1 if p else -1, 2 * s) for s, p in zip(slots, past)], target)
    proj = dev(torch.cat([f[p:] for f, p in zip(full, past)]), target)
    p = ops.DeltaParams(f32(w.T, target), f32(-torch.exp(a_log), target), f32(bias, target), f32(norm, target), True)
    out = ops.delta_rule(proj, proj[:, a_off:a_off + heads], proj[:, g_off:], p, bk, st, seq, b_off, heads, kv, dim, vdim, nv + 5, 1e-4)
    sync(target)
    close(out[:, :nv], torch.cat(want_o), target)
    assert float(out[:, nv:].abs().sum()) == 0
    for slot, s1, f in zip(slots, want_s, full):
        close(st[slot], s1, (target[0], "float32"))
        if taps > 1:
            assert torch.equal(bk[2 * slot].double().cpu(), history(f[:, :C], taps))
    assert torch.equal(st[2].cpu(), state[2])


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("channels,taps,bias", [(24, 4, True), (64, 1, True), (1000, 3, False), (130, 2, True), (40, 7, True), (33, 4, True)])
def test_convolution_with_silu(target, channels, taps, bias):
    """Decode rows, portions shorter and longer than the history, unused entries; the banks of the next step."""
    g = torch.Generator().manual_seed(channels)
    past, now, banks = [9, 0, 1, 0, 6], [1, 1, 2, 29, 1], [(0, 1), (-1, 3), (4, 5), (-1, 7), (9, 8)]
    x = [rounded(torch.randn(p + n, channels + 8, generator=g), target) for p, n in zip(past, now)]
    w, b = torch.randn(channels, taps, generator=g).double(), torch.randn(channels, generator=g).double() if bias else None
    bank = rounded(torch.randn(10, max(taps - 1, 1), channels, generator=g), target)
    for f, p, (rd, _) in zip(x, past, banks):
        if rd >= 0 and taps > 1:
            bank[rd] = history(f[:p, :channels], taps)
    proj, state = dev(torch.cat([f[p:] for f, p in zip(x, past)]), target), dev(bank, target) if taps > 1 else None
    got = ops.conv_silu(proj, f32(w.T, target), f32(b, target) if bias else None, state, seq_rows(now, banks, target))
    sync(target)
    want = [N.silu(N.conv(f[:, :channels], w) + (b if bias else 0.0))[p:] for f, p in zip(x, past)]
    close(got, torch.cat(want), target)
    if taps > 1:
        for f, (_, wr) in zip(x, banks):
            assert torch.equal(state[wr].double().cpu(), history(f[:, :channels], taps))


def scan_inputs(g, T, C, S, target):
    """Step sizes and rates that make states forget at once, or over thousands of rows."""
    dt, u, z = torch.randn(T, C, generator=g) * 2, *(rounded(torch.randn(T, C, generator=g), target) for _ in range(2))
    b, c = (rounded(torch.randn(T, S, generator=g), target) for _ in range(2))
    A = -torch.exp(torch.rand(C, S, generator=g).double() * 7 - 5)
    return dt.float(), u, z, b, c, A, torch.randn(C, generator=g) - 2.0, torch.randn(C, generator=g)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("channels,states,size", [(8, 4, 3), (40, 8, 8), (64, 16, 12), (136, 16, 16), (32, 32, 32), (24, 64, 40), (16, 128, 128), (8, 256, 200),
                                                  (8192, 16, 16), (4096, 32, 32)])
def test_selective_scan(target, channels, states, size):
    """Decode rows beside portions of several lengths, fresh sequences and ones with history, an unused entry; states land in their
    slots, other slots stay as they are, and a fresh sequence ignores what its slot held. States past `size` are padding."""
    if channels > 1000 and target[0] == "cpu":
        pytest.skip("sizes of the kernels' variants")
    g = torch.Generator().manual_seed(channels + states)
    lens = [1] * 11 + [37, 2, 70, 5, 16] if channels < 1000 else [1, 1, 1, 20, 3] + [17] * 12
    n, T = len(lens), sum(lens)
    slots = torch.randperm(n + 2, generator=g)[:n].tolist()
    fresh = [i % 3 == 1 for i in range(n)]
    banks = [(-1 if f else 2 * s, 2 * s + 1) for f, s in zip(fresh, slots)]
    banks[2] = (-1, -1)
    dt, u, z, b, c, A, bias, d = scan_inputs(g, T, channels, states, target)
    for t in (b, c, A):
        t[:, size:] = 0.0
    state = torch.randn(n + 2, channels, states, generator=g)
    state[..., size:] = 0.0
    st = f32(state, target)
    mid = dev(torch.cat([b, c, torch.zeros(T, 8).double()], 1), target)      # column slices of one product
    p = ops.ScanParams(f32(A * math.log2(math.e), target), f32(bias, target), f32(d, target))
    got = ops.selective_scan(f32(dt, target), dev(u, target), dev(z, target), mid[:, :states], mid[:, states:2 * states], p, st, seq_rows(lens, banks, target))
    sync(target)
    row, last, step = 0, state.double(), N.softplus(dt.double() + bias.double())
    for m, f, s, (_, wr) in zip(lens, fresh, slots, banks):
        at = slice(row, row + m)
        row += m
        if wr < 0:
            continue
        y, last[s] = N.scan(step[at], A, u[at], b[at], c[at], d.double(), None if f else last[s])
        close(got[at], y * N.silu(z[at]), target)
    close(st, last, (target[0], "float32"))


@pytest.mark.parametrize("target", TARGETS)
def test_scan_does_not_depend_on_the_cuts(target):
    """Long prompts in one piece, in portions and token by token, with states that hardly decay: the same outputs and state, and
    those of the plain recurrence."""
    g = torch.Generator().manual_seed(1)
    T, C, S = 700, 16, 16
    dt, u, z, b, c, A, bias, d = scan_inputs(g, T, C, S, target)
    A, bias = A * 0.02, bias - 2.0
    p = ops.ScanParams(f32(A * math.log2(math.e), target), f32(bias, target), f32(d, target))
    args = [f32(dt, target)] + [dev(t, target) for t in (u, z, b, c)]

    def run(cuts):
        st, out, a = torch.full((2, C, S), 9.0, device=target[0]), [], 0
        for i, n in enumerate(cuts):
            out.append(ops.selective_scan(*(t[a:a + n] for t in args), p, st, seq_rows([n], [(-1 if i == 0 else 2 + (i + 1) % 2, 2 + i % 2)], target)))
            a += n
        sync(target)
        return torch.cat(out).float().cpu(), st[1].cpu()

    y, S_last = N.scan(N.softplus(dt.double() + bias.double()), A, u, b, c, d.double())
    for cuts in ([T], [2] * 350, [1] * T, [64, 1, 3, 1, 560, 71], [T - 1, 1]):
        got = run(cuts)
        close(got[0], y * N.silu(z), target)
        close(got[1], S_last, (target[0], "float32"), f32=3e-6 if target[1] == "float32" else 2e-5)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("experts,top,rows", [(1, 1, 3), (7, 3, 40), (16, 1, 300), (64, 6, 200), (300, 5, 300), (5, 5, 10), (40, 32, 20)])
def test_weights_on_the_experts_input(target, experts, top, rows):
    """Sigmoid scores, not divided by their sum; a score multiplies what its expert reads, which the gated unit does not undo."""
    g = torch.Generator().manual_seed(experts + rows)
    W, f = 72, 32
    h = rounded(torch.randn(rows, W, generator=g), target)
    router = rounded(torch.randn(experts, W, generator=g) * 1.5 * W ** -0.5, target)
    w = {"router": router}
    for e in range(experts):
        w.update({f"e{e}.gate": rounded(torch.randn(f, W, generator=g) * 3 * W ** -0.5, target), f"e{e}.up": rounded(torch.randn(f, W, generator=g) * 2 * W ** -0.5, target),
                  f"e{e}.down": rounded(torch.randn(W, f, generator=g) * f ** -0.5, target)})
    gaps = []
    want = N.mixture(h, w, "", {"router": {"experts": experts, "top": top}}, gaps)
    sure = gaps[0] > 1e-4 if gaps else torch.ones(rows, dtype=torch.bool)
    assert sure.float().mean() > 0.9
    gu = torch.stack([ops.reference.interleave_gate_up(w[f"e{e}.gate"].float(), w[f"e{e}.up"].float()) for e in range(experts)])
    down = torch.stack([w[f"e{e}.down"] for e in range(experts)])
    p = ops.MoeWeights(dev(torch.cat([router, torch.zeros(-experts % 8, W).double()]), target), dev(gu, target), dev(down, target), experts, top, "sigmoid", on_input=True)
    hd = dev(h, target)
    for _ in range(2):                                                       # the counters are clean again afterwards
        ex = ops.moe_experts(hd, p)
        assert ex.weights is None and ex.own is None
        close(ex.rows.double().cpu()[ex.slot.long().cpu()].sum(1)[sure], want[sure], target, bf16=0.02)
    assert ex.slot.unique().numel() == rows * top
    sync(target)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("scoring", ["sigmoid", "softmax"])
def test_choice_among_scores_that_round_to_the_same(target, scoring):
    """Where scores are one (or zero) in 32 bits, the larger logit still goes first."""
    E, top, rows, W = 24, 3, 50, 16
    g = torch.Generator().manual_seed(2)
    logits = torch.stack([torch.randperm(E, generator=g) * (0.25 if scoring == "sigmoid" else 8.0) + (20.0 if scoring == "sigmoid" else -100.0) for _ in range(rows)])
    h = torch.zeros(rows, W) + 1.0
    gu, down = torch.zeros(E, 32, W), torch.zeros(E, W, 16)
    for e in range(E):                                                       # an expert's result names it
        gu[e, :, 0], down[e, :, 0] = 1.0, e + 1.0
    p = ops.MoeWeights(dev(torch.zeros(E, W), target), dev(gu, target), dev(down, target), E, top, scoring)
    ex = ops.moe_experts(dev(h, target), p, f32(logits, target))
    sync(target)
    name = ex.rows.float().cpu()[ex.slot.long().cpu()][..., 0] / (1.0 / (1.0 + math.exp(-1.0)))
    assert torch.equal(name.round().long() - 1, logits.topk(top, dim=1).indices)


# ------------------------------------------------------------------------------------------------------
# configuration and bookkeeping
# ------------------------------------------------------------------------------------------------------


def test_config_reading_and_refusals(tmp_path):
    from mojo_b200.models import build_model, get_config

    cfg, w = weights_of("mixed")
    N.write_checkpoint(tmp_path / "m", cfg, w)
    mc = get_config(str(tmp_path / "m"))
    assert (mc.architecture, mc.num_layers, mc.hidden_size, mc.vocab_size, mc.max_position_embeddings) == ("noridra", 6, 96, 101, 512)
    assert (mc.residual_alpha, mc.norm_groups, mc.input_taps, mc.rms_norm_eps) == (1.5, 3, 4, 1e-5)
    assert (mc.layers[1].chunk, mc.layers[1].softcap, mc.layers[1].moe.top, mc.layers[3].moe) == (37, 8.0, 2, None)
    assert (mc.layers[2].inner, mc.layers[2].state, mc.layers[2].dt_rank, mc.layers[2].conv_taps, mc.layers[0].conv_taps) == (80, 12, 7, 4, 3)
    model = build_model(mc)
    assert model.kv_bytes_per_page(16) == 2 * (2 * 24 + 4 * 16) * 16 * 4 and mc.kv_bytes_per_token(4) * 16 == model.kv_bytes_per_page(16)
    conv = 2 * (2 * (4 * 24 + 240) + 3 * 80 + 3 * (2 * 64 + 32) + 48)
    assert model.state_bytes_per_slot() == (6 * 24 * 40 + 80 * 16 + 2 * 32 * 16 + 48 * 16 + conv + 2 * 3 * 96 * 9) * 4
    caches = model.allocate_kv_cache(3, 16, 5)
    held = sum(t.numel() * t.element_size() for c in caches for t in vars(c).values() if t is not None)
    assert held == 3 * model.kv_bytes_per_page(16) + 5 * model.state_bytes_per_slot()

    def broken(edit):
        bad = json.loads(json.dumps(cfg))
        edit(bad)
        (tmp_path / "m" / "config.json").write_text(json.dumps(bad))
        return get_config(str(tmp_path / "m"))

    for edit, match in ((lambda c: c["layers"][0].update(type="other"), "mixer"), (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "key heads"),
                        (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "experts"), (lambda c: c["layers"][0]["mlp"].update(kind="other"), "feed-forward"),
                        (lambda c: c["layers"][1]["mixer"].update(vdim=8), "values"), (lambda c: c["norm"].update(groups=5), "groups")):
        with pytest.raises(ValueError, match=match):
            broken(edit)
    for edit, match in ((lambda c: c["canon"].update(taps=17), "taps"), (lambda c: c["layers"][2]["mixer"].update(state=300), "states"),
                        (lambda c: c["layers"][0]["mixer"].update(dim=300), "columns")):
        with pytest.raises(ValueError, match=match):
            build_model(broken(edit))
    for name in ("l1.mix.k.norm", "head", "pos", "l1.mlp.e5.down", "l0.mix.q.conv", "l2.mix.A_log", "l3.canon1"):
        N.write_checkpoint(tmp_path / "bad", cfg, {**w, name: w[name][:-1]})
        with pytest.raises(ValueError, match=name.split(".", 1)[-1]):
            LLM(PipelineConfig(model=str(tmp_path / "bad"), device="cpu"))


def test_positions_end_with_their_table(tmp_path):
    """The context limit is the number of learned positions, whatever is asked for; the last one can be used."""
    cfg, w = weights_of("single")
    cfg, w = {**cfg, "max_positions": 40}, {**w, "pos": w["pos"][:40]}
    N.write_checkpoint(tmp_path / "s", cfg, w)
    llm = LLM(PipelineConfig(model=str(tmp_path / "s"), device="cpu", page_size=16, num_pages=8, max_num_seqs=2, max_model_len=100))
    assert llm.engine.cfg.max_model_len == 40
    toks = tokens_of(cfg, 40, 1)
    check(run_schedule(llm.engine, {"a": toks}, [[("a", 30)], [("a", 10)]])["a"], N.forward(cfg, N.as_double(w), toks), ("cpu", "float32"))
    with pytest.raises(ValueError):
        llm.engine.run_tokens([(7, toks + [1], [])], [7])
    assert len(llm.generate([toks[:38]], SamplingParams(max_tokens=9, ignore_eos=True))[0].token_ids) == 2


def test_presets_generate():
    from mojo_b200.models import build_model, get_config

    assert 20e9 > get_config("noridra-lite").num_params() > 5e9
    mc = get_config("tiny-noridra")
    model = build_model(mc)
    n = sum(int(np.prod(s)) for s in model.global_shapes().values())
    n += sum(int(np.prod(s)) for spec in mc.layers for s in model.tensor_shapes(spec, mc.hidden_size).values())
    assert abs(n - mc.num_params()) < 0.01 * n
    llm = LLM(PipelineConfig(model="tiny-noridra", device="cpu", random_init=True, page_size=16, num_pages=16, max_num_seqs=2, max_model_len=64))
    assert len(llm.generate([[1, 2, 3]], SamplingParams(max_tokens=3))[0].token_ids) == 3
