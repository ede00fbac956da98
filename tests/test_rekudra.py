"""Rekudra against the plain implementation in `rekudra_oracle`: every mechanism alone, whole prompts, decoding, cut
prompts, mixed batches, pages and slots used again, and greedy generation through the scheduler. The same tests run on
the CPU engine and, marked `gpu`, on the kernels in f32 and bf16."""
import json

import numpy as np
import pytest
import rekudra_oracle as R
import torch

from mojo_b200 import ops
from mojo_b200.pipelines import LLM, PipelineConfig, SamplingParams

gpu = pytest.mark.gpu
TARGETS = [pytest.param(("cpu", "float32"), id="cpu"), pytest.param(("cuda", "float32"), id="f32", marks=gpu),
           pytest.param(("cuda", "bfloat16"), id="bf16", marks=gpu)]
LLAMA_SCALING = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}


def model_mixed():
    """Grouped heads everywhere, key size != value size, partial rotation, layers with and without a feed-forward of both kinds."""
    return R.config(96, 101, 2, [
        R.layer_delta(4, 2, 32, 48, taps=3, ff=72),
        R.layer_attention(6, 2, 48, 32, 32, taps=2),
        R.layer_attention(6, 2, 48, 32, 32, taps=3, kv_from=1, ff=88),
        R.layer_delta(3, 1, 20, 24, taps=4),
        R.layer_attention(4, 4, 32, 64, 16, taps=4, ff=40, scaling=LLAMA_SCALING)], eps=1e-3, scale=2.0)


def model_plain_residual():
    """One stream, more query heads per key head than an MMA tile has rows, width no multiple of 8, long and missing taps."""
    return R.config(132, 64, 1, [
        R.layer_attention(20, 1, 64, 64, 64, taps=5, ff=64, scaling=LLAMA_SCALING),
        R.layer_delta(2, 2, 64, 128, taps=1),
        R.layer_attention(20, 1, 64, 64, 64, taps=1, kv_from=0)], scale=1.5)


def model_wide_heads():
    """Heads of 128 in pages of 128 tokens: tensor-core prefill and captured mixed steps on the GPU."""
    return R.config(256, 200, 4, [
        R.layer_delta(2, 1, 128, 128, taps=4, ff=128),
        R.layer_attention(4, 2, 128, 128, 128, taps=4, ff=160, base=500000.0),
        R.layer_delta(2, 2, 64, 96, taps=2),
        R.layer_attention(4, 2, 128, 128, 128, taps=4, kv_from=1, ff=96, base=500000.0)])


def model_odd_heads():
    """Heads above 128 and sizes that are multiples of nothing much."""
    return R.config(120, 77, 3, [
        R.layer_delta(3, 3, 140, 36, taps=4, ff=50),
        R.layer_attention(3, 1, 160, 90, 100, taps=3, scale=0.2),
        R.layer_delta(5, 1, 12, 13, taps=2)])


MODELS = {"mixed": model_mixed, "plain_residual": model_plain_residual, "wide_heads": model_wide_heads, "odd_heads": model_odd_heads}
_oracle_cache: dict = {}


def weights_of(name):
    cfg = MODELS[name]()
    return cfg, R.random_weights(cfg, seed=len(name), decay=-3.0)      # slow decay: the state remembers hundreds of tokens


def tokens_of(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def expected(name, tokens):
    """Oracle logits of one sequence in float64, computed once per (model, tokens)."""
    key = (name, tuple(tokens))
    if key not in _oracle_cache:
        cfg, w = weights_of(name)
        _oracle_cache[key] = R.forward(cfg, R.as_double(w), tokens)
    return _oracle_cache[key]


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
    llm = open_llm(tmp_path, name, target, page_size=128 if name == "wide_heads" else 32)
    toks = tokens_of(cfg, 150, 4)
    for cuts in ([2] * 10 + [3] * 5 + [2, 27, 1, 31, 2, 50, 2], [31, 2, 30, 1, 1, 2, 33, 50]):
        assert sum(cuts) == 150
        check(run_schedule(llm.engine, {"a": toks}, [[("a", c)] for c in cuts])["a"], expected(name, toks), target)


@pytest.mark.parametrize("page", [16, 64, 128])
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["mixed", "wide_heads"])
def test_unequal_batches_with_reuse(tmp_path, target, name, page):
    """Four live requests in one batch, portions beside decoded tokens, some left out of steps; the pool and the state
    slots only fit the live ones, so later requests use pages and slots that others gave back."""
    cfg, _ = weights_of(name)
    lengths = {"a": 150, "b": 33, "c": 70, "d": 1, "e": 90, "f": 33}
    req = {k: tokens_of(cfg, n, {"a": 4, "b": 3}.get(k, ord(k))) for k, n in lengths.items()}
    llm = open_llm(tmp_path, name, target, page_size=page, num_pages=-(-150 // page) + -(-90 // page) + -(-70 // page) + -(-33 // page))
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
    assert llm.engine.kv.free_state_slots() == 4 and llm.engine.kv.available_pages() == llm.engine.kv.num_pages


@pytest.mark.parametrize("target", TARGETS)
def test_long_decoding(tmp_path, target):
    """Hundreds of decoded tokens: state and cache far beyond the prompt, several pages."""
    cfg, _ = weights_of("mixed")
    toks = tokens_of(cfg, 300, 9)
    llm = open_llm(tmp_path, "mixed", target)
    check(run_schedule(llm.engine, {"a": toks}, [[("a", 4)]] + [[("a", 1)]] * 296)["a"], expected("mixed", toks), target)


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
    """`LLM.generate` with more requests than state slots, a token budget that cuts prompts and a pool that runs out of
    pages (preemption and recomputation): the tokens of the plain implementation."""
    cfg, _ = weights_of("mixed")
    prompts = [tokens_of(cfg, n, 20 + i) for i, n in enumerate((30, 14, 30, 1, 20))]
    want = [greedy("mixed", p, 12) for p in prompts]
    llm = open_llm(tmp_path, "mixed", target, page_size=16, num_pages=5, max_num_seqs=3, max_num_batched_tokens=24, max_model_len=96)
    outs = llm.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    for o, (toks, margins) in zip(outs, want):
        # bf16: compare up to the first step whose two best logits are closer than rounding can tell apart
        n = 12 if target[1] == "float32" else next((i for i, m in enumerate(margins) if m < 0.1), 12)
        assert o.token_ids[:n] == toks[:n]
    assert llm.engine.scheduler.total_preemptions() > 0
    assert llm.engine.kv.check_invariants() == "" and llm.engine.kv.free_state_slots() == 3


@gpu
@pytest.mark.parametrize("async_scheduling", [False, True])
def test_captured_steps_give_the_eager_tokens(tmp_path, async_scheduling):
    """Decode and mixed steps replayed as CUDA graphs, step by step and pipelined, against eager launches."""
    from mojo_b200.engine import EngineConfig, LLMEngine

    cfg, _ = weights_of("wide_heads")
    prompts = [tokens_of(cfg, n, 40 + n) for n in (200, 7, 130, 64, 3, 90)]
    eager = open_llm(tmp_path, "wide_heads", ("cuda", "bfloat16"), page_size=128, use_cuda_graphs=False)
    sp = SamplingParams(max_tokens=24, ignore_eos=True)
    want = [o.token_ids for o in eager.generate(prompts, sp)]
    assert eager.engine.runner.graph_launches == 0
    ecfg = EngineConfig(model=eager.model_config, device="cuda", dtype=torch.bfloat16, page_size=128, num_pages=24, max_num_seqs=4,
                        max_num_batched_tokens=512, max_model_len=512, async_scheduling=async_scheduling)
    eng = LLMEngine(ecfg, model=eager.engine.model)
    assert eng.generate(prompts, sp) == want
    assert eng.runner.mixed_launches > 0 and eng.runner.graph_launches > eng.runner.mixed_launches and not eng.runner.failed_buckets


def test_command_line_generate_and_replay(tmp_path, capsys, monkeypatch):
    """Both command-line entries on a checkpoint folder, on the CPU engine."""
    import io

    from mojo_b200 import cli

    cfg, w = weights_of("mixed")
    R.write_checkpoint(tmp_path / "m", cfg, w)
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
    tol = f32 if target[1] == "float32" else bf16
    err = (got - want).abs().max() / want.abs().max().clamp_min(1e-6)
    assert err < tol, f"{err:.2e}"


def dev(t, target, dtype=None):
    return t.to(device=target[0], dtype=dtype or getattr(torch, target[1])).contiguous()


def seq_rows(lengths, banks, device, order=None):
    """SeqRows of sequences with these row counts; the first ones of one row are the decode rows. banks: [(read, write)]."""
    ends = np.cumsum(lengths)
    rows = np.stack([ends - lengths, ends], axis=1).astype(np.int32)
    n_dec = next((i for i, n in enumerate(lengths) if n != 1), len(lengths))
    return ops.SeqRows(torch.from_numpy(np.repeat(np.arange(len(lengths), dtype=np.int32), lengths)).to(device), torch.from_numpy(rows).to(device),
                       torch.tensor(banks, dtype=torch.int32, device=device), n_dec, n_dec, len(lengths) - n_dec)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("streams,width", [(1, 64), (2, 20), (3, 160), (4, 1000), (7, 96), (8, 2048)])
def test_hyper_connections(target, streams, width):
    g = torch.Generator().manual_seed(streams)

    def rnd(*s):
        return torch.randn(*s, generator=g, dtype=torch.float64).float().double()

    T = 5
    w = {"a.in": rnd(streams), "a.out": rnd(streams), "a.mix": rnd(streams, streams), "b.in": rnd(streams)}
    norm_w, x = rnd(width) * 0.3, rnd(streams, T, width)
    y = dev(rnd(T, width).float(), target)
    new = R.hyper_write(x, w, "a.", y.double().cpu())
    want = R.norm_zero_centred(R.hyper_read(new, w, "b."), norm_w, 1e-2)

    def mix(p):
        f = lambda n, *s: dev(w.get(p + n, torch.zeros(s)).float(), target, torch.float32)  # noqa: E731
        return ops.HyperMix(f("in"), f("out", streams), f("mix", streams, streams))

    xs = dev(x.transpose(0, 1).float(), target, torch.float32)
    kept = xs.clone()
    weight = dev(1 + norm_w.float(), target, torch.float32)
    dtype = getattr(torch, target[1])
    rows = torch.tensor([3, 0], device=target[0])
    h = ops.hyper_norm(xs, weight, 1e-2, dtype, mix("b."), mix("a."), y, rows=rows, store=False)
    close(h, want[[3, 0]], target)
    assert torch.equal(xs, kept)
    close(ops.hyper_norm(xs, weight, 1e-2, dtype, mix("b."), mix("a."), y), want, target)
    close(xs.transpose(0, 1), new, (target[0], "float32"))            # the streams stay f32 in both forms
    # first read: the embedding; last read: the plain sum
    embed, ids = dev(rnd(11, width).float(), target), torch.tensor([4, 0, 10, 4, 7], device=target[0])
    ops.hyper_norm(xs, weight, 1e-2, dtype, mix("b."), ids=ids, embed=embed, embed_scale=2.5)
    start = (embed.double().cpu()[ids.cpu()] * 2.5).expand(streams, T, width)
    close(xs.transpose(0, 1), start, (target[0], "float32"))
    close(ops.hyper_norm(xs, weight, 1e-2, dtype, None, store=False), R.norm_zero_centred(start.sum(0), norm_w, 1e-2), target)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,taps", [(6, 2, 32, 32, 32, 4), (3, 3, 48, 64, 16, 2), (4, 1, 130, 20, 64, 7), (2, 1, 5, 9, 4, 3), (2, 2, 64, 64, 0, 1)])
def test_convolution_rotation_and_head_norm(target, heads, kv, dim, vdim, rot, taps):
    """Three sequences (decode row, two portions) continued from their banks: queries, cache rows and new banks."""
    g = torch.Generator().manual_seed(dim)
    C, page, eps = heads * dim + kv * (dim + vdim), 8, 1e-3
    act = getattr(torch, target[1])
    past, now = [21, 1, 0], [1, 2, 13]       # rows already run, rows of this step (the second is shorter than most histories)
    full = [torch.randn(p + n, C, generator=g).to(act).double() for p, n in zip(past, now)]
    w = torch.randn(C, taps, generator=g).double()
    spec = {"dims": rot, "base": 100.0, "scaling": LLAMA_SCALING}
    table = torch.zeros(64, rot)
    if rot:
        ang = torch.arange(64, dtype=torch.float64)[:, None] * torch.tensor(R.rope_frequencies(spec), dtype=torch.float64)
        table = torch.cat([ang.cos(), ang.sin()], 1)
    pad = dim if target[1] == "float32" else next(p for p in (64, 128, 256) if p >= max(dim, vdim))
    pad_v = vdim if target[1] == "float32" else pad
    kc, vc = (dev(torch.zeros(8, kv, page, p), target) for p in (pad, pad_v))
    bank = torch.randn(6, max(taps - 1, 1), C, generator=g)       # stale contents everywhere
    for s, (f, p) in enumerate(zip(full, past)):
        if p:
            bank[2 * s, :taps - 1] = torch.cat([torch.zeros(taps, C).double(), f[:p]])[-(taps - 1):].float() if taps > 1 else 0
    bank = dev(bank, target) if taps > 1 else None
    seq = seq_rows(now, [(0, 1), (2, 3), (-1, 5)], target[0])
    proj = dev(torch.cat([torch.cat([f[p:] for f, p in zip(full, past)]), torch.randn(sum(now), 3, generator=g).double()], 1), target)
    if target[1] == "bfloat16" and proj.shape[1] % 2:
        proj = torch.nn.functional.pad(proj, (0, 1))
    positions = torch.tensor([p + i for p, n in zip(past, now) for i in range(n)], dtype=torch.int32, device=target[0])
    slots = torch.tensor([50 - 3 * i if i != 2 else -1 for i in range(sum(now))], device=target[0])
    q = ops.conv_qkv(proj, dev(w.T, target, torch.float32), bank, dev(table, target, torch.float32), positions, seq, slots, kc, vc, heads, kv, dim, vdim,
                     pad, eps).view(sum(now), heads, pad)
    row = 0
    for s, (f, p, n) in enumerate(zip(full, past, now)):
        u = R.causal_conv(f, w)

        def heads_of(z, k):
            z = z.view(p + n, k, dim)
            return R.rms(R.rotate(z, spec) if rot else z, eps)[p:]

        want_q, want_k = heads_of(u[:, :heads * dim].contiguous(), heads), heads_of(u[:, heads * dim:(heads + kv) * dim].contiguous(), kv)
        want_v = u[p:, (heads + kv) * dim:].reshape(n, kv, vdim)
        close(q[row:row + n, :, :dim], want_q, target)
        assert float(q[row:row + n, :, dim:].abs().sum()) == 0
        for i in range(n):
            slot = int(slots[row + i])
            if slot >= 0:
                close(kc[slot // page, :, slot % page, :dim], want_k[i], target)
                close(vc[slot // page, :, slot % page, :vdim], want_v[i], target)
        if taps > 1:
            last = torch.cat([torch.zeros(taps, C).double(), f])[-(taps - 1):]
            assert torch.equal(bank[2 * s + 1, :taps - 1].double().cpu(), last)
        row += n
    if target[0] == "cuda":
        ops.check_status()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,kv,dim,vdim,taps", [(4, 2, 32, 48, 4), (2, 2, 128, 128, 4), (3, 1, 20, 13, 2), (2, 1, 200, 256, 3), (1, 1, 8, 64, 1), (2, 2, 64, 20, 4)])
def test_gated_delta_rule(target, heads, kv, dim, vdim, taps):
    """Decode rows and portions continued from given matrices and banks; slow decay, so that the old state matters."""
    g = torch.Generator().manual_seed(dim + vdim)
    act = getattr(torch, target[1])
    past, now = [9, 40, 2, 0], [1, 1, 21, 37]
    H, ck = heads, kv * dim
    C, n_rows = 2 * ck + H * vdim, sum(now)
    b_off = C + 3
    full = [torch.randn(p + n, C + 3 + H, generator=g).to(act).double() for p, n in zip(past, now)]
    dgf = [torch.randn(p + n, H * (dim + vdim), generator=g).to(act).double() for p, n in zip(past, now)]
    w, a_log = torch.randn(C, taps, generator=g).double() * 0.7, torch.randn(H, generator=g).double() * 0.3
    bias, norm = torch.randn(H * dim, generator=g).double() - 4.0, 1 + torch.randn(vdim, generator=g).double() * 0.2
    m = {"heads": H, "kv_heads": kv, "dim": dim, "vdim": vdim}

    def oracle(f, dg):
        u = R.silu(R.causal_conv(f[:, :C], w))
        T = f.shape[0]
        q, k = (R.unit(u[:, o:o + ck].reshape(T, kv, dim)).repeat_interleave(H // kv, 1) for o in (0, ck))
        dec = torch.exp(-torch.exp(a_log)[None, :, None] * R.softplus(dg[:, :H * dim] + bias).view(T, H, dim))
        args = (q * dim ** -0.5, k, u[:, 2 * ck:].reshape(T, H, vdim), dec, R.sigmoid(f[:, b_off:b_off + H]))
        gate = R.sigmoid(dg[:, H * dim:]).view(T, H, vdim)
        return args, gate

    state, bank = torch.randn(5, H, dim, vdim, generator=g), torch.randn(10, max(taps - 1, 1), C, generator=g)
    want_o, want_s = [], []
    slots = [3, 0, 4, 1]
    for f, dg, p, slot in zip(full, dgf, past, slots):
        args, gate = oracle(f, dg)
        _, s0 = R.delta_rule(*(a[:p] for a in args))
        o, s1 = R.delta_rule(*(a[p:] for a in args), s0=s0)
        want_o.append((R.rms(o, 1e-4) * norm * gate[p:]).reshape(-1, H * vdim))
        want_s.append(s1)
        if p:
            state[slot] = s0.float()
            if taps > 1:
                bank[2 * slot + 1, :taps - 1] = torch.cat([torch.zeros(taps, C).double(), f[:p, :C]])[-(taps - 1):].float()
    state = dev(state, target, torch.float32)
    bank = dev(bank, target) if taps > 1 else None
    seq = seq_rows(now, [(2 * s + 1 if p else -1, 2 * s) for s, p in zip(slots, past)], target[0])
    proj = dev(torch.cat([f[p:] for f, p in zip(full, past)]), target)
    dg = dev(torch.cat([d[p:] for d, p in zip(dgf, past)]), target)
    f32 = lambda t: dev(t, target, torch.float32)  # noqa: E731
    params = ops.DeltaParams(f32(w.T), f32(-torch.exp(a_log)), f32(bias), f32(norm))
    cols = H * vdim + 5
    out = ops.delta_rule(proj, dg[:, :H * dim], dg[:, H * dim:H * (dim + vdim)], params, bank, state, seq, b_off, H, kv, dim, vdim, cols, 1e-4)
    if target[0] == "cuda":
        ops.check_status()
    close(out[:, :H * vdim], torch.cat(want_o), target)
    assert float(out[:, H * vdim:].abs().sum()) == 0 and out.shape == (n_rows, cols)
    for slot, s1, f in zip(slots, want_s, full):
        close(state[slot], s1, (target[0], "float32"))        # f32 in both forms
        if taps > 1:
            assert torch.equal(bank[2 * slot, :taps - 1].double().cpu(), torch.cat([torch.zeros(taps, C).double(), f[:, :C]])[-(taps - 1):])


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("page", [16, 64, 128])
@pytest.mark.parametrize("n_q,n_kv,dim,vdim", [(4, 2, 64, 64), (20, 1, 64, 64), (2, 1, 128, 128), (3, 1, 256, 256)])
def test_gated_attention_finds_one_key(target, page, n_q, n_kv, dim, vdim):
    """One key matches the last query far better than all others: wherever it lies (first token, page borders, far back,
    the query's own place), decode rows and portions return its value through the head gate."""
    g = torch.Generator().manual_seed(page + n_q)
    ctx = 300
    spots = [0, 1, page - 1, page, page + 1, 2 * page - 1, 127, 128, 255, ctx - 2, ctx - 1]
    spots = sorted({s for s in spots if s < ctx})
    act = getattr(torch, target[1])
    pages = -(-ctx // page)
    q_len = [1] * len(spots) + [5] * len(spots)
    B = len(q_len)
    K, V = torch.randn(B, ctx, n_kv, dim, generator=g) * 0.3, torch.randn(B, ctx, n_kv, vdim, generator=g)
    q = torch.randn(sum(q_len), n_q, dim, generator=g)
    ends = np.cumsum(q_len)
    for b in range(B):
        spot = spots[b % len(spots)]
        row = q[ends[b] - 1].view(n_kv, n_q // n_kv, dim)
        row[:] = row[:, :1]                                    # the heads of a group ask for the same key
        K[b, spot] = row[:, 0] * (12.0 / row[:, 0].norm(dim=-1, keepdim=True) ** 2) * dim ** 0.5
    K, V, q = K.to(act), V.to(act), q.to(act)
    table = torch.randperm(B * pages, generator=g).view(B, pages).int()
    kc, vc = torch.zeros(B * pages, n_kv, page, dim, dtype=act), torch.zeros(B * pages, n_kv, page, vdim, dtype=act)
    for b in range(B):
        for t in range(ctx):
            p = int(table[b, t // page])
            kc[p, :, t % page], vc[p, :, t % page] = K[b, t], V[b, t]
    gate = torch.randn(sum(q_len), n_q + 2, generator=g).to(act)
    cu = np.concatenate([[0], ends]).astype(np.int32)
    seq = seq_rows(np.array(q_len), [(0, 1)] * B, target[0])
    pos = torch.tensor([ctx - n + i for n in q_len for i in range(n)], dtype=torch.int32, device=target[0])
    meta = ops.AttnMeta(torch.from_numpy(cu).to(target[0]), torch.full((B,), ctx, dtype=torch.int32, device=target[0]), table.to(target[0]),
                        len(spots), 5, ctx, seq=seq)
    out = ops.paged_attention(dev(q.view(sum(q_len), -1), target), dev(kc, target), dev(vc, target), meta, dim ** -0.5, dim,
                              gate=dev(gate, target)[:, 1:1 + n_q], positions=pos)
    if target[0] == "cuda":
        ops.check_status()
    out = out.view(sum(q_len), n_q, vdim)
    for b in range(B):
        rows = slice(ends[b] - q_len[b], ends[b])
        past = torch.zeros(ctx - q_len[b], n_q, dim, dtype=torch.float64)
        o = R.attend(torch.cat([past, q[rows].double()]), K[b].double(), V[b].double(), dim ** -0.5)[-q_len[b]:]
        o = o * R.sigmoid(gate[rows, 1:1 + n_q].double())[:, :, None]
        close(out[rows], o, target)
        # the planted key carries nearly all of the last row's weight
        spot = V[b, spots[b % len(spots)]].double().repeat_interleave(n_q // n_kv, 0) * R.sigmoid(gate[ends[b] - 1, 1:1 + n_q].double())[:, None]
        assert (o[-1] - spot).abs().max() < 0.05 * spot.abs().max()


def test_config_reading_and_refusals(tmp_path):
    from mojo_b200.models import build_model, get_config

    cfg, w = weights_of("mixed")
    R.write_checkpoint(tmp_path / "m", cfg, w)
    mc = get_config(str(tmp_path / "m"))
    assert (mc.architecture, mc.num_layers, mc.hidden_size, mc.residual_streams, mc.vocab_size) == ("rekudra", 5, 96, 2, 101)
    assert mc.layers[2].kv_from == 1 and mc.layers[1].ffn == 0 and mc.layers[0].ffn == 72 and mc.layers[4].rot.scaling == LLAMA_SCALING
    model = build_model(mc)
    # pages: the two layers that own keys and values; state: f32 matrices and two banks per convolution
    assert model.kv_bytes_per_page(16) == (2 * (48 + 32) + 4 * (32 + 64)) * 16 * 4
    caches = model.allocate_kv_cache(3, 16, 2)
    assert caches[2].k is caches[1].k and caches[0].state.shape == (2, 4, 32, 48) and caches[0].conv.shape == (4, 2, 2 * 64 + 192)
    assert sum(t.numel() * 4 for c in caches for t in (c.conv, c.state) if t is not None) == 2 * model.state_bytes_per_slot()
    with pytest.raises(ValueError, match="prefix caching"):
        open_llm(tmp_path, "mixed", ("cpu", "float32"), enable_prefix_cache=True)
    for change, match in (({"kv_from": 0}, "kv_from"), ({"kv_from": 4}, "kv_from"), ({"dim": 40}, "head sizes")):
        bad = json.loads(json.dumps(cfg))
        bad["layers"][2]["mixer"].update(change)
        (tmp_path / "m" / "config.json").write_text(json.dumps(bad))
        with pytest.raises(ValueError, match=match):
            get_config(str(tmp_path / "m"))
    w["l0.mix.a2"] = w["l0.mix.a2"][:-1]
    R.write_checkpoint(tmp_path / "bad", cfg, w)
    with pytest.raises(ValueError, match="mix.a2"):
        LLM(PipelineConfig(model=str(tmp_path / "bad"), device="cpu"))


def test_planned_steps_are_checked_before_anything_changes(tmp_path):
    cfg, _ = weights_of("mixed")
    eng = open_llm(tmp_path, "mixed", ("cpu", "float32"), page_size=16, num_pages=4, max_num_seqs=2, max_num_batched_tokens=64, max_model_len=64).engine
    toks = tokens_of(cfg, 64, 1)
    eng.run_tokens([(0, toks[:20], [])])
    free = eng.kv.available_pages()
    for entries, match in (([(1, toks[:40], [])], "pages"), ([(1, toks[:2], []), (2, toks[:2], [])], "max_num_seqs"), ([(1, [], [])], "without tokens"),
                           ([(0, toks[:2], []), (0, toks[:2], [])], "twice"), ([(0, toks[:50], [])], "max_model_len"), ([(1, [cfg["vocab"]], [])], "vocabulary"),
                           ([(1, toks[:2], [2])], "wanted")):
        with pytest.raises((ValueError, RuntimeError), match=match):
            eng.run_tokens(entries)
    assert eng.kv.available_pages() == free and eng.kv.free_state_slots() == 1 and eng.kv.check_invariants() == ""
    check(eng.run_tokens([(0, toks[20:22], [0, 1])], [0]), expected("mixed", toks[:22])[20:], ("cpu", "float32"))
    assert eng.kv.available_pages() == 4 and eng.kv.free_state_slots() == 2
