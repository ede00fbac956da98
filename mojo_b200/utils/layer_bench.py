"""Rekudra beside Llama at equal layer sizes: prefill and decode throughput of a few layers through the serving engine, and
each design's own kernels against their rooflines. Random weights, synthetic prompts, one GPU (`bench.py --layer-bench`).

Steps are timed with CUDA events around the engine's device work, medians over repeats after warm-up; every step streams
weights and caches larger than L2. Single kernels are timed with an L2 flush before each launch. Rooflines use the copy
bandwidth and the bf16 rate measured on the machine; the scan of the delta rule works on f32 matrices, so its compute
bound is the f32 FMA rate (SMs x 128 lanes x maximum clock)."""
from __future__ import annotations

import json
import statistics
from pathlib import Path

import torch

SIZES = {"2048x16": dict(width=2048, heads=16, kv=4, dim=128, ffn=8192), "4096x32": dict(width=4096, heads=32, kv=8, dim=128, ffn=14336)}
VOCAB, LAYERS = 32000, 8
PREFILL = [(1, 2048), (2, 2048), (8, 512)]        # (prompts, tokens each), one step
DECODE = [(16, 1024), (128, 1024)]                # (sequences, context)


def peaks() -> dict:
    p = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    m = json.loads(p.read_text()) if p.exists() else {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "sm_max_mhz": 1965.0}
    return {"hbm": m["hbm_gbs"] * 1e9, "bf16": m["bf16_tflops"] * 1e12, "fma": 148 * 128 * m.get("sm_max_mhz", 1965.0) * 1e6,
            "source": "measured" if p.exists() else "fallback"}


def model_config(design: str, size: dict):
    from ..models.config import ModelConfig, rekudra

    if design == "rekudra":
        return rekudra(size["width"], LAYERS, size["heads"], size["kv"], size["dim"], size["ffn"], VOCAB)
    return ModelConfig(hidden_size=size["width"], num_layers=LAYERS, num_heads=size["heads"], num_kv_heads=size["kv"], head_dim=size["dim"],
                       intermediate_size=size["ffn"], vocab_size=VOCAB, max_position_embeddings=4096)


class Bench:
    def __init__(self, design: str, size: dict, autotune: bool):
        from ..engine import EngineConfig, LLMEngine

        n_seqs = max(b for b, _ in DECODE)
        cfg = EngineConfig(model=model_config(design, size), device="cuda:0", dtype=torch.bfloat16, page_size=128, num_pages=n_seqs * 12,
                           max_num_seqs=n_seqs, max_num_batched_tokens=4096, max_model_len=2304, autotune=autotune)
        self.engine, self.cfg = LLMEngine(cfg), cfg
        self.gen = torch.Generator().manual_seed(0)

    def prompt(self, n: int) -> list[int]:
        return torch.randint(0, VOCAB, (n,), generator=self.gen).tolist()

    def step_ms(self) -> float:
        s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        self.engine.runner.step_events = (s, e)
        self.engine.step()
        e.synchronize()
        self.engine.runner.step_events = None
        return s.elapsed_time(e)

    def drain(self) -> None:
        self.engine.abort_all()

    def prefill(self, prompts: int, tokens: int, warmup: int = 3, repeats: int = 9) -> dict:
        from ..engine import SamplingParams

        times = []
        for i in range(warmup + repeats):
            for _ in range(prompts):
                self.engine.add_request(self.prompt(tokens), SamplingParams(max_tokens=4, ignore_eos=True))
            t = self.step_ms()
            assert self.engine.runner.last_num_tokens == prompts * tokens
            self.drain()
            if i >= warmup:
                times.append(t)
        ms = statistics.median(times)
        return {"prompts": prompts, "tokens": tokens, "ms": round(ms, 3), "tok_per_s": round(prompts * tokens / ms * 1e3)}

    def decode(self, seqs: int, ctx: int, warmup: int = 4, repeats: int = 24) -> dict:
        from ..engine import SamplingParams

        for _ in range(seqs):
            self.engine.add_request(self.prompt(ctx), SamplingParams(max_tokens=warmup + repeats + 64, ignore_eos=True))
        while self.engine.scheduler.num_waiting() or self.engine.runner.last_num_tokens != seqs:
            self.engine.step()
        times = [self.step_ms() for _ in range(warmup + repeats)][warmup:]
        assert self.engine.runner.last_num_tokens == seqs
        self.drain()
        ms = statistics.median(times)
        return {"sequences": seqs, "context": ctx, "ms": round(ms, 3), "tok_per_s": round(seqs / ms * 1e3)}


# ------------------------------------------------------------------------------------------------------
# single kernels
# ------------------------------------------------------------------------------------------------------


def time_kernel(fn, flush: torch.Tensor, warmup: int = 3, repeats: int = 15) -> float:
    """Median microseconds of `fn`, L2 flushed before every launch."""
    out = []
    for i in range(warmup + repeats):
        flush.zero_()
        s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        s.record()
        fn()
        e.record()
        e.synchronize()
        if i >= warmup:
            out.append(s.elapsed_time(e) * 1e3)
    return statistics.median(out)


def step_rows(n_dec: int, chunks: list[int]):
    """SeqRows of `n_dec` decode rows followed by prompt chunks."""
    import numpy as np

    from .. import ops

    lens = np.array([1] * n_dec + chunks)
    ends = np.cumsum(lens)
    rows = np.stack([ends - lens, ends], axis=1).astype(np.int32)
    banks = np.stack([2 * np.arange(len(lens)) if n_dec else np.full(len(lens), -1), 2 * np.arange(len(lens)) + 1], axis=1).astype(np.int32)
    put = lambda a: torch.from_numpy(np.ascontiguousarray(a)).cuda()  # noqa: E731
    return ops.SeqRows(put(np.repeat(np.arange(len(lens), dtype=np.int32), lens)), put(rows), put(banks), n_dec, n_dec, len(chunks))


def kernel_table(size: dict) -> list[dict]:
    from .. import ops
    from ..ops import reference

    pk = peaks()
    W, H, G, d = size["width"], size["heads"], size["kv"], size["dim"]
    S, taps, page = 4, 4, 128
    dev, bf = torch.device("cuda"), torch.bfloat16
    flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    rows = []

    def add(name, design, case, fn, nbytes, fma=0.0, mma=0.0):
        us = time_kernel(fn, flush)
        floor = max(nbytes / pk["hbm"], fma / pk["fma"], 2 * mma / pk["bf16"]) * 1e6
        bound = "hbm" if floor == nbytes / pk["hbm"] * 1e6 else "fma" if fma and floor == fma / pk["fma"] * 1e6 else "bf16"
        rows.append({"kernel": name, "design": design, "case": case, "us": round(us, 2), "roofline_us": round(floor, 2), "bound": bound,
                     "fraction": round(floor / us, 3)})

    def rnd(*s, dtype=bf, std=1.0):
        return (torch.randn(*s, device=dev) * std).to(dtype)

    table = reference.rope_table(4096, d, 1e4).to(dev)
    for case, seq, ctx, n_seq, T in (("decode 128 x 1024", step_rows(128, []), 1024, 128, 128), ("prefill 2 x 2048", step_rows(0, [2048, 2048]), 2048, 2, 4096)):
        dec = seq.n_decode > 0
        # --- residual and norm
        f = [rnd(n, dtype=torch.float32, std=0.3) for n in (S, S, S * S)]
        hm = ops.HyperMix(f[0], f[1], f[2].view(S, S))
        x, y = rnd(T, S, W, dtype=torch.float32), rnd(T, W)
        w32, w16, res = torch.ones(W, device=dev), torch.ones(W, device=dev, dtype=bf), rnd(T, W)
        add("hyper_norm", "rekudra", case, lambda: ops.hyper_norm(x, w32, 1e-5, bf, hm, hm, y), T * W * (8 * S + 4))
        add("rmsnorm + residual", "llama", case, lambda: ops.rms_norm(y, w16, 1e-5, res), T * W * 8)
        # --- attention front end
        n_pages = n_seq * (ctx // page + 1)
        kc, vc = (torch.zeros(n_pages, G, page, d, device=dev, dtype=bf) for _ in range(2))
        per = ctx // page + 1
        pos = torch.full((T,), ctx, dtype=torch.int32, device=dev) if dec else torch.arange(ctx, dtype=torch.int32, device=dev).repeat(n_seq)
        base = torch.arange(n_seq, device=dev) * per * page
        slots = base + ctx if dec else (base[:, None] + torch.arange(ctx, device=dev)[None]).flatten()
        C = (H + 2 * G) * d
        proj = rnd(T, C + H)
        cw, bank = rnd(taps, C, dtype=torch.float32, std=0.3), rnd(2 * n_seq, taps - 1, C)
        hist = n_seq * (taps - 1) * C * 2 * (2 if dec else 1)
        add("conv_qkv", "rekudra", case, lambda: ops.conv_qkv(proj, cw, bank, table, pos, seq, slots, kc, vc, H, G, d, d, d, 1e-5), T * C * 4 + hist)
        q, k, v = proj[:, :H * d], proj[:, H * d:(H + G) * d], proj[:, (H + G) * d:C]
        add("rope_kvwrite", "llama", case, lambda: ops.rope_kvwrite(q, k, v, table, pos, slots, kc, vc, d), T * (C + (H + G) * d + G * d) * 2)
        # --- attention
        bt = (torch.arange(n_seq, dtype=torch.int32, device=dev)[:, None] * per + torch.arange(per, dtype=torch.int32, device=dev)[None]).contiguous()
        cl = torch.full((n_seq,), ctx, dtype=torch.int32, device=dev)
        cu = torch.arange(n_seq + 1, dtype=torch.int32, device=dev) * (T // n_seq)
        work = None
        if not dec:
            w_np = ops.prefill_work_items(cu.cpu().numpy(), cl.cpu().numpy(), 0)
            work = torch.from_numpy(w_np).cuda()
        meta = ops.AttnMeta(cu, cl, bt, n_seq if dec else 0, T // n_seq, ctx, work=work, n_items=0 if work is None else work.shape[0])
        qq, gate = rnd(T, H * d), proj[:, C:]
        kv_bytes, pairs = n_seq * ctx * G * d * 4, n_seq * ctx * (ctx + 1) / 2
        fl = 0.0 if dec else pairs * H * d * 2
        add("attention, gated", "rekudra", case, lambda: ops.paged_attention(qq, kc, vc, meta, d ** -0.5, d, gate=gate), kv_bytes + T * H * d * 4, mma=fl)
        add("attention", "llama", case, lambda: ops.paged_attention(qq, kc, vc, meta, d ** -0.5, d), kv_bytes + T * H * d * 4, mma=fl)
        # --- delta rule
        Cd = 2 * H * d + H * d
        pd, dg = rnd(T, Cd + H), rnd(T, 2 * H * d)
        dp = ops.DeltaParams(rnd(taps, Cd, dtype=torch.float32, std=0.3), -torch.ones(H, device=dev), torch.full((H * d,), -3.0, device=dev), torch.ones(d, device=dev))
        st, bd = torch.zeros(n_seq, H, d, d, device=dev), rnd(2 * n_seq, taps - 1, Cd)
        state_bytes = n_seq * H * d * d * 4 * (2 if dec else 1)
        io = T * (Cd + H + 3 * H * d) * 2
        hist = n_seq * (taps - 1) * Cd * 2 * (2 if dec else 1)
        add("delta_decode" if dec else "delta_scan + out", "rekudra", case,
            lambda: ops.delta_rule(pd, dg, dp, bd, st, seq, Cd, H, H, d, d, H * d, 1e-5), state_bytes + io + hist, fma=4.0 * T * H * d * d)
    return rows


def run(args) -> dict:
    from .clocks import ClockSampler

    out = {"metric": "layer throughput, Rekudra beside Llama at equal layer sizes", "unit": "tok/s", "n_gpus": 1, "dtype": "bf16", "layers": LAYERS,
           "data": "synthetic: uniform-random token ids, random weights", "peaks": peaks(), "sizes": {}}
    with ClockSampler(0) as clocks:
        for name, size in SIZES.items():
            rec = {"kernels": kernel_table(size)}
            for design in ("llama", "rekudra"):
                b = Bench(design, size, autotune=not args.no_autotune)
                rec[design] = {"weight_bytes": b.engine.model.weight_bytes(), "prefill": [b.prefill(*c) for c in PREFILL], "decode": [b.decode(*c) for c in DECODE]}
                del b
                torch.cuda.empty_cache()
            out["sizes"][name] = rec
    summary = clocks.summary()
    out["clocks"] = {k: summary.get(k) for k in ("sm_mhz", "sm_max_mhz", "reasons", "power_w_max")}
    from .. import ops

    ops.check_status()
    return out
