"""A design beside the closest one at equal layer sizes: prefill and decode throughput of a few layers through the serving
engine, and each design's own kernels against their rooflines. Random weights, synthetic prompts, one GPU
(`bench.py --layer-bench`: Rekudra beside Llama; `bench.py --layer-bench rerupel`: Rerupel beside DeepSeek-V2;
`bench.py --layer-bench pilutar`: Pilutar beside Rerupel, its single kernels also beside the like ones of Llama and Rekudra;
`bench.py --layer-bench noridra`: Noridra beside Pilutar, its single kernels also beside those of Rekudra).

Steps are timed with CUDA events around the engine's device work, medians over repeats after warm-up; every step streams
weights and caches larger than L2. Single kernels are timed with an L2 flush before each launch. Rooflines use the copy
bandwidth and the bf16 rate measured on the machine; the scans of recurrent layers work on f32 matrices, so their compute
bound is the f32 FMA rate (SMs x 128 lanes x maximum clock), or for exponentials that of the special-function units (16 lanes)."""
from __future__ import annotations

import json
import statistics
from pathlib import Path

import torch

DESIGNS = {"rekudra": ("llama", "rekudra"), "rerupel": ("deepseek", "rerupel"), "pilutar": ("rerupel_plain", "pilutar"),
           "noridra": ("pilutar_short", "noridra")}      # (closest model, design)
SIZES = {"2048x16": dict(width=2048, heads=16, kv=4, dim=128, ffn=8192), "4096x32": dict(width=4096, heads=32, kv=8, dim=128, ffn=14336)}
# DeepSeek-V2-Lite's layers, and the same at twice the width; latents of 512 columns, 64 experts of which 6 are used
MOE_SIZES = {"2048x16": dict(width=2048, heads=16, dim=128, rank=512, rope=64, ffn=10944, experts=64, top=6, expert_ffn=1408),
             "4096x32": dict(width=4096, heads=32, dim=128, rank=512, rope=64, ffn=14336, experts=64, top=6, expert_ffn=1408)}
PILUTAR_SIZES = {k: dict(v, kv=4 * (i + 1), rope=32, window=1024, groups=8, keep=4, identity=2) for i, (k, v) in enumerate(MOE_SIZES.items())}
NORIDRA_SIZES = {k: dict(v, chunk=1024, state=16, norm_groups=4) for k, v in PILUTAR_SIZES.items()}
VOCAB, LAYERS = 32000, 8
MOE_RUNS = 9           # one dense layer and eight with experts (the design: four, passed twice)
PREFILL = [(1, 2048), (2, 2048), (8, 512)]        # (prompts, tokens each), one step
DECODE = [(16, 1024), (128, 1024)]                # (sequences, context)


def peaks() -> dict:
    p = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    m = json.loads(p.read_text()) if p.exists() else {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "sm_max_mhz": 1965.0}
    return {"hbm": m["hbm_gbs"] * 1e9, "bf16": m["bf16_tflops"] * 1e12, "fma": 148 * 128 * m.get("sm_max_mhz", 1965.0) * 1e6,
            "sfu": 148 * 16 * m.get("sm_max_mhz", 1965.0) * 1e6,
            "source": "measured" if p.exists() else "fallback"}


def model_config(design: str, size: dict):
    from ..models.config import ModelConfig, noridra, pilutar, rekudra, rerupel

    if design == "noridra":
        return noridra(size["width"], LAYERS, size["heads"], size["kv"], size["dim"], VOCAB, size["experts"], size["top"], size["expert_ffn"], size["chunk"],
                       size["state"], size["norm_groups"], positions=4096)
    if design in ("pilutar", "pilutar_short"):
        return pilutar(size["width"], LAYERS if design == "pilutar_short" else MOE_RUNS, size["heads"], size["kv"], size["dim"], size["rank"], size["rope"], size["ffn"], VOCAB,
                       size["experts"] - size["identity"], size["top"], size["expert_ffn"], 2 * size["expert_ffn"], size["window"], size["groups"], size["keep"],
                       size["identity"])
    if design == "rerupel_plain":      # every layer run with weights of its own
        return rerupel(size["width"], MOE_RUNS, size["heads"], size["dim"], size["rank"], size["ffn"], VOCAB, size["experts"], size["top"], size["expert_ffn"],
                       2 * size["expert_ffn"])
    if design == "rerupel":
        return rerupel(size["width"], 5, size["heads"], size["dim"], size["rank"], size["ffn"], VOCAB, size["experts"], size["top"], size["expert_ffn"],
                       2 * size["expert_ffn"], (1, 5, 2))
    if design == "deepseek":
        return ModelConfig(architecture="deepseek_v2", hidden_size=size["width"], num_layers=MOE_RUNS, num_heads=size["heads"], num_kv_heads=size["heads"],
                           head_dim=size["dim"] + size["rope"], intermediate_size=size["ffn"], vocab_size=VOCAB, rms_norm_eps=1e-6, rope_theta=10000.0,
                           max_position_embeddings=4096, kv_lora_rank=size["rank"], qk_rope_head_dim=size["rope"], qk_nope_head_dim=size["dim"],
                           v_head_dim=size["dim"], n_routed_experts=size["experts"], n_shared_experts=2, num_experts_per_tok=size["top"],
                           moe_intermediate_size=size["expert_ffn"], first_k_dense_replace=1, rope_interleaved=True)
    if design == "rekudra":
        return rekudra(size["width"], LAYERS, size["heads"], size["kv"], size["dim"], size["ffn"], VOCAB)
    return ModelConfig(hidden_size=size["width"], num_layers=LAYERS, num_heads=size["heads"], num_kv_heads=size["kv"], head_dim=size["dim"],
                       intermediate_size=size["ffn"], vocab_size=VOCAB, max_position_embeddings=4096)


def local_experts(size: dict, max_tokens: int):
    from ..parallel.dist import DistInfo
    from ..parallel.ep import EPComm

    return EPComm(DistInfo(0, 1, 0, torch.device("cuda:0"), None, None), size["experts"], size["width"], size["expert_ffn"], size["top"], max_tokens=max_tokens,
                  timeout_s=5.0)


class Bench:
    def __init__(self, design: str, size: dict, autotune: bool):
        from ..engine import EngineConfig, LLMEngine

        n_seqs = max(b for b, _ in DECODE)
        cfg = EngineConfig(model=model_config(design, size), device="cuda:0", dtype=torch.bfloat16, page_size=128, num_pages=n_seqs * 12,
                           max_num_seqs=n_seqs, max_num_batched_tokens=4096, max_model_len=2304, autotune=autotune)
        model = None
        if design == "deepseek":      # its experts run through the expert-parallel kernels, here with a world of one
            from ..models.deepseek_v2 import DeepseekV2Model

            model = DeepseekV2Model(cfg.model, "cuda:0", cfg.dtype, ep=local_experts(size, cfg.max_num_batched_tokens)).init_random(0)
        self.engine, self.cfg = LLMEngine(cfg, model=model), cfg
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


class KernelTable:
    """Rows of timed kernels: `add` times a call with a cold L2 and sets it against its roofline (bytes moved, f32
    multiply-adds, bf16 multiply-adds)."""

    def __init__(self):
        self.pk, self.rows = peaks(), []
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def add(self, name, design, case, fn, nbytes, fma=0.0, mma=0.0, sfu=0.0):
        pk = self.pk
        us = time_kernel(fn, self.flush)
        bound, floor = max((("hbm", nbytes / pk["hbm"]), ("fma", fma / pk["fma"]), ("bf16", 2 * mma / pk["bf16"]), ("sfu", sfu / pk["sfu"])), key=lambda b: b[1])
        floor *= 1e6
        self.rows.append({"kernel": name, "design": design, "case": case, "us": round(us, 2), "roofline_us": round(floor, 2), "bound": bound,
                          "fraction": round(floor / us, 3)})


def rnd(*s, dtype=torch.bfloat16, std=1.0):
    return (torch.randn(*s, device="cuda") * std).to(dtype)


def kernel_table(size: dict) -> list[dict]:
    from .. import ops
    from ..ops import reference

    W, H, G, d = size["width"], size["heads"], size["kv"], size["dim"]
    S, taps, page = 4, 4, 128
    dev, bf = torch.device("cuda"), torch.bfloat16
    tab = KernelTable()
    add = tab.add
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
            lambda: ops.delta_rule(pd, dg[:, :H * d], dg[:, H * d:2 * H * d], dp, bd, st, seq, Cd, H, H, d, d, H * d, 1e-5), state_bytes + io + hist, fma=4.0 * T * H * d * d)
    return tab.rows


def latent_kernel_table(size: dict) -> list[dict]:
    """Rerupel's kernels beside those of DeepSeek-V2."""
    from .. import ops

    W, H, d, R, E, k, F = size["width"], size["heads"], size["dim"], size["rank"], size["experts"], size["top"], size["expert_ffn"]
    P, page, dev, bf = size["rope"], 128, torch.device("cuda"), torch.bfloat16
    tab = KernelTable()
    add, st, C = tab.add, ops._state.get(torch.device("cuda", 0)), ops._ext.require()
    ep = local_experts(size, 4096)
    gu, down = rnd(E, 2 * F, W, std=W ** -0.5), rnd(E, W, F, std=F ** -0.5)
    router = rnd(E, W, std=W ** -0.5)
    w_qk, w_kv = rnd(H * R, d, std=d ** -0.5), rnd(2 * H * d, R, std=R ** -0.5)
    ones, w32 = torch.ones(W, device=dev, dtype=bf), torch.ones(W, device=dev)
    for case, n_seq, ctx, T in (("decode 128 x 1024", 128, 1024, 128), ("prefill 2 x 2048", 2, 2048, 4096)):
        dec = n_seq == T
        per = ctx // page + 1
        # --- residual and norm
        x, y, res = rnd(T, W, dtype=torch.float32), rnd(T, W), rnd(T, W)
        add("residual_norm", "rerupel", case, lambda: ops.residual_norm(x, w32, 1e-6, bf, ops.Finished(w32, y)), T * W * 12)
        add("rmsnorm + residual", "deepseek", case, lambda: ops.rms_norm(y, ones, 1e-6, res), T * W * 8)
        # --- attention
        cache, mla_cache = rnd(n_seq * per, page, R), rnd(n_seq * per, page, R + P)
        bt = torch.arange(n_seq * per, dtype=torch.int32, device=dev).view(n_seq, per)
        cl = torch.full((n_seq,), ctx, dtype=torch.int32, device=dev)
        cu = torch.arange(n_seq + 1, dtype=torch.int32, device=dev) * (T // n_seq)
        base = torch.arange(n_seq, device=dev) * per * page
        slots = base + ctx - 1 if dec else (base[:, None] + torch.arange(ctx, device=dev)[None]).flatten()
        pos = torch.full((T,), ctx - 1, dtype=torch.int32, device=dev) if dec else torch.arange(ctx, dtype=torch.int32, device=dev).repeat(n_seq)
        meta = ops.AttnMeta(cu, cl, bt, n_seq if dec else 0, T // n_seq, ctx)
        proj = rnd(T, 2 * H * d + R)
        norm = torch.ones(R, device=dev)
        c16 = rnd(T, R)
        add("latent_write", "rerupel", case, lambda: ops.latent_write(proj[:, H * d:H * d + R], norm, 1e-6, slots, cache), T * R * 4)

        def mla_write():
            c, _ = ops.rms_norm(c16, ones[:R], 1e-6)
            ops.scatter_rows(c, slots, cache.view(-1, R))

        add("rmsnorm, scatter", "deepseek", case, mla_write, T * R * 4)
        rows = ops.token_rows(meta, T, dev)
        q_lat, q_rope, gate = rnd(T, H * R), rnd(T, H, P), proj[:, H * d + R:]
        pairs = float(n_seq * ctx) if dec else n_seq * ctx * (ctx + 1) / 2
        if dec:
            add("latent_attend", "rerupel", case, lambda: ops.latent_attend(q_lat, cache, meta, rows, H, 0.1, pos), n_seq * ctx * R * 2 + T * H * R * 4,
                mma=pairs * H * 2 * R)
            add("mla_attend", "deepseek", case, lambda: ops.mla_attend(q_lat.view(T, H, R), q_rope, mla_cache, meta, 0.1),
                n_seq * ctx * (R + P) * 2 + T * H * (2 * R + P) * 2, mma=pairs * H * (2 * R + P))
        else:
            plan = ops.plan_latent_prefill(cu.cpu().numpy(), cl.cpu().numpy(), 0, R, H, d, d)
            meta.expand = tuple(torch.from_numpy(a).cuda() for a in plan)
            work = torch.from_numpy(ops.prefill_work_items(cu.cpu().numpy(), cl.cpu().numpy(), 0)).cuda()
            meta.work, meta.n_items = work, work.shape[0]
            out = torch.empty(T, H * d, device=dev, dtype=bf)
            expand = float(len(plan[0]) * 128) * R * 2 * H * d      # multiply-adds of the expansion
            add("latent_prefill (gather, expand, attend)", "rerupel", case,
                lambda: ops.latent_prefill(proj[:, :H * d], cache, w_kv, meta, H, 0.1, gate, out), T * H * d * 8, mma=pairs * H * 2 * d + expand)
            add("mla_attend", "deepseek", case, lambda: ops.mla_attend(q_lat.view(T, H, R), q_rope, mla_cache, meta, 0.1), T * H * (2 * R + P) * 2,
                mma=pairs * H * (2 * d + P) + expand)
        # --- per-head maps beside a plain product of the same operations
        q = proj[:, :H * d]
        add("head_gemm (queries)", "rerupel", case, lambda: ops.head_linear(q, w_qk, H), T * H * (d + R) * 2 + H * R * d * 2, mma=float(T) * H * R * d)
        add("head_gemm (values, gated)", "rerupel", case, lambda: ops.head_linear(q_lat, w_kv[H * d:], H, gate=gate), T * H * (2 * d + R) * 2 + H * R * d * 2,
            mma=float(T) * H * R * d)
        xs, ws = rnd(T, H * d), rnd(R, H * d)
        add("gemm_bf16, same operations", "deepseek", case, lambda: ops.linear(xs, ws), T * (H * d + R) * 2 + H * R * d * 2, mma=float(T) * H * R * d)
        # --- experts
        h = rnd(T, W)
        p = ops.MoeWeights(router, gu, down, E, k, "sigmoid", False, 1.0, ops.Glu(7.0, 1.702, 1.0))
        used = min(E, T * k)
        wbytes, flops = used * 3 * W * F * 2, float(T) * k * 3 * W * F
        add("router, experts", "rerupel", case, lambda: ops.moe_experts(h, p), wbytes + T * k * (3 * W + 2 * F) * 2, mma=flops)
        l16 = rnd(T, E)
        add("experts (dispatch, products, combine)", "deepseek", case, lambda: ep.moe(h, l16, gu, down), wbytes + T * k * (5 * W + 2 * F) * 2, mma=flops)
        ex = ops.moe_experts(h, p)
        add("residual_norm of expert rows", "rerupel", case, lambda: ops.residual_norm(x, w32, 1e-6, bf, ops.Finished(w32, y, ex)), T * W * (12 + 2 * k))
        lay, ow = ep.layout, torch.empty(T, W, device=dev, dtype=bf)
        wts = torch.rand(T, k, device=dev)
        add("ep_combine", "deepseek", case, lambda: C.ep_combine(ep.y_local, wts, y, ow, 0, ep.peers, lay, k, (ep._calls - 1) & 1, ep.timeout_ns, st.status),
            T * W * (4 + 6 * k))
        logits, bn = ops.linear_f32(h, router), ops.moe.tile_rows(T * k / E)
        ids, place, slot = (torch.empty(T, k, dtype=torch.int32, device=dev) for _ in range(3))
        xr, tiles, nt = torch.empty(T * k, W, device=dev, dtype=bf), torch.empty(E + T * k // bn, 4, dtype=torch.int32, device=dev), torch.empty(1, dtype=torch.int32, device=dev)

        def route():
            C.moe_route(logits, wts, ids, place, st.moe_counts, E, 1, False, 1.0)
            C.moe_gather(h, ids, place, st.moe_counts, slot, xr, tiles, nt, E, bn, st.status)

        def dispatch():
            slot_ = ep._calls & 1
            ep._calls += 1
            C.ep_dispatch(h, l16, wts, ids, 0, ep.peers, lay, k, False, 1.0, slot_, ep.timeout_ns, st.status)

        add("moe_route, moe_gather", "rerupel", case, route, T * W * 2 * (k + 1) + T * E * 4)
        add("ep_dispatch", "deepseek", case, dispatch, T * W * 2 * (k + 1) + T * E * 2)
        act, yr = torch.empty(T * k, F, device=dev, dtype=bf), torch.empty(T * k, W, device=dev, dtype=bf)
        recv, cnt = ep.region.view(lay.off_recv_x, (E * ep.cap, W), bf), ep.region.view(lay.off_recv_count + ((ep._calls - 1) & 1) * E * 4, (E,), torch.int32)
        ebn = ep._bn(T * k / E)
        add("expert products, gate / up", "rerupel", case, lambda: C.moe_tiles_gemm(xr, gu, tiles, nt, act, ops.EPI_SWIGLU, bn, (7.0, 1.702, 1.0, 0.0), st.status),
            used * 2 * W * F * 2 + T * k * (W + F) * 2, mma=flops * 2 / 3)
        add("expert products, gate / up", "deepseek", case, lambda: C.moe_grouped_gemm(recv, gu, cnt, ep.act, ep.cap, True, ebn, st.status),
            used * 2 * W * F * 2 + T * k * (W + F) * 2, mma=flops * 2 / 3)
        add("expert products, down", "rerupel", case, lambda: C.moe_tiles_gemm(act, down, tiles, nt, yr, ops.EPI_NONE, bn, None, st.status),
            used * W * F * 2 + T * k * (W + F) * 2, mma=flops / 3)
        add("expert products, down", "deepseek", case, lambda: C.moe_grouped_gemm(ep.act, down, cnt, ep.y_local, ep.cap, False, ebn, st.status),
            used * W * F * 2 + T * k * (W + F) * 2, mma=flops / 3)
        # --- dense feed-forward and router
        ff = size["ffn"]
        up, gup = rnd(ff, W, std=W ** -0.5), rnd(2 * ff, W, std=W ** -0.5)
        add("gemm, squared ReLU", "rerupel", case, lambda: ops.linear_relu2(h, up), (ff * W + T * (W + ff)) * 2, mma=float(T) * W * ff)
        add("gemm, SwiGLU", "deepseek", case, lambda: ops.linear_swiglu(h, gup), (2 * ff * W + T * (W + ff)) * 2, mma=2.0 * T * W * ff)
        add("router gemm, f32", "rerupel", case, lambda: ops.linear_f32(h, router), (E * W + T * W) * 2 + T * E * 4, mma=float(T) * W * E)
        add("router gemm", "deepseek", case, lambda: ops.linear(h, router), (E * W + T * W + T * E) * 2, mma=float(T) * W * E)
        cat, lin = rnd(T, 2 * W), rnd(W, 2 * W, std=W ** -0.5)
        add("loop entry gemm, f32", "rerupel", case, lambda: ops.linear_f32(cat, lin), (2 * W * W + T * 2 * W) * 2 + T * W * 4, mma=2.0 * T * W * W)
        add("gemm of the same size", "deepseek", case, lambda: ops.linear(cat, lin), (2 * W * W + T * 3 * W) * 2, mma=2.0 * T * W * W)
    return tab.rows


def pilutar_kernel_table(size: dict) -> list[dict]:
    """Pilutar's kernels beside those of Rerupel, and of Llama and Rekudra where those have the like one."""
    from .. import ops
    from ..ops import reference

    W, H, G, d, R, E, k, F = (size[n] for n in ("width", "heads", "kv", "dim", "rank", "experts", "top", "expert_ffn"))
    r, win, real, page, dev, bf = size["rope"], size["window"], size["experts"] - size["identity"], 128, torch.device("cuda"), torch.bfloat16
    tab = KernelTable()
    add, st, C = tab.add, ops._state.get(torch.device("cuda", 0)), ops._ext.require()
    f32 = lambda *s, std=1.0: rnd(*s, dtype=torch.float32, std=std)  # noqa: E731
    ones, table, table_r = torch.ones(max(W, H * d), device=dev), reference.rope_table(4096, d // 2, 1e4).to(dev), reference.rope_table(4096, r, 5e4).to(dev)
    table_d = reference.rope_table(4096, d, 1e4).to(dev)
    up, gu, down = rnd(E, F, W, std=W ** -0.5), rnd(E, 2 * F, W, std=W ** -0.5), rnd(E, W, F, std=F ** -0.5)
    router, corr = rnd(E + 8, W, std=W ** -0.5), f32(E, std=0.02)
    Q = 64                                             # columns of the rotated part in the cache
    for case, seq, ctx, n_seq, T in (("decode 128 x 1024", step_rows(128, []), 1024, 128, 128), ("prefill 2 x 2048", step_rows(0, [2048, 2048]), 2048, 2, 4096)):
        dec = seq.n_decode > 0
        per = ctx // page + 1
        bt = torch.arange(n_seq * per, dtype=torch.int32, device=dev).view(n_seq, per)
        cl = torch.full((n_seq,), ctx, dtype=torch.int32, device=dev)
        cu = torch.arange(n_seq + 1, dtype=torch.int32, device=dev) * (T // n_seq)
        host = cu.cpu().numpy(), cl.cpu().numpy()
        base = torch.arange(n_seq, device=dev) * per * page
        slots = base + ctx - 1 if dec else (base[:, None] + torch.arange(ctx, device=dev)[None]).flatten()
        pos = torch.full((T,), ctx - 1, dtype=torch.int32, device=dev) if dec else torch.arange(ctx, dtype=torch.int32, device=dev).repeat(n_seq)
        work = None if dec else torch.from_numpy(ops.prefill_work_items(*host, 0)).cuda()
        meta = ops.AttnMeta(cu, cl, bt, n_seq if dec else 0, T // n_seq, ctx, work=work, n_items=0 if dec else work.shape[0])
        # (query, key) pairs, all and inside the window; keys a sequence's rows see
        pairs = float(n_seq * ctx) if dec else n_seq * ctx * (ctx + 1) / 2
        near = float(n_seq * min(ctx, win)) if dec else n_seq * sum(min(t + 1, win) for t in range(ctx))
        keys = n_seq * min(ctx, win) if dec else n_seq * ctx
        # --- residual and norm
        x, y, sh, z = f32(T, W), rnd(T, W), rnd(T, W), f32(T, 8)
        h = rnd(T, W)
        p = ops.MoeWeights(router[:E], up[:real], down[:real], real, k, "softmax", True, 1.0, None, corr, size["groups"], size["keep"], size["identity"])
        pr = ops.MoeWeights(router[:E], gu, down, E, k, "sigmoid", False, 1.0, ops.Glu(7.0, 1.702, 1.0))
        ex, exr = ops.moe_experts(h, p), ops.moe_experts(h, pr)
        w1 = ones[:W]
        add("residual_norm, layer norm", "pilutar", case, lambda: ops.residual_norm(x, w1, 1e-5, bf, ops.Finished(None, y), bias=w1), T * W * 12)
        add("residual_norm", "rerupel", case, lambda: ops.residual_norm(x, w1, 1e-6, bf, ops.Finished(w1, y)), T * W * 12)
        add("residual_norm, layer norm, of experts and gated row", "pilutar", case,
            lambda: ops.residual_norm(x, w1, 1e-5, bf, ops.Finished(None, y, ex, sh, z[:, 0]), bias=w1), T * W * (14 + 2 * k))
        add("residual_norm of expert rows", "rerupel", case, lambda: ops.residual_norm(x, w1, 1e-6, bf, ops.Finished(w1, y, exr)), T * W * (12 + 2 * k))
        # --- attention beside the recurrence
        nq, nk = H * d, G * d
        kc, vc = (rnd(n_seq * per, G, page, d) for _ in range(2))
        proj = rnd(T, nq + 2 * nk)
        qp = ops.QkvNorm(f32(nq + 2 * nk), ones[:nq], ones[:nk])
        add("norm_qkv", "pilutar", case, lambda: ops.norm_qkv(proj, qp, table, pos, slots, kc, vc, H, G, d, d, d, 1e-5), T * (nq + 2 * nk) * 4)
        add("rope_kvwrite", "llama", case, lambda: ops.rope_kvwrite(proj[:, :nq], proj[:, nq:nq + nk], proj[:, nq + nk:], table_d, pos, slots, kc, vc, d),
            T * (2 * nq + 4 * nk) * 2)
        q, cat = rnd(T, nq), torch.empty(T, 2 * nq, device=dev, dtype=bf)
        mods = ops.ScoreMods(win, 30.0, 0.5)
        add("attention, window, capped", "pilutar", case, lambda: ops.paged_attention(q, kc, vc, meta, d ** -0.5, d, out=cat[:, :nq], mods=mods),
            keys * G * d * 4 + T * nq * 4, mma=0.0 if dec else near * H * d * 2)
        add("attention", "llama", case, lambda: ops.paged_attention(q, kc, vc, meta, d ** -0.5, d), n_seq * ctx * G * d * 4 + T * nq * 4,
            mma=0.0 if dec else pairs * H * d * 2)
        # --- recurrences
        state = torch.zeros(n_seq, H, d, d, device=dev)
        pg, zg = rnd(T, 4 * nq), f32(T, nq)
        gp = ops.GatedLinearParams(torch.full((nq,), 2.0, device=dev), ones[:d], 16.0)
        state_bytes = n_seq * H * d * d * 4 * (2 if dec else 1)
        add("gated_linear", "pilutar", case, lambda: ops.gated_linear(pg, zg, gp, state, seq, H, d, d, 1e-5, cat[:, nq:], 0.5), state_bytes + T * nq * 14,
            fma=0.0 if dec else 3.0 * T * H * d * d)
        pd, dg, taps = rnd(T, 3 * nq + H), rnd(T, 2 * nq), 4
        dp = ops.DeltaParams(f32(taps, 3 * nq, std=0.3), -ones[:H], torch.full((nq,), -3.0, device=dev), ones[:d])
        bank = rnd(2 * n_seq, taps - 1, 3 * nq)
        add("delta_rule", "rekudra", case, lambda: ops.delta_rule(pd, dg[:, :nq], dg[:, nq:2 * nq], dp, bank, state, seq, 3 * nq, H, H, d, d, nq, 1e-5),
            state_bytes + T * (6 * nq + H) * 2 + n_seq * (taps - 1) * 6 * nq * (2 if dec else 1), fma=0.0 if dec else 4.0 * T * H * d * d)
        # --- latent attention
        cache, plain = rnd(n_seq * per, page, R + Q), rnd(n_seq * per, page, R)
        pl = rnd(T, nq + R + r + H)
        rope = ops.SharedRope(pl[:, nq + R:nq + R + r], pl[:, :nq], H, d - r, R, table_r, pos)
        add("latent_write, rotated", "pilutar", case, lambda: ops.latent_write(pl[:, nq:nq + R], ones[:R], 1e-5, slots, cache, rope), T * ((R + r) * 4 + H * r * 4))
        add("latent_write", "rerupel", case, lambda: ops.latent_write(pl[:, nq:nq + R], ones[:R], 1e-6, slots, plain), T * R * 4)
        w_qk, w_kv = rnd(H * (R + Q), d, std=d ** -0.5), rnd(2 * nq, R + Q, std=R ** -0.5)
        w_qk_p, w_kv_p = w_qk[:H * R], rnd(2 * nq, R, std=R ** -0.5)
        gate, gate_e = pl[:, nq + R + r:], rnd(T, nq)
        rows = ops.token_rows(meta, T, dev)
        q_lat, q_lat_p = rnd(T, H * (R + Q)), rnd(T, H * R)
        if dec:
            add("latent_attend, rotated, window", "pilutar", case, lambda: ops.latent_attend(q_lat, cache, meta, rows, H, 0.1, pos, R, win),
                keys * (R + r) * 2 + T * H * (2 * R + r) * 2, mma=near * H * (2 * R + r))
            add("latent_attend", "rerupel", case, lambda: ops.latent_attend(q_lat_p, plain, meta, rows, H, 0.1, pos), n_seq * ctx * R * 2 + T * H * R * 4,
                mma=pairs * H * 2 * R)
        else:
            out = torch.empty(T, nq, device=dev, dtype=bf)
            plan = ops.plan_latent_prefill(*host, 0, R, H, d, d, win)
            meta.expand = tuple(torch.from_numpy(a).cuda() for a in plan)
            expand = float(len(plan[0]) * 128) * R * 2 * nq
            add("latent_prefill, rotated, window", "pilutar", case, lambda: ops.latent_prefill(pl[:, :nq], cache, w_kv, meta, H, 0.1, gate, out, win), T * nq * 6,
                mma=near * H * 2 * d + expand)
            add("latent_prefill", "rerupel", case, lambda: ops.latent_prefill(pl[:, :nq], plain, w_kv_p, meta, H, 0.1, gate_e, out), T * nq * 8,
                mma=pairs * H * 2 * d + expand)
        if dec:                                        # prompts take the expanded form
            add("head_gemm (queries)", "pilutar", case, lambda: ops.head_linear(pl[:, :nq], w_qk, H), T * H * (d + R + r) * 2 + H * R * (d - r) * 2,
                mma=float(T) * H * R * (d - r))
            add("head_gemm (queries)", "rerupel", case, lambda: ops.head_linear(pl[:, :nq], w_qk_p, H), T * H * (d + R) * 2 + H * R * d * 2, mma=float(T) * H * R * d)
            add("head_gemm (values, gate per head)", "pilutar", case, lambda: ops.head_linear(q_lat_p, w_kv[nq:, :R], H, gate=gate), T * H * (d + R) * 2 + H * R * d * 2,
                mma=float(T) * H * R * d)
            add("head_gemm (values, gated)", "rerupel", case, lambda: ops.head_linear(q_lat_p, w_kv_p[nq:], H, gate=gate_e), T * H * (2 * d + R) * 2 + H * R * d * 2,
                mma=float(T) * H * R * d)
        # --- experts
        logits = ops.linear_f32(h, router)
        n_id = float((ex.slot < 0).float().mean()) if size["identity"] else 0.0
        run_k, used = k * (1.0 - n_id), float(min(real, T * k))
        add("router, experts", "pilutar", case, lambda: ops.moe_experts(h, p, logits), used * 2 * W * F * 2 + T * run_k * (3 * W + 2 * F) * 2,
            mma=float(T) * run_k * 2 * W * F)
        add("router, experts", "rerupel", case, lambda: ops.moe_experts(h, pr, logits), min(E, T * k) * 3 * W * F * 2 + T * k * (3 * W + 2 * F) * 2,
            mma=float(T) * k * 3 * W * F)
        wts, bn = torch.empty(T, k, device=dev), ops.moe.tile_rows(T * k / E)
        ids, place, slot = (torch.empty(T, k, dtype=torch.int32, device=dev) for _ in range(3))
        xr, tiles, nt = torch.empty(T * k, W, device=dev, dtype=bf), torch.empty(E + T * k // bn, 4, dtype=torch.int32, device=dev), torch.empty(1, dtype=torch.int32, device=dev)

        def route(grouped: bool):
            n = real if grouped else E
            if grouped:
                C.moe_route(logits, wts, ids, place, st.moe_counts, n, 0, True, 1.0, corr, size["groups"], size["keep"], size["identity"])
            else:
                C.moe_route(logits, wts, ids, place, st.moe_counts, n, 1, False, 1.0)
            C.moe_gather(h, ids, place, st.moe_counts, slot, xr, tiles, nt, n, bn, st.status)

        act, yr = torch.empty(T * k, F, device=dev, dtype=bf), torch.empty(T * k, W, device=dev, dtype=bf)
        add("moe_route, moe_gather, groups", "pilutar", case, lambda: route(True), T * W * 2 * (run_k + 1) + T * E * 4)
        add("expert products, squared ReLU", "pilutar", case, lambda: C.moe_tiles_gemm(xr, up[:real], tiles, nt, act, ops.EPI_RELU2, bn, None, st.status),
            used * W * F * 2 + T * run_k * (W + F) * 2, mma=float(T) * run_k * W * F)
        add("moe_route, moe_gather", "rerupel", case, lambda: route(False), T * W * 2 * (k + 1) + T * E * 4)
        add("expert products, gate / up", "rerupel", case, lambda: C.moe_tiles_gemm(xr, gu, tiles, nt, act, ops.EPI_SWIGLU, bn, (7.0, 1.702, 1.0, 0.0), st.status),
            min(E, T * k) * 2 * W * F * 2 + T * k * (W + F) * 2, mma=float(T) * k * 2 * W * F)
        # --- products that only this design has in this form
        ff = size["ffn"]
        w_gu, w_dec, w_out = rnd(2 * ff, W, std=W ** -0.5), rnd(nq, 16), rnd(W, 2 * nq + ff, std=(2 * nq + ff) ** -0.5)
        wide = rnd(T, 2 * nq + ff)
        add("gemm, ReLU-gated, into columns", "pilutar", case, lambda: ops.linear_swiglu(h, w_gu, out=wide[:, 2 * nq:], glu=ops.REGLU), (2 * ff * W + T * (W + ff)) * 2,
            mma=2.0 * T * W * ff)
        add("gemm, gated unit", "rerupel", case, lambda: ops.linear_swiglu(h, w_gu, glu=ops.Glu(7.0, 1.702, 1.0)), (2 * ff * W + T * (W + ff)) * 2, mma=2.0 * T * W * ff)
        add("gemm, all output projections", "pilutar", case, lambda: ops.linear(wide, w_out), (w_out.numel() + wide.numel() + T * W) * 2, mma=float(T) * w_out.numel())
        w_plain, x_plain = w_out[:, :nq].contiguous(), wide[:, :nq].contiguous()
        add("gemm, output projection", "rerupel", case, lambda: ops.linear(x_plain, w_plain), (w_plain.numel() + x_plain.numel() + T * W) * 2, mma=float(T) * w_plain.numel())
        low = rnd(T, 4 * nq)[:, :16]
        add("gemm, decay logits, f32", "pilutar", case, lambda: ops.linear_f32(low, w_dec), (w_dec.numel() + T * 16) * 2 + T * nq * 4, mma=float(T) * w_dec.numel())
    return tab.rows


def noridra_kernel_table(size: dict) -> list[dict]:
    """Noridra's kernels beside those of Pilutar, and of Rekudra where that has the like one."""
    from .. import ops
    from ..ops import reference

    W, H, G, d, E, k, F, S = (size[n] for n in ("width", "heads", "kv", "dim", "experts", "top", "expert_ffn", "state"))
    win, chunk, page, dev, bf, taps, I, dr = size["window"], size["chunk"], 128, torch.device("cuda"), torch.bfloat16, 4, 2 * W, W // 16
    tab = KernelTable()
    add = tab.add
    f32 = lambda *s, std=1.0: rnd(*s, dtype=torch.float32, std=std)  # noqa: E731
    ones = torch.ones(max(W, H * d, I), device=dev)
    table, table_d = reference.rope_table(4096, d // 2, 1e4).to(dev), reference.rope_table(4096, d, 1e4).to(dev)
    gu, down, up = rnd(E, 2 * F, W, std=W ** -0.5), rnd(E, W, F, std=F ** -0.5), rnd(E, F, W, std=W ** -0.5)
    router = rnd(E + 8, W, std=W ** -0.5)
    for case, seq, ctx, n_seq, T in (("decode 128 x 1024", step_rows(128, []), 1024, 128, 128), ("prefill 2 x 2048", step_rows(0, [2048, 2048]), 2048, 2, 4096)):
        dec = seq.n_decode > 0
        per = ctx // page + 1
        bt = torch.arange(n_seq * per, dtype=torch.int32, device=dev).view(n_seq, per)
        cl = torch.full((n_seq,), ctx, dtype=torch.int32, device=dev)
        cu = torch.arange(n_seq + 1, dtype=torch.int32, device=dev) * (T // n_seq)
        base = torch.arange(n_seq, device=dev) * per * page
        slots = base + ctx - 1 if dec else (base[:, None] + torch.arange(ctx, device=dev)[None]).flatten()
        pos = torch.full((T,), ctx - 1, dtype=torch.int32, device=dev) if dec else torch.arange(ctx, dtype=torch.int32, device=dev).repeat(n_seq)
        work = None if dec else torch.from_numpy(ops.prefill_work_items(cu.cpu().numpy(), cl.cpu().numpy(), 0)).cuda()
        meta = ops.AttnMeta(cu, cl, bt, n_seq if dec else 0, T // n_seq, ctx, work=work, n_items=0 if dec else work.shape[0])
        near_c = float(n_seq * min(ctx, chunk)) if dec else n_seq * sum(t % chunk + 1 for t in range(ctx))      # (query, key) pairs
        near_w = float(n_seq * min(ctx, win)) if dec else n_seq * sum(min(t + 1, win) for t in range(ctx))
        keys = n_seq * min(ctx, chunk) if dec else n_seq * ctx
        # --- residual, norm, convolution ahead of a sublayer
        x, y, h, w1 = f32(T, W), rnd(T, W), rnd(T, W), ones[:W]
        conv = ops.InputConv(f32(taps, W, std=0.3), f32(2 * n_seq, taps - 1, W))
        norm = ops.GroupNorm(size["norm_groups"], 1e-6, W)
        p = ops.MoeWeights(router[:E], gu, down, E, k, "sigmoid", on_input=True)
        pp = ops.MoeWeights(router[:E], up, down, E, k, "softmax", True, 1.0, None, f32(E, std=0.02), size["groups"], size["keep"])
        ex, exp = ops.moe_experts(h, p), ops.moe_experts(h, pp)
        banks = n_seq * (taps - 1) * W * 4 * (2 if dec else 1)
        add("post_norm, convolution", "noridra", case, lambda: ops.post_norm(x, norm, bf, seq, ops.Finished(w1, y), w1, 2.0, conv=conv), T * W * 12 + banks)
        add("residual_norm, layer norm", "pilutar", case, lambda: ops.residual_norm(x, w1, 1e-5, bf, ops.Finished(None, y), bias=w1), T * W * 12)
        add("post_norm, convolution, of experts", "noridra", case, lambda: ops.post_norm(x, norm, bf, seq, ops.Finished(w1, None, ex), w1, 2.0, conv=conv),
            T * W * (2 * k + 10) + banks)
        add("residual_norm, layer norm, of experts", "pilutar", case, lambda: ops.residual_norm(x, w1, 1e-5, bf, ops.Finished(None, None, exp), bias=w1),
            T * W * (2 * k + 10))
        # --- attention
        nq, nk = H * d, G * d
        kc, vc = (rnd(n_seq * per, G, page, d) for _ in range(2))
        pa, q = rnd(T, 2 * nq + nk), rnd(T, nq)
        add("head_norm_qkv", "noridra", case, lambda: ops.head_norm_qkv(pa, ones[:d], ones[:d], slots, kc, vc, H, G, d, nq, d, 1e-6), T * (4 * nq + 6 * nk))
        qn, pn = ops.QkvNorm(ones.new_zeros(nq + 2 * nk), ones[:nq], ones[:nk]), rnd(T, nq + 2 * nk)
        add("norm_qkv", "pilutar", case, lambda: ops.norm_qkv(pn, qn, table, pos, slots, kc, vc, H, G, d, d, d, 1e-5), T * (nq + 2 * nk) * 4)
        mods = ops.ScoreMods(softcap=30.0, chunk=chunk, sink=True, distance=torch.full((2, H), 0.5, device=dev))
        gate = pa[:, nq + nk:]
        add("attention, chunks, bias, sink, gate", "noridra", case, lambda: ops.paged_attention(q, kc, vc, meta, d ** -0.5, d, gate=gate, mods=mods),
            keys * G * d * 4 + T * nq * 6, mma=0.0 if dec else near_c * H * d * 2)
        mw = ops.ScoreMods(win, 30.0, 0.5)
        add("attention, window, capped", "pilutar", case, lambda: ops.paged_attention(q, kc, vc, meta, d ** -0.5, d, mods=mw),
            n_seq * (min(ctx, win) if dec else ctx) * G * d * 4 + T * nq * 4, mma=0.0 if dec else near_w * H * d * 2)
        # --- recurrences
        state = torch.zeros(n_seq, H, d, d, device=dev)
        state_bytes = n_seq * H * d * d * 4 * (2 if dec else 1)
        pd, bank = rnd(T, 4 * nq + 2 * H), rnd(2 * n_seq, taps - 1, 3 * nq)
        cw = f32(taps, 3 * nq, std=0.3)
        dn = ops.DeltaParams(cw, -ones[:H], torch.full((H,), -3.0, device=dev), ones[:d], True)
        hist = n_seq * (taps - 1) * 6 * nq * (2 if dec else 1)
        add("delta_rule, decay per head", "noridra", case,
            lambda: ops.delta_rule(pd, pd[:, 3 * nq + H:3 * nq + 2 * H], pd[:, 3 * nq + 2 * H:], dn, bank, state, seq, 3 * nq, H, H, d, d, nq, 1e-6),
            state_bytes + T * (5 * nq + 2 * H) * 2 + hist, fma=0.0 if dec else 4.0 * T * H * d * d)
        dg, dk = rnd(T, 2 * nq), ops.DeltaParams(cw, -ones[:H], torch.full((nq,), -3.0, device=dev), ones[:d])
        add("delta_rule", "rekudra", case, lambda: ops.delta_rule(pd, dg[:, :nq], dg[:, nq:], dk, bank, state, seq, 3 * nq, H, H, d, d, nq, 1e-5),
            state_bytes + T * (6 * nq + H) * 2 + hist, fma=0.0 if dec else 4.0 * T * H * d * d)
        xz, f, dt = rnd(T, 2 * I), rnd(T, dr + 2 * S), f32(T, I)
        cs, cws = rnd(2 * n_seq, taps - 1, I), f32(taps, I, std=0.3)
        add("conv_silu", "noridra", case, lambda: ops.conv_silu(xz, cws, ones[:I], cs, seq), T * I * 4 + n_seq * (taps - 1) * I * 2 * (2 if dec else 1))
        kq, vq = rnd(n_seq * per, G, page, d), rnd(n_seq * per, G, page, d)
        cq, bq = f32(taps, nq + 2 * nk, std=0.3), rnd(2 * n_seq, taps - 1, nq + 2 * nk)
        add("conv_qkv", "rekudra", case, lambda: ops.conv_qkv(pn, cq, bq, table_d, pos, seq, slots, kq, vq, H, G, d, d, d, 1e-5),
            T * (nq + 2 * nk) * 4 + n_seq * (taps - 1) * (nq + 2 * nk) * 2 * (2 if dec else 1))
        sp = ops.ScanParams(-torch.rand(I, S, device=dev) - 0.1, torch.full((I,), -4.0, device=dev), ones[:I])
        ss = torch.zeros(n_seq, I, S, device=dev)
        add("selective_scan", "noridra", case, lambda: ops.selective_scan(dt, xz[:, :I], xz[:, I:], f[:, dr:dr + S], f[:, dr + S:], sp, ss, seq),
            n_seq * I * S * 4 * (2 if dec else 1) + T * I * 10, sfu=0.0 if dec else float(T) * I * S)
        pg, zg = rnd(T, 4 * nq), f32(T, nq)
        gp, og = ops.GatedLinearParams(torch.full((nq,), 2.0, device=dev), ones[:d], 16.0), rnd(T, nq)
        add("gated_linear", "pilutar", case, lambda: ops.gated_linear(pg, zg, gp, state, seq, H, d, d, 1e-5, og), state_bytes + T * nq * 14,
            fma=0.0 if dec else 3.0 * T * H * d * d)
        # --- experts
        logits = ops.linear_f32(h, router)
        used = float(min(E, T * k))
        add("router, experts, weighted inputs", "noridra", case, lambda: ops.moe_experts(h, p, logits), used * 3 * W * F * 2 + T * k * (3 * W + 2 * F) * 2,
            mma=float(T) * k * 3 * W * F)
        add("router, experts", "pilutar", case, lambda: ops.moe_experts(h, pp, logits), used * 2 * W * F * 2 + T * k * (3 * W + 2 * F) * 2, mma=float(T) * k * 2 * W * F)
        # --- products of the scan's small matrices
        w_x, w_dt, low, w_dec = rnd(dr + 2 * S, I, std=I ** -0.5), rnd(I, dr, std=dr ** -0.5), rnd(T, 4 * nq)[:, :16], rnd(nq, 16)
        u = xz[:, :I].contiguous()
        add("gemm, step sizes | B | C", "noridra", case, lambda: ops.linear(u, w_x), (w_x.numel() + u.numel() + T * (dr + 2 * S)) * 2, mma=float(T) * w_x.numel())
        add("gemm, step sizes, f32", "noridra", case, lambda: ops.linear_f32(f[:, :dr], w_dt), (w_dt.numel() + T * dr) * 2 + T * I * 4, mma=float(T) * w_dt.numel())
        add("gemm, decay logits, f32", "pilutar", case, lambda: ops.linear_f32(low, w_dec), (w_dec.numel() + T * 16) * 2 + T * nq * 4, mma=float(T) * w_dec.numel())
    return tab.rows


def run(args) -> dict:
    from .clocks import ClockSampler

    base, design = DESIGNS[args.layer_bench]
    sizes, table = {"rekudra": (SIZES, kernel_table), "rerupel": (MOE_SIZES, latent_kernel_table), "pilutar": (PILUTAR_SIZES, pilutar_kernel_table),
                    "noridra": (NORIDRA_SIZES, noridra_kernel_table)}[design]
    out = {"metric": f"layer throughput, {design} beside {base} at equal layer sizes", "unit": "tok/s", "n_gpus": 1, "dtype": "bf16",
           "layers": LAYERS if design in ("rekudra", "noridra") else MOE_RUNS, "data": "synthetic: uniform-random token ids, random weights", "peaks": peaks(), "sizes": {}}
    with ClockSampler(0) as clocks:
        for name, size in sizes.items():
            rec = {"kernels": table(size)}
            torch.cuda.empty_cache()
            for d in (base, design):
                b = Bench(d, size, autotune=not args.no_autotune)
                rec[d] = {"weight_bytes": b.engine.model.weight_bytes(), "prefill": [b.prefill(*c) for c in PREFILL], "decode": [b.decode(*c) for c in DECODE]}
                del b
                torch.cuda.empty_cache()
            out["sizes"][name] = rec
    summary = clocks.summary()
    out["clocks"] = {k: summary.get(k) for k in ("sm_mhz", "sm_max_mhz", "reasons", "power_w_max")}
    from .. import ops

    ops.check_status()
    return out
