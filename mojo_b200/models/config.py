"""Architecture descriptions. Field names follow the Hugging Face `config.json` keys so a checkpoint directory
can be read directly; named presets cover the architectures the engine is benchmarked on."""
from __future__ import annotations

import json
from dataclasses import dataclass, field, asdict
from pathlib import Path


@dataclass
class RotarySpec:
    """Rotary embedding of one layer: the first `dims` dimensions of a head turn, the rest pass. `scaling` is the Llama-3.1
    frequency rescale (factor, low, high, original) or None. `interleaved`: neighbours pair up instead of halves."""
    dims: int = 0
    base: float = 10000.0
    scaling: dict | None = None
    interleaved: bool = False


@dataclass
class ExpertSpec:
    """Size and constants of one gated feed-forward: min(g, limit), clamp(u, -limit, limit)."""
    ffn: int = 0
    limit: float = float("inf")


@dataclass
class MoeSpec:
    """Mixture of experts of one layer. The shared expert runs for every token. Experts (identity ones included) form `groups`
    runs of neighbours, of which a token's choice keeps `keep`."""
    experts: int = 0
    top: int = 0
    scale: float = 1.0                     # on the router's weights
    expert: ExpertSpec = field(default_factory=ExpertSpec)
    shared: ExpertSpec | None = None
    groups: int = 1
    keep: int = 1
    identity: int = 0                      # router outputs past the experts whose result is the input itself


@dataclass
class LoopSpec:
    """Layers start .. stop - 1 run `times` times in a row with the same weights."""
    start: int = 0
    stop: int = 0
    times: int = 1


@dataclass
class BigramSpec:
    """Hashed bigram embedding: row (previous * mul_prev + current * mul_cur) mod buckets."""
    buckets: int = 0
    mul_prev: int = 0
    mul_cur: int = 0


@dataclass
class LayerSpec:
    """One layer of a decoder whose layers differ: which mixer it has, the mixer's sizes, and its feed-forward."""
    mixer: str = "attention"               # "attention" | "channel_delta" | "delta" | "latent_attention" | "gated_linear" | "mamba1" | "parallel"
    heads: int = 0
    kv_heads: int = 0
    dim: int = 0                           # query / key size of a head
    vdim: int = 0                          # value size of a head
    conv_taps: int = 1                     # short causal convolution (1: none)
    scale: float = 1.0                     # attention: factor on the scores
    rot: RotarySpec = field(default_factory=RotarySpec)
    kv_from: int | None = None             # attention: use the keys and values of this earlier layer
    ffn: int = 0                           # feed-forward width (0: the layer has no feed-forward)
    decay_rank: int = 0                    # delta rule: ranks of the decay and gate projections (0: taken from the checkpoint)
    gate_rank: int = 0
    kv_rank: int = 0                       # latent attention: size of the cached latent
    moe: MoeSpec | None = None             # mixture of experts in place of a dense feed-forward
    window: int = 0                        # attention: positions a token sees, itself included (0: all before it)
    softcap: float = 0.0                   # attention: scores become softcap * tanh(score / softcap) (0: they do not)
    chunk: int = 0                         # attention: positions see only those of their own run of `chunk` (0: all before them)
    inner: int = 0                         # selective scan: channels, states of a channel, rank of the step sizes
    state: int = 0
    dt_rank: int = 0
    tau: float = 1.0                       # gated linear attention: decays are sigmoid(z)^(1 / tau)
    parts: list["LayerSpec"] | None = None # "parallel": the mixers that run side by side ...
    part_scales: list[float] | None = None # ... and the factors of their results


@dataclass
class ModelConfig:
    architecture: str = "llama"            # "llama" | "deepseek_v2" | "rekudra" | "rerupel" | "pilutar" | "noridra"
    hidden_size: int = 4096
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 8
    head_dim: int = 128
    intermediate_size: int = 14336
    vocab_size: int = 128256
    rms_norm_eps: float = 1e-5
    rope_theta: float = 500000.0
    rope_scaling: dict | None = None
    max_position_embeddings: int = 8192
    tie_word_embeddings: bool = False
    # quantisation of the linear weights: None | "fp8_block" (128x128 e4m3 + f32 scales) | "gguf"
    quantization: str | None = None
    # DeepSeek-V2 (MLA + MoE)
    kv_lora_rank: int = 0
    q_lora_rank: int = 0
    qk_rope_head_dim: int = 0
    qk_nope_head_dim: int = 0
    v_head_dim: int = 0
    n_routed_experts: int = 0
    n_shared_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    first_k_dense_replace: int = 0
    routed_scaling_factor: float = 1.0
    norm_topk_prob: bool = False
    rope_interleaved: bool = False
    # decoders whose layers differ from one another, and whose residual is several mixed streams
    layers: list[LayerSpec] | None = None
    residual_streams: int = 1
    embedding_scale: float = 1.0
    bigram: BigramSpec | None = None
    loop: LoopSpec | None = None           # layers that run several times
    residual_mult: float = 1.0             # on everything a sublayer adds to the residual
    logit_softcap: float | None = None
    logit_scale: float = 1.0
    # decoders that normalise after the sum: x <- norm(residual_alpha * x + sublayer(x + conv(x)))
    residual_alpha: float = 1.0
    norm_groups: int = 1                   # runs of columns that the norm treats one by one
    input_taps: int = 1                    # taps of the convolution over time on what a sublayer reads
    extra: dict = field(default_factory=dict)

    def to_dict(self) -> dict:
        return asdict(self)

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0

    @property
    def is_moe(self) -> bool:
        return self.n_routed_experts > 0

    def layer_runs(self) -> list[tuple[int, bool]]:
        """The layers in the order they run, as (layer, whether a pass of the loop begins right before it)."""
        n, lp = self.num_layers, self.loop
        if lp is None:
            return [(i, False) for i in range(n)]
        body = [(i, i == lp.start) for i in range(lp.start, lp.stop)]
        return [(i, False) for i in range(lp.start)] + body * lp.times + [(i, False) for i in range(lp.stop, n)]

    def mixers(self) -> list[LayerSpec]:
        """Every mixer of a config that lists its layers; those that run side by side one by one."""
        return [m for s in self.layers for m in (s.parts or [s])]

    def kv_bytes_per_token(self, dtype_bytes: int = 2, tp: int = 1) -> int:
        if self.architecture == "pilutar":
            return sum(s.kv_heads * (s.dim + s.vdim) if s.mixer == "attention" else s.kv_rank + s.rot.dims for s in self.mixers()
                       if s.mixer != "gated_linear") * dtype_bytes
        if self.architecture == "rerupel":
            return sum(self.layers[i].kv_rank for i, _ in self.layer_runs()) * dtype_bytes
        if self.layers is not None:
            return sum(s.kv_heads * (s.dim + s.vdim) for s in self.layers if s.mixer == "attention" and s.kv_from is None) * dtype_bytes
        if self.is_mla:
            return self.num_layers * (self.kv_lora_rank + self.qk_rope_head_dim) * dtype_bytes
        return self.num_layers * 2 * max(1, self.num_kv_heads // tp) * self.head_dim * dtype_bytes

    def num_params(self) -> int:
        h = self.hidden_size
        emb = self.vocab_size * h * (1 if self.tie_word_embeddings else 2)
        if self.architecture == "rerupel":
            n = emb + h + (self.bigram.buckets + 1 if self.bigram else 0) * h + (2 * h * h if self.loop else 0)
            for s in self.layers:
                n += h * (s.heads * (s.dim + 2 * s.vdim) + s.kv_rank + 4) + s.heads * (s.dim + s.vdim) * s.kv_rank + 2 * h * s.ffn
                if s.moe is not None:
                    n += h * (s.moe.experts + 3 * s.moe.experts * s.moe.expert.ffn + 3 * (s.moe.shared.ffn if s.moe.shared else 0))
            return n
        if self.architecture == "pilutar":
            n = emb + 2 * h
            for s in self.mixers():
                out = s.heads * s.vdim
                if s.mixer == "attention":
                    n += h * (s.heads * s.dim + s.kv_heads * (s.dim + s.vdim) + out)
                elif s.mixer == "latent_attention":
                    n += h * (s.heads * (s.dim + s.rot.dims + 1) + s.kv_rank + s.rot.dims + out) + s.heads * (s.dim + s.vdim) * s.kv_rank
                else:
                    n += h * (2 * s.heads * s.dim + 3 * out + s.decay_rank) + s.heads * s.dim * s.decay_rank
            for s in self.layers:
                n += 2 * h + 3 * h * s.ffn
                if s.moe is not None:
                    n += h * (s.moe.experts + s.moe.identity + 2 * s.moe.experts * s.moe.expert.ffn + (2 * s.moe.shared.ffn + 1 if s.moe.shared else 0))
            return n
        if self.architecture == "noridra":
            n = emb + h + self.max_position_embeddings * h
            for s in self.layers:
                if s.mixer == "mamba1":
                    n += s.inner * (3 * h + 2 * s.dt_rank + 3 * s.state + s.conv_taps + 3)
                elif s.mixer == "delta":
                    n += h * (2 * s.kv_heads * s.dim + 3 * s.heads * s.vdim + 2 * s.heads) + s.conv_taps * (2 * s.kv_heads * s.dim + s.heads * s.vdim)
                else:
                    n += h * (3 * s.heads + s.kv_heads) * s.dim
                n += (2 if s.moe else 1) * h * (2 + self.input_taps)
                if s.moe is not None:
                    n += h * (s.moe.experts + 3 * s.moe.experts * s.moe.expert.ffn)
            return n
        if self.layers is not None:
            n = emb + h
            for s in self.layers:
                kv = 0 if s.kv_from is not None else s.kv_heads
                n += h * (s.heads * s.vdim + 3 * s.ffn)
                if s.mixer == "attention":
                    n += h * (s.heads * (s.dim + 1) + kv * (s.dim + s.vdim))
                else:
                    n += h * (2 * s.kv_heads * s.dim + s.heads * (s.vdim + 1) + s.decay_rank + s.gate_rank)
                    n += s.heads * (s.dim * s.decay_rank + s.vdim * s.gate_rank)
            return n
        if self.architecture == "llama":
            attn = h * (self.num_heads + 2 * self.num_kv_heads) * self.head_dim + self.num_heads * self.head_dim * h
            mlp = 3 * h * self.intermediate_size
            return emb + self.num_layers * (attn + mlp + 2 * h) + h
        attn = h * self.num_heads * (self.qk_nope_head_dim + self.qk_rope_head_dim) + h * (self.kv_lora_rank + self.qk_rope_head_dim) \
            + self.kv_lora_rank * self.num_heads * (self.qk_nope_head_dim + self.v_head_dim) + self.num_heads * self.v_head_dim * h
        dense = 3 * h * self.intermediate_size
        moe = 3 * h * self.moe_intermediate_size * (self.n_routed_experts + self.n_shared_experts) + h * self.n_routed_experts
        nd = self.first_k_dense_replace
        return emb + self.num_layers * attn + nd * dense + (self.num_layers - nd) * moe

    @staticmethod
    def from_hf(path: str | Path) -> "ModelConfig":
        cfg = json.loads((Path(path) / "config.json").read_text())
        if cfg.get("architecture") in LAYERED_ARCHITECTURES:
            return ModelConfig.from_layered(cfg)
        arch = (cfg.get("architectures") or ["LlamaForCausalLM"])[0]
        n_heads = cfg["num_attention_heads"]
        c = ModelConfig(
            architecture="deepseek_v2" if "Deepseek" in arch else "llama",
            hidden_size=cfg["hidden_size"], num_layers=cfg["num_hidden_layers"], num_heads=n_heads,
            num_kv_heads=cfg.get("num_key_value_heads", n_heads),
            head_dim=cfg.get("head_dim") or cfg["hidden_size"] // n_heads,
            intermediate_size=cfg["intermediate_size"], vocab_size=cfg["vocab_size"],
            rms_norm_eps=cfg.get("rms_norm_eps", 1e-5), rope_theta=cfg.get("rope_theta", 10000.0),
            rope_scaling=cfg.get("rope_scaling"), max_position_embeddings=cfg.get("max_position_embeddings", 8192),
            tie_word_embeddings=cfg.get("tie_word_embeddings", False),
        )
        q = cfg.get("quantization_config") or {}
        if q.get("quant_method") == "fp8" and q.get("weight_block_size"):
            c.quantization = "fp8_block"
        if c.architecture == "deepseek_v2":
            c.kv_lora_rank = cfg["kv_lora_rank"]; c.q_lora_rank = cfg.get("q_lora_rank") or 0
            c.qk_rope_head_dim = cfg["qk_rope_head_dim"]; c.qk_nope_head_dim = cfg["qk_nope_head_dim"]
            c.v_head_dim = cfg["v_head_dim"]; c.n_routed_experts = cfg["n_routed_experts"]
            c.n_shared_experts = cfg.get("n_shared_experts") or 0; c.num_experts_per_tok = cfg["num_experts_per_tok"]
            c.moe_intermediate_size = cfg["moe_intermediate_size"]; c.first_k_dense_replace = cfg.get("first_k_dense_replace", 0)
            c.routed_scaling_factor = cfg.get("routed_scaling_factor", 1.0); c.norm_topk_prob = cfg.get("norm_topk_prob", False)
            c.rope_interleaved = True
        return c


    @staticmethod
    def from_layered(cfg: dict) -> "ModelConfig":
        """A config that lists its layers one by one (`layers[i]`: type, mixer sizes, feed-forward)."""
        if LAYERED_ARCHITECTURES[cfg["architecture"]] == "rerupel":
            return ModelConfig._from_latent_layers(cfg)
        if LAYERED_ARCHITECTURES[cfg["architecture"]] == "pilutar":
            return ModelConfig._from_parallel_layers(cfg)
        if LAYERED_ARCHITECTURES[cfg["architecture"]] == "noridra":
            return ModelConfig._from_postnorm_layers(cfg)
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            m, mlp = entry["mixer"], entry.get("mlp")
            if entry["type"] not in ("attention", "channel_delta"):
                raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            rot = m.get("rot") or {}
            spec = LayerSpec(
                mixer=entry["type"], heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], conv_taps=m.get("conv") or 1,
                scale=m.get("scale", 1.0), rot=RotarySpec(rot.get("dims", 0), rot.get("base", 10000.0), rot.get("scaling")),
                kv_from=m.get("kv_from"), ffn=mlp["ff"] if mlp is not None else 0)
            if spec.kv_from is not None:
                src = layers[spec.kv_from] if 0 <= spec.kv_from < i else None
                if src is None or src.mixer != "attention" or src.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with keys and values of its own")
                if (src.kv_heads, src.dim, src.vdim) != (spec.kv_heads, spec.dim, spec.vdim):
                    raise ValueError(f"layer {i}: head sizes differ from those of layer {spec.kv_from}, whose keys and values it uses")
            layers.append(spec)
        first = next((s for s in layers if s.mixer == "attention"), layers[0])
        return ModelConfig(architecture=LAYERED_ARCHITECTURES[cfg["architecture"]], hidden_size=cfg["width"], num_layers=len(layers),
                           num_heads=first.heads, num_kv_heads=first.kv_heads, head_dim=first.dim,
                           intermediate_size=max((s.ffn for s in layers), default=0), vocab_size=cfg["vocab"], rms_norm_eps=cfg["norm"]["eps"],
                           max_position_embeddings=0, layers=layers, residual_streams=cfg.get("streams", 1),
                           embedding_scale=cfg.get("embedding", {}).get("scale", 1.0))


    @staticmethod
    def _from_latent_layers(cfg: dict) -> "ModelConfig":
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            m, mlp = entry["mixer"], entry.get("mlp")
            if entry["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
            spec = LayerSpec(mixer="latent_attention", heads=m["heads"], kv_heads=1, dim=m["dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], scale=m["scale"])
            if mlp is not None and mlp["kind"] == "dense":
                spec.ffn = mlp["ff"]
            elif mlp is not None and mlp["kind"] == "moe":
                r, sh = mlp["router"], mlp.get("shared")
                spec.moe = MoeSpec(r["experts"], r["top"], r.get("scale", 1.0), ExpertSpec(mlp["expert"]["ff"], mlp["expert"]["limit"]),
                                   ExpertSpec(sh["ff"], sh["limit"]) if sh else None)
                if not 1 <= spec.moe.top <= spec.moe.experts:
                    raise ValueError(f"layer {i}: {spec.moe.top} of {spec.moe.experts} experts")
            elif mlp is not None:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(spec)
        emb, lp = cfg.get("embedding", {}), cfg.get("loop")
        bg = emb.get("bigram")
        if lp and not (0 <= lp["start"] < lp["stop"] <= len(layers) and lp["times"] >= 1):
            raise ValueError(f"loop over layers {lp['start']} .. {lp['stop']}, {lp['times']} times, of {len(layers)}")
        first = layers[0]
        return ModelConfig(architecture="rerupel", hidden_size=cfg["width"], num_layers=len(layers), num_heads=first.heads, num_kv_heads=1, head_dim=first.dim,
                           intermediate_size=max(s.ffn for s in layers), vocab_size=cfg["vocab"], rms_norm_eps=cfg["norm"]["eps"], max_position_embeddings=0,
                           tie_word_embeddings=True, layers=layers, embedding_scale=emb.get("scale", 1.0), residual_mult=cfg.get("residual_mult", 1.0),
                           logit_softcap=cfg.get("logit_softcap"), bigram=BigramSpec(bg["buckets"], bg["mul_prev"], bg["mul_cur"]) if bg else None,
                           loop=LoopSpec(lp["start"], lp["stop"], lp["times"]) if lp else None)

    @staticmethod
    def _from_parallel_layers(cfg: dict) -> "ModelConfig":
        def window(m):
            size = (m.get("mask") or {}).get("size") or 0
            if size < 0:
                raise ValueError(f"a window of {size} positions")
            return size

        def rotary(m, interleaved, dims=None):
            rot = m.get("rot") or {}
            spec = RotarySpec(rot.get("dims", 0) if dims is None else dims, rot.get("base", 10000.0), None, interleaved)
            if spec.dims % 2 or rot.get("dims", spec.dims) != spec.dims or (dims is None and spec.dims > m["dim"]):
                raise ValueError(f"rotary embedding of {rot.get('dims')} dimensions")
            return spec

        def mixer(kind, m):
            if kind == "latent_attention":
                return LayerSpec("latent_attention", m["heads"], 1, m["dim"], m["vdim"], scale=m["scale"], rot=rotary(m, True, m["rot_dim"]),
                                 kv_rank=m["kv_rank"], window=window(m))
            if kind != "parallel":
                raise ValueError(f"unknown mixer {kind!r}")
            a, b = m["left"], m["right"]
            if a["heads"] % a["kv_heads"]:
                raise ValueError(f"{a['heads']} query heads on {a['kv_heads']} key heads")
            left = LayerSpec("attention", a["heads"], a["kv_heads"], a["dim"], a["vdim"], scale=a["scale"], rot=rotary(a, False), window=window(a),
                             softcap=a.get("softcap") or 0.0)
            right = LayerSpec("gated_linear", b["heads"], 0, b["dim"], b["vdim"], tau=b["tau"])
            return LayerSpec("parallel", left.heads, left.kv_heads, left.dim, left.vdim, parts=[left, right],
                             part_scales=[m.get("left_scale", 1.0), m.get("right_scale", 1.0)])

        def feed_forward(spec, mlp):
            if mlp is None:
                return
            if mlp.get("kind", "dense") == "dense":
                spec.ffn = mlp["ff"]
                return
            if mlp["kind"] != "moe":
                raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
            r, sh, g = mlp["router"], mlp.get("shared"), mlp["router"].get("groups") or {}
            moe = spec.moe = MoeSpec(r["experts"], r["top"], 1.0, ExpertSpec(mlp["expert"]["ff"]), ExpertSpec(sh["ff"]) if sh else None,
                                     g.get("count") or 1, g.get("keep") or 1, r.get("identity") or 0)
            n = moe.experts + moe.identity
            if n % moe.groups or not 1 <= moe.keep <= moe.groups or not 1 <= moe.top <= n // moe.groups * moe.keep:
                raise ValueError(f"{moe.top} of {n} experts in {moe.groups} groups, {moe.keep} kept")

        layers = []
        for i, entry in enumerate(cfg["layers"]):
            try:
                spec = mixer(entry["type"], entry["mixer"])
                feed_forward(spec, entry.get("mlp"))
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
            layers.append(spec)
        first = layers[0]
        return ModelConfig(architecture="pilutar", hidden_size=cfg["width"], num_layers=len(layers), num_heads=first.heads, num_kv_heads=first.kv_heads,
                           head_dim=first.dim, intermediate_size=max(s.ffn for s in layers), vocab_size=cfg["vocab"], rms_norm_eps=cfg["norm"]["eps"],
                           max_position_embeddings=0, layers=layers, embedding_scale=cfg.get("embedding", {}).get("scale", 1.0),
                           logit_scale=cfg.get("logit_scale", 1.0))

    @staticmethod
    def _from_postnorm_layers(cfg: dict) -> "ModelConfig":
        def mixer(kind, m):
            if kind == "mamba1":
                return LayerSpec("mamba1", inner=m["inner"], state=m["state"], dt_rank=m["dt_rank"], conv_taps=m["conv"])
            if kind not in ("delta", "attention"):
                raise ValueError(f"unknown mixer {kind!r}")
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"{m['heads']} heads on {m['kv_heads']} key heads")
            if kind == "delta":
                return LayerSpec("delta", m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
            chunk = (m.get("mask") or {}).get("size") or 0
            if m["vdim"] != m["dim"] or chunk < 0:
                raise ValueError(f"values of size {m['vdim']} that are keys of size {m['dim']}" if chunk >= 0 else f"chunks of {chunk} positions")
            return LayerSpec("attention", m["heads"], m["kv_heads"], m["dim"], m["vdim"], scale=m["scale"], softcap=m.get("softcap") or 0.0, chunk=chunk)

        layers, norm = [], cfg["norm"]
        if cfg["width"] % norm["groups"]:
            raise ValueError(f"{cfg['width']} columns in {norm['groups']} groups")
        for i, entry in enumerate(cfg["layers"]):
            try:
                spec, mlp = mixer(entry["type"], entry["mixer"]), entry.get("mlp")
                if mlp is not None:
                    if mlp["kind"] != "moe":
                        raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
                    spec.moe = MoeSpec(mlp["router"]["experts"], mlp["router"]["top"], 1.0, ExpertSpec(mlp["expert"]["ff"]))
                    if not 1 <= spec.moe.top <= spec.moe.experts:
                        raise ValueError(f"{spec.moe.top} of {spec.moe.experts} experts")
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
            layers.append(spec)
        first = next((s for s in layers if s.mixer == "attention"), layers[0])
        return ModelConfig(architecture="noridra", hidden_size=cfg["width"], num_layers=len(layers), num_heads=first.heads, num_kv_heads=first.kv_heads,
                           head_dim=first.dim, intermediate_size=0, vocab_size=cfg["vocab"], rms_norm_eps=norm["eps"],
                           max_position_embeddings=cfg["max_positions"], layers=layers, residual_alpha=cfg["postln_alpha"], norm_groups=norm["groups"],
                           input_taps=cfg["canon"]["taps"])


# `architecture` values of configs that list their layers -> model class key
LAYERED_ARCHITECTURES = {"Rekudra": "rekudra", "Rerupel": "rerupel", "Pilutar": "pilutar", "Noridra": "noridra"}
# model classes that also run in f32 on CUDA (every operation has a true 32-bit kernel)
F32_ARCHITECTURES = ("rekudra", "rerupel", "pilutar", "noridra")


def tiny_llama() -> ModelConfig:
    """The CPU plumbing/numerics configuration: 2 layers, hidden 256, 4 q / 2 kv heads of 64, FFN 688,
    vocab 32000, tied embeddings."""
    return ModelConfig(hidden_size=256, num_layers=2, num_heads=4, num_kv_heads=2, head_dim=64, intermediate_size=688,
                       vocab_size=32000, rms_norm_eps=1e-5, rope_theta=500000.0, tie_word_embeddings=True,
                       max_position_embeddings=2048)


def llama31_8b() -> ModelConfig:
    return ModelConfig(hidden_size=4096, num_layers=32, num_heads=32, num_kv_heads=8, head_dim=128, intermediate_size=14336,
                       vocab_size=128256, rope_theta=500000.0, max_position_embeddings=8192,
                       rope_scaling={"rope_type": "llama3", "factor": 8.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0,
                                     "original_max_position_embeddings": 8192})


def llama33_70b_fp8() -> ModelConfig:
    return ModelConfig(hidden_size=8192, num_layers=80, num_heads=64, num_kv_heads=8, head_dim=128, intermediate_size=28672,
                       vocab_size=128256, rope_theta=500000.0, max_position_embeddings=8192, quantization="fp8_block",
                       rope_scaling={"rope_type": "llama3", "factor": 8.0, "low_freq_factor": 1.0, "high_freq_factor": 4.0,
                                     "original_max_position_embeddings": 8192})


def deepseek_v2_lite() -> ModelConfig:
    return ModelConfig(architecture="deepseek_v2", hidden_size=2048, num_layers=27, num_heads=16, num_kv_heads=16, head_dim=192,
                       intermediate_size=10944, vocab_size=102400, rms_norm_eps=1e-6, rope_theta=10000.0,
                       max_position_embeddings=4096, kv_lora_rank=512, qk_rope_head_dim=64, qk_nope_head_dim=128,
                       v_head_dim=128, n_routed_experts=64, n_shared_experts=2, num_experts_per_tok=6,
                       moe_intermediate_size=1408, first_k_dense_replace=1, routed_scaling_factor=1.0, norm_topk_prob=False,
                       rope_interleaved=True)


def tiny_deepseek() -> ModelConfig:
    """Small MLA + MoE model with the DeepSeek-V2-Lite head geometry, for tests."""
    return ModelConfig(architecture="deepseek_v2", hidden_size=256, num_layers=3, num_heads=16, num_kv_heads=16, head_dim=192,
                       intermediate_size=512, vocab_size=1024, rms_norm_eps=1e-6, rope_theta=10000.0,
                       max_position_embeddings=1024, kv_lora_rank=512, qk_rope_head_dim=64, qk_nope_head_dim=128,
                       v_head_dim=128, n_routed_experts=8, n_shared_experts=2, num_experts_per_tok=2,
                       moe_intermediate_size=128, first_k_dense_replace=1, rope_interleaved=True)


def rekudra(width: int, n_layers: int, heads: int, kv_heads: int, dim: int, ffn: int, vocab: int, streams: int = 4, taps: int = 4) -> ModelConfig:
    """A Rekudra decoder: pairs of a delta-rule layer and an attention layer with feed-forward; the second half of the
    attention layers shares the keys and values of the last one that has its own."""
    rot = RotarySpec(dim, 500000.0, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192})
    layers, own = [], None
    for i in range(n_layers // 2):
        layers.append(LayerSpec("channel_delta", heads, heads, dim, dim, taps, decay_rank=dim, gate_rank=dim))
        shared = own if i >= (n_layers // 2 + 1) // 2 and own is not None else None
        layers.append(LayerSpec("attention", heads, kv_heads, dim, dim, taps, scale=dim ** -0.5, rot=rot, kv_from=shared, ffn=ffn))
        if shared is None:
            own = len(layers) - 1
    return ModelConfig(architecture="rekudra", hidden_size=width, num_layers=len(layers), num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
                       intermediate_size=ffn, vocab_size=vocab, max_position_embeddings=0, layers=layers, residual_streams=streams,
                       embedding_scale=float(width) ** 0.5)


def rekudra_8b() -> ModelConfig:
    """Layers of the size of an 8B Llama's (width 4096, 32 heads of 128, FFN 14336)."""
    return rekudra(4096, 32, 32, 8, 128, 14336, 128256)


def rekudra_1b() -> ModelConfig:
    return rekudra(2048, 16, 16, 4, 128, 8192, 128256)


def tiny_rekudra() -> ModelConfig:
    return rekudra(256, 4, 4, 2, 64, 512, 1024, streams=2)


def rerupel(width: int, n_layers: int, heads: int, dim: int, kv_rank: int, ffn: int, vocab: int, experts: int, top: int, expert_ffn: int,
            shared_ffn: int, loop: tuple[int, int, int] | None = None) -> ModelConfig:
    """A Rerupel decoder: one layer with a dense feed-forward, then layers with experts; `loop` = (start, stop, times)."""
    moe = MoeSpec(experts, top, 1.0, ExpertSpec(expert_ffn, 7.0), ExpertSpec(shared_ffn, 7.0))
    layers = [LayerSpec("latent_attention", heads, 1, dim, dim, scale=dim ** -0.5, kv_rank=kv_rank, ffn=0 if i else ffn, moe=moe if i else None)
              for i in range(n_layers)]
    return ModelConfig(architecture="rerupel", hidden_size=width, num_layers=n_layers, num_heads=heads, num_kv_heads=1, head_dim=dim, intermediate_size=ffn,
                       vocab_size=vocab, rms_norm_eps=1e-6, max_position_embeddings=0, tie_word_embeddings=True, layers=layers,
                       embedding_scale=float(width) ** 0.5, logit_softcap=30.0, bigram=BigramSpec(16381, 10007, 31),
                       loop=LoopSpec(*loop) if loop else None)


def rerupel_lite() -> ModelConfig:
    """Layers of the size of DeepSeek-V2-Lite's; the upper half runs twice."""
    return rerupel(2048, 14, 16, 128, 512, 10944, 102400, 64, 6, 1408, 2816, (2, 14, 2))


def tiny_rerupel() -> ModelConfig:
    return rerupel(256, 3, 4, 64, 128, 512, 1024, 8, 2, 128, 192, (1, 3, 2))


def pilutar(width: int, n_layers: int, heads: int, kv_heads: int, dim: int, kv_rank: int, rot_dim: int, ffn: int, vocab: int, experts: int, top: int,
            expert_ffn: int, shared_ffn: int, window: int, groups: int = 1, keep: int = 1, identity: int = 0, latent_every: int = 4) -> ModelConfig:
    """A Pilutar decoder: windowed attention beside gated linear attention, every `latent_every`-th layer latent attention
    instead; one layer with a dense feed-forward, then layers with experts."""
    moe = MoeSpec(experts, top, 1.0, ExpertSpec(expert_ffn), ExpertSpec(shared_ffn), groups, keep, identity)
    layers = []
    for i in range(n_layers):
        if i % latent_every == latent_every - 1:
            s = LayerSpec("latent_attention", heads, 1, dim - rot_dim, dim, scale=dim ** -0.5, rot=RotarySpec(rot_dim, 50000.0, None, True), kv_rank=kv_rank,
                          window=window)
        else:
            left = LayerSpec("attention", heads, kv_heads, dim, dim, scale=dim ** -0.5, rot=RotarySpec(dim // 2, 10000.0), window=window, softcap=30.0)
            right = LayerSpec("gated_linear", heads, 0, dim, dim, tau=16.0, decay_rank=16)
            s = LayerSpec("parallel", heads, kv_heads, dim, dim, parts=[left, right], part_scales=[0.5, 0.5])
        s.ffn, s.moe = (ffn, None) if i == 0 else (0, moe)
        layers.append(s)
    return ModelConfig(architecture="pilutar", hidden_size=width, num_layers=n_layers, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
                       intermediate_size=ffn, vocab_size=vocab, max_position_embeddings=0, layers=layers, embedding_scale=float(width) ** 0.5)


def pilutar_lite() -> ModelConfig:
    """Layers of the size of DeepSeek-V2-Lite's."""
    return pilutar(2048, 24, 16, 4, 128, 512, 32, 10944, 102400, 62, 6, 1408, 2816, 1024, groups=8, keep=4, identity=2)


def tiny_pilutar() -> ModelConfig:
    return pilutar(256, 4, 4, 2, 64, 128, 32, 512, 1024, 7, 2, 128, 192, 48, groups=2, identity=1)


def noridra(width: int, n_layers: int, heads: int, kv_heads: int, dim: int, vocab: int, experts: int, top: int, expert_ffn: int, chunk: int,
            state: int = 16, groups: int = 4, taps: int = 4, positions: int = 8192) -> ModelConfig:
    """A Noridra decoder: in every four layers two with the gated delta rule, one with attention inside chunks, one selective
    scan over twice the width; experts in all of them."""
    moe = MoeSpec(experts, top, 1.0, ExpertSpec(expert_ffn))
    kinds = {"delta": lambda: LayerSpec("delta", heads, heads, dim, dim, taps),
             "mamba1": lambda: LayerSpec("mamba1", inner=2 * width, state=state, dt_rank=width // 16, conv_taps=taps),
             "attention": lambda: LayerSpec("attention", heads, kv_heads, dim, dim, scale=dim ** -0.5, softcap=30.0, chunk=chunk)}
    layers = [kinds[("delta", "mamba1", "delta", "attention")[i % 4]]() for i in range(n_layers)]
    for s in layers:
        s.moe = moe
    return ModelConfig(architecture="noridra", hidden_size=width, num_layers=n_layers, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
                       intermediate_size=0, vocab_size=vocab, rms_norm_eps=1e-6, max_position_embeddings=positions, layers=layers,
                       residual_alpha=(2.0 * n_layers) ** 0.25, norm_groups=groups, input_taps=taps)


def noridra_lite() -> ModelConfig:
    """Layers of the size of DeepSeek-V2-Lite's."""
    return noridra(2048, 24, 16, 4, 128, 102400, 64, 6, 1408, 1024)


def tiny_noridra() -> ModelConfig:
    return noridra(192, 4, 3, 1, 64, 1024, 6, 2, 112, 48, state=8, groups=3, taps=3, positions=1024)


PRESETS = {
    "tiny-llama": tiny_llama,
    "llama-3.1-8b": llama31_8b,
    "llama-3.3-70b-fp8": llama33_70b_fp8,
    "deepseek-v2-lite": deepseek_v2_lite,
    "tiny-deepseek": tiny_deepseek,
    "rekudra-8b": rekudra_8b,
    "rekudra-1b": rekudra_1b,
    "tiny-rekudra": tiny_rekudra,
    "rerupel-lite": rerupel_lite,
    "tiny-rerupel": tiny_rerupel,
    "pilutar-lite": pilutar_lite,
    "tiny-pilutar": tiny_pilutar,
    "noridra-lite": noridra_lite,
    "tiny-noridra": tiny_noridra,
}


def get_config(name_or_path: str) -> ModelConfig:
    key = name_or_path.lower()
    if key in PRESETS:
        return PRESETS[key]()
    p = Path(name_or_path)
    if (p / "config.json").exists():
        return ModelConfig.from_hf(p)
    raise ValueError(f"unknown model {name_or_path!r}; presets: {sorted(PRESETS)}")
