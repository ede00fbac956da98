"""Architecture descriptions. Field names follow the Hugging Face `config.json` keys so a checkpoint directory
can be read directly; named presets cover the architectures the engine is benchmarked on."""
from __future__ import annotations

import json
from dataclasses import dataclass, field, asdict
from pathlib import Path


@dataclass
class RotarySpec:
    """Rotary embedding of one layer: the first `dims` dimensions of a head turn, the rest pass. `scaling` is the Llama-3.1
    frequency rescale (factor, low, high, original) or None."""
    dims: int = 0
    base: float = 10000.0
    scaling: dict | None = None


@dataclass
class LayerSpec:
    """One layer of a decoder whose layers differ: which mixer it has, the mixer's sizes, and its feed-forward width."""
    mixer: str = "attention"               # "attention" | "channel_delta"
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


@dataclass
class ModelConfig:
    architecture: str = "llama"            # "llama" | "deepseek_v2" | "rekudra"
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
    extra: dict = field(default_factory=dict)

    def to_dict(self) -> dict:
        return asdict(self)

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0

    @property
    def is_moe(self) -> bool:
        return self.n_routed_experts > 0

    def kv_bytes_per_token(self, dtype_bytes: int = 2, tp: int = 1) -> int:
        if self.layers is not None:
            return sum(s.kv_heads * (s.dim + s.vdim) for s in self.layers if s.mixer == "attention" and s.kv_from is None) * dtype_bytes
        if self.is_mla:
            return self.num_layers * (self.kv_lora_rank + self.qk_rope_head_dim) * dtype_bytes
        return self.num_layers * 2 * max(1, self.num_kv_heads // tp) * self.head_dim * dtype_bytes

    def num_params(self) -> int:
        h = self.hidden_size
        emb = self.vocab_size * h * (1 if self.tie_word_embeddings else 2)
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


# `architecture` values of configs that list their layers -> model class key
LAYERED_ARCHITECTURES = {"Rekudra": "rekudra"}


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


PRESETS = {
    "tiny-llama": tiny_llama,
    "llama-3.1-8b": llama31_8b,
    "llama-3.3-70b-fp8": llama33_70b_fp8,
    "deepseek-v2-lite": deepseek_v2_lite,
    "tiny-deepseek": tiny_deepseek,
    "rekudra-8b": rekudra_8b,
    "rekudra-1b": rekudra_1b,
    "tiny-rekudra": tiny_rekudra,
}


def get_config(name_or_path: str) -> ModelConfig:
    key = name_or_path.lower()
    if key in PRESETS:
        return PRESETS[key]()
    p = Path(name_or_path)
    if (p / "config.json").exists():
        return ModelConfig.from_hf(p)
    raise ValueError(f"unknown model {name_or_path!r}; presets: {sorted(PRESETS)}")
