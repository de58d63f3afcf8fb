"""Model shape + precision description, parsed from a HF ``config.json`` or built from a preset.

Covers the architectures the engine serves: dense GQA decoders (Llama / Qwen3 style),
hybrid gated-delta-net + gated-attention MoE (Qwen3.5 / 3.6 style), Nemotron-H hybrids
(Mamba2 + attention + squared-ReLU MLP / MoE) and DeepSeek-V3 style MLA MoE.
Role of the reference's ``crates/config`` (``ModelConfig`` and the per-family parsers in
``crates/config/src/parsers/``) and of ``kernels/circuits/*.config.toml``: unknown
``model_type`` values are refused rather than guessed.
"""
from __future__ import annotations

import json
import math
from dataclasses import asdict, dataclass, field, replace
from pathlib import Path
from typing import List, Optional

WEIGHT_FORMATS = ("bf16", "nvfp4", "fp8_block", "fp8_row", "fp32")
KV_DTYPES = ("bf16", "fp8", "fp32")
LAYER_KINDS = ("attention", "gdn", "mamba2", "mla", "kda", "parallel", "lightning", "latent", "gla", "gated", "twin",
               "delta")
KV_KINDS = ("attention", "mla", "parallel", "latent", "gated", "twin")   # kinds that own a KV pool
STATE_KINDS = ("gdn", "mamba2", "kda", "parallel", "lightning", "gla", "twin", "delta")   # kinds that own a recurrent state
FFN_KINDS = ("dense", "moe", "none")


@dataclass
class ModelConfig:
    name: str = "model"
    arch: str = "dense_gqa"            # dense_gqa | qwen_hybrid | nemotron_h | deepseek_mla | fabulix | finelix | pivipel | ledinex
    vocab_size: int = 4096
    hidden_size: int = 256
    num_layers: int = 2
    # attention
    num_heads: int = 4
    num_kv_heads: int = 2
    head_dim: int = 64
    rope_theta: float = 1e6
    rope_scaling: Optional[dict] = None     # HF `rope_scaling` (linear / llama3 / yarn); None = plain RoPE
    rotary_dim: int = 0                 # 0 -> head_dim; -1 -> no RoPE (Nemotron-H attention)
    rope_identity: bool = False         # keep the rotary slots of the layout but rotate by nothing (Kimi-Linear's NoPE MLA layers)
    qk_norm: bool = False
    qk_norm_full: bool = False          # the q / k RMSNorm spans all heads of the projection (MiniMax-M2), not one head
    attn_output_gate: bool = False      # q_proj emits [Q_h | G_h] per head, o = attn * sigmoid(G)
    sliding_window: int = 0
    attn_scale: float = 0.0             # softmax scale; 0 -> head_dim ** -0.5 (Gemma: query_pre_attn_scalar ** -0.5)
    window_layers: List[int] = field(default_factory=list)   # per-layer window (0 = full); empty -> sliding_window everywhere
    rope_local_theta: float = 0.0       # RoPE base of the windowed layers when it differs (Gemma 3); 0 = rope_theta
    attn_bias: bool = False             # q / k / v projections carry a bias (Qwen2 family)
    # norms
    rms_eps: float = 1e-6
    norm_plus_one: bool = False         # (1 + w) scaling (Qwen3.5 family)
    # ffn
    intermediate_size: int = 688
    ffn_act: str = "swiglu"             # swiglu | relu2 | geglu (tanh-approximated GELU gate)
    post_norms: bool = False            # Gemma / GLM-4: RMSNorm on the attention / FFN output before the residual add
    post_norm_names: str = "gemma"      # checkpoint spelling of the norms: gemma | glm | olmo2
    pre_norms: bool = True              # False: blocks read the residual stream un-normalised (OLMo 2: post-norm only)
    rope_interleaved: bool = False      # checkpoint rotates (2i, 2i+1) pairs; q / k rows are re-ordered at load
    embed_scale: float = 1.0            # embeddings are multiplied by this (Gemma: sqrt(hidden))
    final_logit_softcap: float = 0.0    # logits = cap * tanh(logits / cap); 0 = off
    residual_multiplier: float = 1.0    # Granite: a block's output is scaled by this before it joins the stream
    logits_divisor: float = 1.0         # Granite: logits are divided by this
    tie_embeddings: bool = False
    # fabulix, finelix, pivipel, ledinex: per-layer mixer and feed-forward sizes and constants, [{"mixer": {...}, "mlp": {...} | None}, ...]
    layer_specs: List[dict] = field(default_factory=list)
    spec_types: List[str] = field(default_factory=list)      # pivipel, ledinex: the layers' own type names (variants of one layer kind)
    weights_of: List[int] = field(default_factory=list)      # per layer: the layer whose tensors it uses, -1 = its own; empty = all their own
    streams: int = 0                    # static hyper-connections: the residual is this many fp32 copies (0 = a single residual)
    canon_taps: int = 0                 # every sublayer reads the stream through a causal convolution of this many taps (0 = as it is)
    logit_scale: float = 1.0            # logits are multiplied by this (folded into the final norm at load)
    loop: Optional[dict] = None         # layers start .. stop - 1 run `times` times with the same weights: {"start", "stop", "times"}
    token_side_dim: int = 0             # width of a layer's slice of the token side embedding (0 = none)
    glu_alpha: float = 1.702            # sigmoid slope of the clamped GLU
    # per-layer structure
    layer_types: List[str] = field(default_factory=list)   # mixer per layer
    ffn_types: List[str] = field(default_factory=list)     # ffn per layer
    # gated delta net
    gdn_k_heads: int = 0
    gdn_v_heads: int = 0
    gdn_k_dim: int = 128
    gdn_v_dim: int = 128
    conv_kernel: int = 4
    # vision input (Qwen-VL family): the tower's configuration, the placeholder token and the rotary sections
    vision: Optional[dict] = None       # HF vision_config of the checkpoint (vision.VisionConfig.from_hf)
    image_token_id: int = -1
    vision_start_token_id: int = -1
    mrope_sections: Optional[List[int]] = None      # rotary frequencies per (time, height, width) axis
    # hyper-connections: the residual stream is hc_mult fp32 copies mixed in and out of every block
    hc_mult: int = 0                    # 0 / 1 = a single residual stream
    hc_sinkhorn_iters: int = 20
    hc_eps: float = 1e-6
    # sparse attention over MLA (DeepSeek sparse attention): a light indexer picks index_topk tokens per query
    index_topk: int = 0                 # 0 = dense attention
    index_n_heads: int = 64
    index_head_dim: int = 128
    # Kimi delta attention (per-channel gated delta rule)
    kda_heads: int = 0
    kda_head_dim: int = 128
    kda_gate_rank: int = 0              # inner width of the low-rank decay (f_a / f_b) and output-gate (g_a / g_b) projections; 0 = head_dim
    kda_gate_lower_bound: float = -5.0
    # mamba2
    mamba_heads: int = 0
    mamba_head_dim: int = 64
    mamba_state: int = 128
    mamba_groups: int = 8
    mamba_conv_bias: bool = True
    # moe
    num_experts: int = 0
    experts_per_token: int = 0
    moe_intermediate_size: int = 0
    num_shared_experts: int = 0
    shared_expert_gate: bool = False
    shared_expert_name: str = ""        # "" = by architecture ("shared_expert" for the Qwen families)
    router: str = "softmax"             # softmax | sigmoid
    router_n_group: int = 1
    router_topk_group: int = 1
    router_scaling: float = 1.0
    router_renormalize: bool = True
    first_dense_layers: int = 0
    dense_intermediate_size: int = 0    # FFN width of the leading dense layers (DeepSeek)
    # MLA
    q_lora_rank: int = 0
    kv_lora_rank: int = 0
    qk_nope_dim: int = 0
    qk_rope_dim: int = 0
    v_head_dim: int = 0
    # speculative
    mtp_layers: int = 0
    # precision
    weight_format: str = "bf16"
    kv_dtype: str = "bf16"
    kv_high_precision_layers: tuple = ()    # model layers whose KV stays bf16 when kv_dtype is fp8
    max_position: int = 32768

    def __post_init__(self):
        if not self.layer_types:
            self.layer_types = ["attention"] * self.num_layers
        if not self.ffn_types:
            self.ffn_types = ["dense"] * self.num_layers
        if self.rotary_dim == 0:
            self.rotary_dim = self.head_dim if self.arch != "deepseek_mla" else self.qk_rope_dim
        assert len(self.layer_types) == self.num_layers, "layer_types length"
        assert len(self.ffn_types) == self.num_layers, "ffn_types length"
        assert all(t in LAYER_KINDS for t in self.layer_types)
        assert all(t in FFN_KINDS for t in self.ffn_types)
        assert self.weight_format in WEIGHT_FORMATS and self.kv_dtype in KV_DTYPES

    # ---- derived sizes
    @property
    def q_size(self) -> int:
        return self.num_heads * self.head_dim * (2 if self.attn_output_gate else 1)

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    @property
    def gdn_qk_size(self) -> int:
        return self.gdn_k_heads * self.gdn_k_dim

    @property
    def gdn_v_size(self) -> int:
        return self.gdn_v_heads * self.gdn_v_dim

    @property
    def mamba_inner(self) -> int:
        return self.mamba_heads * self.mamba_head_dim

    @property
    def mamba_conv_dim(self) -> int:
        return self.mamba_inner + 2 * self.mamba_groups * self.mamba_state

    def attention_layers(self) -> List[int]:
        return [i for i, t in enumerate(self.layer_types) if t in KV_KINDS]

    @property
    def stream32(self) -> bool:
        """The residual stream is kept in 32-bit, and the layers' sizes are per layer (``layer_specs``)."""
        return self.arch in ("fabulix", "finelix", "pivipel", "ledinex")

    def layer_owner(self, i: int) -> int:
        """The layer whose tensors layer i uses (its cache or state is its own all the same)."""
        while self.weights_of and self.weights_of[i] >= 0:
            i = self.weights_of[i]
        return i

    def layer_runs(self) -> List[tuple]:
        """(layer, pass) of every layer run in order. A looped layer appears once per pass, and each of its runs
        has a cache or state of its own; `pass` is given on the first run of a pass only, else None."""
        lo, hi, times = (self.loop["start"], self.loop["stop"], self.loop["times"]) if self.loop else (0, 0, 0)
        if times == 0:
            return [(i, None) for i in range(self.num_layers)]
        return ([(i, None) for i in range(lo)]
                + [(i, t if i == lo else None) for t in range(times) for i in range(lo, hi)]
                + [(i, None) for i in range(hi, self.num_layers)])

    @property
    def act_fmt(self) -> str:
        """Activation type of models with a 32-bit residual stream: bf16, or fp32 when served in 32-bit."""
        return "fp32" if self.weight_format == "fp32" else "bf16"

    def kv_layer_dims(self) -> List[tuple]:
        """(kv heads, K row, V row) of every KV pool (one per layer run) of a model whose layers have their own head
        sizes; the rows are padded to what the attention kernels tile. Latent layers cache one row per token
        that serves as key and value."""
        from ..ops.latent import latent_row
        from ..ops.mixers import padded_head_dims
        out = []
        for i, _ in self.layer_runs() if self.layer_specs else ():
            t, m = self.layer_types[i], self.layer_specs[i]["mixer"]
            if t == "parallel":
                m = m["left"]
                out.append((m["kv_heads"], *padded_head_dims(m["dim"], m["vdim"], self.act_fmt)))
            elif t == "gated":
                out.append((m["kv_heads"], *padded_head_dims(m["dim"], m["vdim"], self.act_fmt)))
            elif t == "twin":
                m = m["left"]
                out.append((m["kv_heads"], *padded_head_dims(m["dim"], m.get("vdim", m["dim"]), self.act_fmt)))
            elif t == "latent":
                out.append((1, latent_row(m["kv_rank"], m["rot_dim"], self.act_fmt).row, 0))
        return out

    def kv_bytes_per_token(self) -> int:
        e = 1 if self.kv_dtype == "fp8" else 2
        n = 0
        for t in self.layer_types:
            if t == "attention":
                n += 2 * self.num_kv_heads * self.head_dim * e
            elif t == "mla":
                n += (self.kv_lora_rank + self.qk_rope_dim) * e
        n += sum(h * (dk + dv) * (4 if self.kv_dtype == "fp32" else 2) for h, dk, dv in self.kv_layer_dims())
        return n + self.mtp_layers * 2 * self.num_kv_heads * self.head_dim * e * (self.arch != "deepseek_mla")

    def param_count(self) -> int:
        """Approximate parameter count (linear layers + embeddings)."""
        h = self.hidden_size
        if self.stream32:
            from ..weights.source import spec_shapes
            return sum(math.prod(s) for s, _ in spec_shapes(self).values())
        n = self.vocab_size * h * (1 if self.tie_embeddings else 2)
        for lt, ft in zip(self.layer_types, self.ffn_types):
            if lt == "attention":
                n += h * (self.q_size + 2 * self.kv_size) + self.num_heads * self.head_dim * h
            elif lt == "gdn":
                n += h * (2 * self.gdn_qk_size + 2 * self.gdn_v_size + 2 * self.gdn_v_heads) + self.gdn_v_size * h
            elif lt == "kda":
                hd, r = self.kda_heads * self.kda_head_dim, self.kda_gate_rank or self.kda_head_dim
                n += 4 * h * hd + 2 * (h * r + r * hd) + h * self.kda_heads
            elif lt == "mamba2":
                n += h * (2 * self.mamba_inner + 2 * self.mamba_groups * self.mamba_state + self.mamba_heads)
                n += self.mamba_inner * h
            elif lt == "mla":
                qh = self.qk_nope_dim + self.qk_rope_dim
                n += h * self.q_lora_rank + self.q_lora_rank * self.num_heads * qh
                n += h * (self.kv_lora_rank + self.qk_rope_dim)
                n += self.kv_lora_rank * self.num_heads * (self.qk_nope_dim + self.v_head_dim)
                n += self.num_heads * self.v_head_dim * h
            mult = 3 if self.ffn_act == "swiglu" else 2
            if ft == "dense":
                n += mult * h * (self.dense_intermediate_size or self.intermediate_size)
            elif ft == "moe":
                n += self.num_experts * mult * h * self.moe_intermediate_size + h * self.num_experts
                n += self.num_shared_experts * mult * h * self.moe_intermediate_size
        return n

    def to_json(self) -> str:
        return json.dumps(asdict(self), indent=1)

    @staticmethod
    def from_json(s: str) -> "ModelConfig":
        return ModelConfig(**json.loads(s))

    def scaled(self, **kw) -> "ModelConfig":
        return replace(self, **kw)


# ----------------------------------------------------------------------------- presets
def tiny_dense(**kw) -> ModelConfig:
    """Tiny dense Qwen3-style decoder that runs on CPU in fp32-equivalent precision: 2 layers,
    hidden 256, 4 q / 2 kv heads of 64, SwiGLU 688, vocab 4096, tied embeddings."""
    base = dict(name="tiny-dense", arch="dense_gqa", vocab_size=4096, hidden_size=256, num_layers=2,
                num_heads=4, num_kv_heads=2, head_dim=64, rope_theta=1e6, intermediate_size=688,
                tie_embeddings=True, rms_eps=1e-6, qk_norm=True, max_position=2048)
    base.update(kw)
    return ModelConfig(**base)


def dense_27b_nvfp4(**kw) -> ModelConfig:
    """Dense ~27B decoder: 64 layers, hidden 5120, 40 q / 8 kv heads of 128, SwiGLU 17408,
    vocab 151936, NVFP4 weights (bf16 embeddings and lm_head), fp8 KV, one MTP layer."""
    base = dict(name="dense-27b-nvfp4", arch="dense_gqa", vocab_size=151936, hidden_size=5120,
                num_layers=64, num_heads=40, num_kv_heads=8, head_dim=128, rope_theta=1e6,
                intermediate_size=17408, tie_embeddings=False, qk_norm=True, mtp_layers=1,
                weight_format="nvfp4", kv_dtype="fp8", max_position=32768)
    base.update(kw)
    return ModelConfig(**base)


def qwen_hybrid_moe_35b(**kw) -> ModelConfig:
    """Hybrid GDN + gated attention MoE, ~35B total / ~3B active, FP8 128x128 block weights:
    40 layers in a 3:1 pattern, hidden 2048, GDN 16 value heads x 128 (16 key heads), conv 4;
    attention 16 q / 2 kv heads of 256 with an output gate; 256 experts top-8 softmax + 1 shared
    expert with a sigmoid gate, expert FFN 512."""
    L = kw.pop("num_layers", 40)
    base = dict(name="qwen-hybrid-moe-35b-fp8", arch="qwen_hybrid", vocab_size=151936, hidden_size=2048,
                num_layers=L, num_heads=16, num_kv_heads=2, head_dim=256, rotary_dim=64, rope_theta=1e7,
                qk_norm=True, attn_output_gate=True, norm_plus_one=True,
                layer_types=[("attention" if (i + 1) % 4 == 0 else "gdn") for i in range(L)],
                ffn_types=["moe"] * L, gdn_k_heads=16, gdn_v_heads=16, gdn_k_dim=128, gdn_v_dim=128,
                conv_kernel=4, num_experts=256, experts_per_token=8, moe_intermediate_size=512,
                num_shared_experts=1, shared_expert_gate=True, router="softmax", mtp_layers=0,
                weight_format="fp8_block", kv_dtype="bf16", intermediate_size=512)
    base.update(kw)
    return ModelConfig(**base)


def nemotron_h_8b(**kw) -> ModelConfig:
    """Nemotron-H style hybrid, ~8B, FP8 per-row weights: 52 layers, each one mixer *or* one MLP
    (24 Mamba2 mixers with 128 heads x 64, state 128, 8 groups, conv 4; 4 attention layers with
    32 q / 8 kv heads of 128, no RoPE; 24 squared-ReLU MLPs of 21504), hidden 4096, vocab 131072."""
    # 52 blocks = 28 mixers (24 Mamba2 + 4 attention) + 24 MLPs. A layer here is one mixer plus
    # the MLP block that follows it, if any; the Mamba2 mixer right before each attention
    # block has none ("...M*-..." in the block pattern).
    n_mix = kw.pop("num_layers", 28)
    attn_at = {4 + 6 * j for j in range(4)} if n_mix == 28 else {n_mix // 2}
    layer_types = ["attention" if i in attn_at else "mamba2" for i in range(n_mix)]
    ffn_types = ["none" if (i + 1) in attn_at else "dense" for i in range(n_mix)]
    base = dict(name="nemotron-h-8b-fp8", arch="nemotron_h", vocab_size=131072, hidden_size=4096,
                num_layers=len(layer_types), num_heads=32, num_kv_heads=8, head_dim=128, rotary_dim=-1,
                layer_types=layer_types, ffn_types=ffn_types, intermediate_size=21504, ffn_act="relu2",
                mamba_heads=128, mamba_head_dim=64, mamba_state=128, mamba_groups=8, conv_kernel=4,
                weight_format="fp8_row", kv_dtype="bf16", rms_eps=1e-5, max_position=16384)
    base.update(kw)
    return ModelConfig(**base)


def deepseek_v3_671b(**kw) -> ModelConfig:
    """DeepSeek-V3 shaped MLA MoE: 61 layers (first 3 dense, FFN 18432), hidden 7168, MLA 128
    heads (q_lora 1536, kv_lora 512, nope 128, rope 64, v 128), 256 routed experts top-8 with a
    sigmoid group-limited router (8 groups, top-4) + 1 shared expert, expert FFN 2048,
    vocab 129280, one MTP layer, FP8 128x128 block weights."""
    L = kw.pop("num_layers", 61)
    fd = kw.pop("first_dense_layers", 3)
    base = dict(name="deepseek-v3-671b-fp8", arch="deepseek_mla", vocab_size=129280, hidden_size=7168,
                num_layers=L, num_heads=128, num_kv_heads=128, head_dim=192, rope_theta=10000.0,
                layer_types=["mla"] * L, ffn_types=["dense"] * fd + ["moe"] * (L - fd),
                first_dense_layers=fd, dense_intermediate_size=18432, intermediate_size=18432,
                q_lora_rank=1536, kv_lora_rank=512, qk_nope_dim=128, qk_rope_dim=64, v_head_dim=128,
                num_experts=256, experts_per_token=8, moe_intermediate_size=2048, num_shared_experts=1,
                router="sigmoid", router_n_group=8, router_topk_group=4, router_scaling=2.5,
                mtp_layers=1, weight_format="fp8_block", kv_dtype="bf16", max_position=16384)
    base.update(kw)
    return ModelConfig(**base)


def tiny_hybrid_moe(**kw) -> ModelConfig:
    """Four-layer instance of the hybrid GDN + gated-attention MoE family (tests, smoke runs)."""
    base = dict(num_layers=4, hidden_size=512, num_heads=4, num_kv_heads=2, gdn_k_heads=4, gdn_v_heads=4,
                num_experts=8, experts_per_token=2, moe_intermediate_size=256, intermediate_size=256,
                vocab_size=4096, max_position=1024, name="tiny-hybrid-moe")
    base.update(kw)
    return qwen_hybrid_moe_35b(**base)


def tiny_nemotron_h(**kw) -> ModelConfig:
    """Four-mixer instance of the Mamba2 + attention hybrid family (tests, smoke runs)."""
    base = dict(num_layers=4, hidden_size=512, num_heads=8, num_kv_heads=2, intermediate_size=1024,
                mamba_heads=16, mamba_groups=2, vocab_size=4096, max_position=1024, name="tiny-nemotron-h")
    base.update(kw)
    return nemotron_h_8b(**base)


def tiny_dense_hc(**kw) -> ModelConfig:
    """The tiny dense model with a four-stream hyper-connection highway (tests, smoke runs)."""
    base = dict(hc_mult=4, hc_sinkhorn_iters=4, name="tiny-dense-hc")
    base.update(kw)
    return tiny_dense(**base)


def tiny_kimi_linear(**kw) -> ModelConfig:
    """Four-layer instance of the Kimi-Linear family: three Kimi-delta-attention layers per full-attention
    layer, MoE feed-forward (tests, smoke runs)."""
    base = dict(num_layers=4, hidden_size=512, num_heads=4, num_kv_heads=2, gdn_k_heads=0, gdn_v_heads=0,
                kda_heads=4, kda_head_dim=128, kda_gate_rank=64,
                layer_types=["kda", "kda", "kda", "attention"],
                num_experts=8, experts_per_token=2, moe_intermediate_size=256, intermediate_size=256,
                vocab_size=4096, max_position=1024, name="tiny-kimi-linear")
    base.update(kw)
    return qwen_hybrid_moe_35b(**base)


def fabulix(num_layers: int = 4, width: int = 256, heads: int = 4, kv_heads: int = 2, dim: int = 64, vdim: int = 64, rot_dims: int = 32,
            rot_base: float = 10000.0, right_heads: int = 4, right_dim: int = 64, lin_heads: int = 4, lin_dim: int = 64, lin_vdim: int = 64,
            ff: int = 512, limit: float = 3.0, side_dim: int = 16, vocab: int = 1024, period: int = 3, eps: float = 1e-5, **kw) -> ModelConfig:
    """Fabulix decoder of uniform layers: every `period`-th layer is a lightning mixer, the others run sink
    attention and RWKV-style time mixing side by side; clamped-GLU feed-forward, Dynamic-Tanh norms before
    and after every sublayer, a token side input per layer, tied embeddings."""
    layers = []
    for i in range(num_layers):
        if i % period == period - 1:
            m = {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim,
                 "decay": [1.0 - 2.0 ** -(1.0 + 6.0 * (h + 1) / lin_heads) for h in range(lin_heads)]}
            layers.append({"type": "lightning", "mixer": m, "mlp": {"kind": "dense", "ff": ff, "limit": limit}})
        else:
            left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5,
                    "rot": {"base": rot_base, "dims": rot_dims}}
            layers.append({"type": "parallel", "mlp": {"kind": "dense", "ff": ff, "limit": limit},
                           "mixer": {"left": left, "right": {"heads": right_heads, "dim": right_dim},
                                     "left_scale": 0.7, "right_scale": 0.7}})
    cfg = {"architecture": "Fabulix", "vocab": vocab, "width": width, "embedding": {"scale": float(width) ** 0.5},
           "norm": {"eps": eps}, "layers": layers}
    if side_dim:
        cfg["token_side"] = {"dim": side_dim}
    return from_fabulix_config(cfg, name=kw.pop("name", "fabulix")).scaled(**kw)


def tiny_fabulix(**kw) -> ModelConfig:
    """Four-layer Fabulix (tests, smoke runs)."""
    return fabulix(**{"name": "tiny-fabulix", **kw})


def fabulix_3b(**kw) -> ModelConfig:
    """Fabulix with the layer sizes of a ~3B model: width 2560, 20 query / 4 key-value heads of 128, 20
    time-mixing heads of 128, lightning layers of 20 heads of 128, feed-forward 6912, 24 layers."""
    base = dict(name="fabulix-3b", num_layers=24, width=2560, heads=20, kv_heads=4, dim=128, vdim=128, rot_dims=128, right_heads=20,
                right_dim=128, lin_heads=20, lin_dim=128, lin_vdim=128, ff=6912, side_dim=128, vocab=65536)
    base.update(kw)
    return fabulix(**base)


def finelix(num_layers: int = 6, width: int = 256, heads: int = 4, dim: int = 48, rot_dim: int = 16, vdim: int = 40, kv_rank: int = 96,
            q_rank: int = 80, rot_base: float = 10000.0, lin_heads: int = 4, lin_dim: int = 64, lin_vdim: int = 64, tau: float = 16.0,
            ff: int = 512, experts: int = 8, top: int = 2, expert_ff: int = 96, shared_ff: int = 160, vocab: int = 1024, period: int = 2,
            loop: Optional[dict] = None, eps: float = 1e-5, **kw) -> ModelConfig:
    """Finelix decoder of uniform layers: every `period`-th layer is latent attention beside a mixture of
    experts, the others gated linear attention beside a dense feed-forward; `loop` repeats a range of layers."""
    layers = []
    for i in range(num_layers):
        if i % period == period - 1:
            m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                 "scale": (dim + rot_dim) ** -0.5, "rot": {"base": rot_base, "dims": rot_dim}}
            mlp = {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top}}
            if shared_ff:
                mlp["shared"] = {"ff": shared_ff}
            layers.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
        else:
            m = {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim, "tau": tau}
            layers.append({"type": "gla", "mixer": m, "mlp": {"kind": "dense", "ff": ff}})
    cfg = {"architecture": "Finelix", "vocab": vocab, "width": width, "embedding": {"scale": float(width) ** 0.5},
           "norm": {"eps": eps}, "layers": layers}
    if loop:
        cfg["loop"] = dict(loop)
    return from_finelix_config(cfg, name=kw.pop("name", "finelix")).scaled(**kw)


def tiny_finelix(**kw) -> ModelConfig:
    """Six-layer Finelix with a looped range (tests, smoke runs)."""
    return finelix(**{"name": "tiny-finelix", "loop": {"start": 1, "stop": 3, "times": 2}, **kw})


def finelix_3b(**kw) -> ModelConfig:
    """Finelix with the layer sizes of a ~3B-active model: width 2560, latent attention of 32 heads (128 + 64, value
    128, latent 512, query latent 1536) beside 64 experts of 1024, top 6, and a shared one; gated linear attention
    of 20 heads of 128 beside a feed-forward of 6912; 24 layers, two of them run three times."""
    base = dict(name="finelix-3b", num_layers=24, width=2560, heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=1536,
                lin_heads=20, lin_dim=128, lin_vdim=128, ff=6912, experts=64, top=6, expert_ff=1024, shared_ff=2048, vocab=65536,
                loop={"start": 2, "stop": 4, "times": 3})
    base.update(kw)
    return finelix(**base)


def pivipel(num_layers: int = 4, width: int = 192, heads: int = 4, kv_heads: int = 2, dim: int = 64, vdim: int = 64, rot_dims: int = 32,
            rot_base: float = 10000.0, window: int = 24, keep: int = 3, ff: int = 512, limit: float = 2.5, experts: int = 8, top: int = 2,
            expert_ff: int = 80, shared_ff: int = 160, groups: int = 4, keep_groups: int = 2, streams: int = 2, vocab: int = 1024,
            positions: int = 4096, period: int = 2, dense_layers: int = 1, share: bool = False, eps: float = 1e-5, **kw) -> ModelConfig:
    """Pivipel decoder of uniform layers: every `period`-th layer has normed attention without positions and a window
    beside kept first tokens, the others rotated sink attention in a plain window; dense feed-forwards in the first
    `dense_layers`, mixtures of experts behind them; `share`: the last layer uses the tensors of the one `period` before."""
    layers = []
    for i in range(num_layers):
        m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5, "mask": {"size": window}}
        t = "attention_2" if i % period == period - 1 else "attention"
        if t == "attention":
            m["rot"] = {"base": rot_base, "dims": rot_dims, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 2048}}
        else:
            m["mask"]["keep_first"] = keep
        mlp = {"kind": "dense", "ff": ff, "limit": limit}
        if i >= dense_layers:
            mlp = {"kind": "moe", "expert": {"ff": expert_ff, "limit": limit},
                   "router": {"experts": experts, "top": top, "scale": 1.25, "groups": {"count": groups, "keep": keep_groups}}}
            if shared_ff:
                mlp["shared"] = {"ff": shared_ff, "limit": limit}
        layers.append({"type": t, "mixer": m, "mlp": mlp})
    if share:
        layers[-1]["weights_of"] = num_layers - 1 - period
    cfg = {"architecture": "Pivipel", "vocab": vocab, "width": width, "streams": streams, "max_positions": positions, "norm": {"eps": eps},
           "layers": layers}
    return from_pivipel_config(cfg, name=kw.pop("name", "pivipel")).scaled(**kw)


def tiny_pivipel(**kw) -> ModelConfig:
    """Four-layer Pivipel whose last layer shares its tensors (tests, smoke runs)."""
    return pivipel(**{"name": "tiny-pivipel", "share": True, **kw})


def pivipel_3b(**kw) -> ModelConfig:
    """Pivipel with the layer sizes of a ~3B-active model: width 2560, 32 query / 8 key-value heads of 128, windows of
    1024, 64 experts of 1024, top 6 from half of 8 groups, and a gated shared one of 2048; two streams, 24 layers."""
    base = dict(name="pivipel-3b", num_layers=24, width=2560, heads=32, kv_heads=8, dim=128, vdim=128, rot_dims=128, window=1024, keep=4,
                ff=6912, limit=7.0, experts=64, top=6, expert_ff=1024, shared_ff=2048, groups=8, keep_groups=4, vocab=65536, positions=16384)
    base.update(kw)
    return pivipel(**base)


def ledinex(num_layers: int = 4, width: int = 192, heads: int = 4, kv_heads: int = 2, dim: int = 64, vdim: int = 64, rot_dims: int = 32,
            window: int = 40, softcap: float = 25.0, right_heads: int = 3, right_dim: int = 64, right_vdim: int = 64, delta_heads: int = 4,
            delta_kv_heads: int = 2, delta_dim: int = 64, delta_vdim: int = 64, conv: int = 4, taps: int = 3, experts: int = 8, top: int = 2,
            expert_ff: int = 80, shared_ff: int = 160, vocab: int = 1024, order=("delta", "parallel", "parallel_2"), eps: float = 1e-6,
            **kw) -> ModelConfig:
    """Ledinex decoder of uniform layers: the types of `order` in turn, a mixture of experts in each."""
    layers = []
    for i in range(num_layers):
        t = order[i % len(order)]
        left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "scale": dim ** -0.5}
        if t == "delta":
            m = {"heads": delta_heads, "kv_heads": delta_kv_heads, "dim": delta_dim, "vdim": delta_vdim, "conv": conv}
        elif t == "parallel":
            left.update(vdim=vdim, softcap=softcap, rot={"base": 500000.0, "dims": dim, "scaling": {"factor": 4.0}})
            right = {"heads": right_heads, "dim": right_dim, "vdim": right_vdim,
                     "decay": [1.0 - 2.0 ** -(1.0 + 6.0 * (h + 1) / right_heads) for h in range(right_heads)]}
            m = {"left": left, "right": right, "left_scale": 0.7, "right_scale": 0.6}
        else:
            left.update(vdim=dim, mask={"size": window},
                        rot={"base": 10000.0, "dims": rot_dims, "scaling": {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}})
            m = {"left": left, "right": {"heads": right_heads, "dim": right_dim}, "left_scale": 0.7, "right_scale": 0.6}
        mlp = {"kind": "moe", "expert": {"ff": expert_ff}, "router": {"experts": experts, "top": top}}
        if shared_ff:
            mlp["shared"] = {"ff": shared_ff}
        layers.append({"type": t, "mixer": m, "mlp": mlp})
    cfg = {"architecture": "Ledinex", "vocab": vocab, "width": width, "embedding": {"scale": float(width) ** 0.5}, "logit_scale": 1.5,
           "canon": {"taps": taps}, "norm": {"eps": eps}, "layers": layers}
    return from_ledinex_config(cfg, name=kw.pop("name", "ledinex")).scaled(**kw)


def tiny_ledinex(**kw) -> ModelConfig:
    """Four-layer Ledinex (tests, smoke runs)."""
    return ledinex(**{"name": "tiny-ledinex", **kw})


def ledinex_3b(**kw) -> ModelConfig:
    """Ledinex with the layer sizes of a ~3B-active model: width 2560, 32 query / 8 key-value heads of 128, 20 recurrent heads
    of 128 x 128, windows of 1024, 64 experts of 1024, top 6, and a shared one of 2048; 24 layers."""
    base = dict(name="ledinex-3b", num_layers=24, width=2560, heads=32, kv_heads=8, dim=128, vdim=128, rot_dims=128, window=1024,
                right_heads=20, right_dim=128, right_vdim=128, delta_heads=20, delta_kv_heads=20, delta_dim=128, delta_vdim=128, experts=64,
                top=6, expert_ff=1024, shared_ff=2048, vocab=65536)
    base.update(kw)
    return ledinex(**base)


PRESETS = {
    "tiny-dense": tiny_dense,
    "tiny-ledinex": tiny_ledinex,
    "ledinex-3b": ledinex_3b,
    "tiny-pivipel": tiny_pivipel,
    "pivipel-3b": pivipel_3b,
    "tiny-finelix": tiny_finelix,
    "finelix-3b": finelix_3b,
    "tiny-fabulix": tiny_fabulix,
    "fabulix-3b": fabulix_3b,
    "tiny-kimi-linear": tiny_kimi_linear,
    "tiny-dense-hc": tiny_dense_hc,
    "tiny-hybrid-moe": tiny_hybrid_moe,
    "tiny-nemotron-h": tiny_nemotron_h,
    "dense-27b-nvfp4": dense_27b_nvfp4,
    "qwen-hybrid-moe-35b-fp8": qwen_hybrid_moe_35b,
    "nemotron-h-8b-fp8": nemotron_h_8b,
    "deepseek-v3-671b-fp8": deepseek_v3_671b,
}


def preset(name: str, **kw) -> ModelConfig:
    if name not in PRESETS:
        raise KeyError(f"unknown preset {name!r}; known: {sorted(PRESETS)}")
    return PRESETS[name](**kw)


# ----------------------------------------------------------------------------- HF config.json
_HF_ARCH = {
    "llama": "dense_gqa", "qwen2": "dense_gqa", "qwen3": "dense_gqa", "mistral": "dense_gqa",
    "granite": "dense_gqa", "olmo2": "dense_gqa", "minimax_m2": "dense_gqa", "glm4": "dense_gqa", "gemma3_text": "dense_gqa", "gemma3": "dense_gqa", "gemma2": "dense_gqa",
    "phi3": "dense_gqa", "qwen3_moe": "dense_gqa", "qwen2_moe": "dense_gqa", "mixtral": "dense_gqa",
    "qwen3_5": "qwen_hybrid", "qwen3_5_moe": "qwen_hybrid", "qwen3_next": "qwen_hybrid",
    "qwen3_5_text": "qwen_hybrid", "qwen3_5_moe_text": "qwen_hybrid",
    "nemotron_h": "nemotron_h", "deepseek_v3": "deepseek_mla", "deepseek_v2": "deepseek_mla",
    "kimi_k2": "deepseek_mla",          # Kimi K2 checkpoints use the DeepSeek-V3 architecture and tensor names
    "deepseek_v32": "deepseek_mla",     # DeepSeek-V3.2: V3 + the sparse-attention indexer
    "kimi_linear": "deepseek_mla",      # Kimi-Linear: Kimi-delta-attention layers + (NoPE) MLA layers, DeepSeek-style MoE
}


# vision-language wrappers -> the text stack they carry (tensor names under model.language_model. are
# unwrapped by weights/remap.py)
_HF_VISION = {"qwen2_vl": "qwen2", "qwen2_5_vl": "qwen2", "qwen2_vl_text": "qwen2", "qwen2_5_vl_text": "qwen2",
              "qwen3_vl": "qwen3", "qwen3_vl_text": "qwen3"}


def detect_weight_format(qc: Optional[dict]) -> str:
    """quantization_config -> serving weight format
    (crates/model-layers/src/quant_format/mod.rs:61-138, weight_map/nvfp4_detect.rs:23-38)."""
    if not qc:
        return "bf16"
    method = str(qc.get("quant_method", "")).lower()
    algo = str(qc.get("quant_algo", "")).upper()
    fmt = str(qc.get("format", "")).lower()
    if method == "modelopt":
        return "nvfp4" if "NVFP4" in algo else ("fp8_row" if "FP8" in algo else "bf16")
    if method == "compressed-tensors":
        if "float-quantized" in fmt or "fp8" in fmt:
            return "fp8_row"
        return "nvfp4"
    if method == "fp8":
        return "fp8_block" if qc.get("weight_block_size") else "fp8_row"
    raise ValueError(f"unsupported quant_method {method!r}")


def from_fabulix_config(cfg: dict, name: str = "model") -> ModelConfig:
    """A Fabulix ``config.json``: sizes and constants are given per layer and kept per layer. Mixer types and
    feed-forward kinds this engine does not know are refused."""
    types, ffns, specs = [], [], []
    for i, L in enumerate(cfg["layers"]):
        t, m, mlp = L["type"], L["mixer"], L.get("mlp")
        if t not in ("parallel", "lightning"):
            raise ValueError(f"layer {i}: unknown mixer type {t!r}")
        if mlp is not None and mlp.get("kind") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        if t == "parallel":
            a = m["left"]
            if a["heads"] % a["kv_heads"] or a["rot"]["dims"] % 2 or a["rot"]["dims"] > a["dim"]:
                raise ValueError(f"layer {i}: attention heads, key/value heads or rotary size do not fit together")
        elif len(m["decay"]) != m["heads"]:
            raise ValueError(f"layer {i}: {len(m['decay'])} decays for {m['heads']} heads")
        types.append(t)
        ffns.append("none" if mlp is None else "dense")
        specs.append({"mixer": m, "mlp": mlp})
    att = next((s["mixer"]["left"] for t, s in zip(types, specs) if t == "parallel"), {"heads": 1, "kv_heads": 1, "dim": 64})
    return ModelConfig(
        name=name, arch="fabulix", vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_layers=len(types), layer_types=types,
        ffn_types=ffns, layer_specs=specs, num_heads=att["heads"], num_kv_heads=att["kv_heads"], head_dim=att["dim"], rotary_dim=-1,
        rms_eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]), tie_embeddings=True,
        intermediate_size=max((s["mlp"]["ff"] for s in specs if s["mlp"]), default=0),
        token_side_dim=int((cfg.get("token_side") or {}).get("dim", 0)), max_position=131072)


_FINELIX_MIXERS = {"latent_attention": "latent", "gla": "gla", "gla_2": "gla"}


def from_finelix_config(cfg: dict, name: str = "model") -> ModelConfig:
    """A Finelix ``config.json``: sizes and constants are given per layer and kept per layer, `loop` names the
    range of layers that runs several times. Mixer types and feed-forward kinds this engine does not know are
    refused."""
    types, ffns, specs = [], [], []
    for i, L in enumerate(cfg["layers"]):
        t, m, mlp = L["type"], L["mixer"], L.get("mlp")
        if t not in _FINELIX_MIXERS:
            raise ValueError(f"layer {i}: unknown mixer type {t!r}")
        if mlp is not None and mlp.get("kind") not in ("dense", "moe"):
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        if _FINELIX_MIXERS[t] == "latent":
            if m["rot_dim"] % 2 or m["rot"]["dims"] != m["rot_dim"]:
                raise ValueError(f"layer {i}: the rotary size is not the rotated part's")
        elif not m["tau"] > 0:
            raise ValueError(f"layer {i}: tau must be positive")
        if mlp is not None and mlp["kind"] == "moe" and not 0 < mlp["router"]["top"] <= min(32, mlp["router"]["experts"]):
            raise ValueError(f"layer {i}: {mlp['router']['top']} of {mlp['router']['experts']} experts per token")
        types.append(_FINELIX_MIXERS[t])
        ffns.append("none" if mlp is None else mlp["kind"])
        specs.append({"mixer": m, "mlp": mlp})
    loop = cfg.get("loop") or None
    if loop is not None:
        loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
        if not (0 <= loop["start"] < loop["stop"] <= len(types) and loop["times"] > 0):
            raise ValueError(f"loop {loop} does not fit {len(types)} layers")
    att = next((s["mixer"] for t, s in zip(types, specs) if t == "latent"), {"heads": 1, "dim": 64, "rot_dim": 0})
    moe = next((s["mlp"] for f, s in zip(ffns, specs) if f == "moe"), None)
    return ModelConfig(
        name=name, arch="finelix", vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_layers=len(types), layer_types=types,
        ffn_types=ffns, layer_specs=specs, loop=loop, num_heads=att["heads"], num_kv_heads=att["heads"], head_dim=att["dim"] + att["rot_dim"],
        rotary_dim=-1, rms_eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]), tie_embeddings=False,
        intermediate_size=max((s["mlp"]["ff"] for s, f in zip(specs, ffns) if f == "dense"), default=0),
        num_experts=moe["router"]["experts"] if moe else 0, experts_per_token=moe["router"]["top"] if moe else 0,
        moe_intermediate_size=moe["expert"]["ff"] if moe else 0, max_position=131072)


def from_pivipel_config(cfg: dict, name: str = "model") -> ModelConfig:
    """A Pivipel ``config.json``: sizes and constants are given per layer and kept per layer; a layer with `weights_of`
    uses another one's tensors. Mixer types and feed-forward kinds this engine does not know are refused."""
    types, ffns, specs, owners = [], [], [], []
    for i, L in enumerate(cfg["layers"]):
        t, m, mlp = L["type"], L["mixer"], L.get("mlp")
        if t not in ("attention", "attention_2"):
            raise ValueError(f"layer {i}: unknown mixer type {t!r}")
        if mlp is not None and mlp.get("kind") not in ("dense", "moe"):
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        rot, mask, of = m.get("rot") or {"dims": 0}, m.get("mask") or {}, L.get("weights_of")
        if m["heads"] % m["kv_heads"] or rot["dims"] % 2 or rot["dims"] > m["dim"]:
            raise ValueError(f"layer {i}: attention heads, key/value heads or rotary size do not fit together")
        if mask.get("size", 1) < 1 or mask.get("keep_first", 0) < 0:
            raise ValueError(f"layer {i}: a window of {mask.get('size')} with {mask.get('keep_first')} kept tokens")
        if mlp is not None and mlp["kind"] == "moe":
            r = mlp["router"]
            g = r.get("groups") or {"count": 1, "keep": 1}
            if r["experts"] > 512 or r["experts"] % g["count"] or not 0 < g["keep"] <= g["count"] <= 32 \
                    or not 0 < r["top"] <= min(32, r["experts"] // g["count"] * g["keep"]):
                raise ValueError(f"layer {i}: {r['top']} of {r['experts']} experts per token from {g['keep']} of {g['count']} groups")
        if of is not None and not (0 <= of < len(cfg["layers"]) and of != i):
            raise ValueError(f"layer {i}: no tensors of layer {of}")
        types.append(t)
        ffns.append("none" if mlp is None else mlp["kind"])
        specs.append({"mixer": m, "mlp": mlp})
        owners.append(-1 if of is None else int(of))
    for i in range(len(owners)):
        seen, j = set(), i
        while owners[j] >= 0:
            if j in seen:
                raise ValueError(f"layer {i}: its tensors are its own by way of others")
            seen.add(j)
            j = owners[j]
        if types[j] != types[i] or specs[j] != specs[i]:
            raise ValueError(f"layer {i}: not like layer {j}, whose tensors it uses")
    if int(cfg["streams"]) < 1:
        raise ValueError(f"{cfg['streams']} residual streams")
    att, moe = specs[0]["mixer"], next((s["mlp"] for f, s in zip(ffns, specs) if f == "moe"), None)
    return ModelConfig(
        name=name, arch="pivipel", vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_layers=len(types), layer_types=["gated"] * len(types),
        ffn_types=ffns, layer_specs=specs, spec_types=types, weights_of=owners, streams=int(cfg["streams"]), num_heads=att["heads"],
        num_kv_heads=att["kv_heads"], head_dim=att["dim"], rotary_dim=-1, rms_eps=float(cfg["norm"]["eps"]), tie_embeddings=True,
        intermediate_size=max((s["mlp"]["ff"] for s, f in zip(specs, ffns) if f == "dense"), default=0),
        num_experts=moe["router"]["experts"] if moe else 0, experts_per_token=moe["router"]["top"] if moe else 0,
        moe_intermediate_size=moe["expert"]["ff"] if moe else 0, max_position=int(cfg["max_positions"]))


_LEDINEX_MIXERS = {"parallel": "twin", "parallel_2": "twin", "delta": "delta"}


def from_ledinex_config(cfg: dict, name: str = "model") -> ModelConfig:
    """A Ledinex ``config.json``: sizes and constants are given per layer and kept per layer. Mixer types and feed-forward
    kinds this engine does not know are refused."""
    types, ffns, specs = [], [], []
    for i, L in enumerate(cfg["layers"]):
        t, m, mlp = L["type"], L["mixer"], L.get("mlp")
        if t not in _LEDINEX_MIXERS:
            raise ValueError(f"layer {i}: unknown mixer type {t!r}")
        if mlp is not None and mlp.get("kind") != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        if t == "delta":
            if m["heads"] % m["kv_heads"] or not 0 < m["conv"] <= 17 or m["dim"] > 256:
                raise ValueError(f"layer {i}: heads, head sizes or taps this engine does not serve")
        else:
            a, r = m["left"], m["right"]
            rot = a["rot"]["dims"]
            if a["heads"] % a["kv_heads"] or rot % 2 or rot > a["dim"] or (t == "parallel" and a["vdim"] % 2):
                raise ValueError(f"layer {i}: attention heads, key/value heads or rotary size do not fit together")
            if t == "parallel_2" and a.get("vdim", a["dim"]) != a["dim"]:
                raise ValueError(f"layer {i}: values that are keys have their size")
            if (a.get("mask") or {}).get("size", 1) < 1:
                raise ValueError(f"layer {i}: a window of {a['mask']['size']}")
            if r["dim"] > 256 or (t == "parallel" and len(r["decay"]) != r["heads"]):
                raise ValueError(f"layer {i}: recurrent heads, head sizes or decays do not fit together")
        if mlp is not None:
            r = mlp["router"]
            if r["experts"] > 512 or not 0 < r["top"] <= min(32, r["experts"]):
                raise ValueError(f"layer {i}: {r['top']} of {r['experts']} experts per token")
        types.append(t)
        ffns.append("none" if mlp is None else "moe")
        specs.append({"mixer": m, "mlp": mlp})
    taps = int(cfg["canon"]["taps"])
    if not 0 < taps <= 21:
        raise ValueError(f"input convolutions of {taps} taps")
    att = next((s["mixer"]["left"] for t, s in zip(types, specs) if t != "delta"), {"heads": 1, "kv_heads": 1, "dim": 64})
    moe = next((s["mlp"] for s in specs if s["mlp"]), None)
    return ModelConfig(
        name=name, arch="ledinex", vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_layers=len(types),
        layer_types=[_LEDINEX_MIXERS[t] for t in types], ffn_types=ffns, layer_specs=specs, spec_types=types, canon_taps=taps,
        num_heads=att["heads"], num_kv_heads=att["kv_heads"], head_dim=att["dim"], rotary_dim=-1, rms_eps=float(cfg["norm"]["eps"]),
        norm_plus_one=True, embed_scale=float(cfg["embedding"]["scale"]), logit_scale=float(cfg["logit_scale"]), tie_embeddings=True,
        intermediate_size=0, ffn_act="relu2", num_experts=moe["router"]["experts"] if moe else 0,
        experts_per_token=moe["router"]["top"] if moe else 0, moe_intermediate_size=moe["expert"]["ff"] if moe else 0, max_position=131072)


def from_hf_config(cfg: dict, name: str = "model") -> ModelConfig:
    """Map a HF ``config.json`` dict (text stack) to ModelConfig; refuses unknown model types."""
    if cfg.get("architecture") == "Ledinex":
        return from_ledinex_config(cfg, name)
    if cfg.get("architecture") == "Pivipel":
        return from_pivipel_config(cfg, name)
    if cfg.get("architecture") == "Fabulix":
        return from_fabulix_config(cfg, name)
    if cfg.get("architecture") == "Finelix":
        return from_finelix_config(cfg, name)
    outer = cfg
    if "text_config" in cfg:
        inner = dict(cfg["text_config"])
        inner.setdefault("quantization_config", cfg.get("quantization_config"))
        cfg = inner
    mt = cfg.get("model_type", "")
    vision_kw = {}
    if outer.get("vision_config") and (outer.get("model_type", "") in _HF_VISION or mt in _HF_VISION):
        rs = cfg.get("rope_scaling") or outer.get("rope_scaling") or {}
        vision_kw = dict(vision=dict(outer["vision_config"]), image_token_id=int(outer.get("image_token_id", -1)),
                         vision_start_token_id=int(outer.get("vision_start_token_id", -1)),
                         mrope_sections=list(rs["mrope_section"]) if rs.get("mrope_section") else None)
        if mt in _HF_VISION:
            mt = _HF_VISION[mt]
        if (rs.get("type") or rs.get("rope_type")) in ("mrope", "default"):
            cfg = dict(cfg)
            cfg["rope_scaling"] = None                     # the sections only say which axis a frequency follows
    if mt not in _HF_ARCH:
        raise ValueError(f"unsupported model_type {mt!r}")
    arch = _HF_ARCH[mt]
    h = cfg["hidden_size"]
    L = cfg["num_hidden_layers"]
    heads = cfg.get("num_attention_heads", 1)
    kw = dict(name=name, arch=arch, vocab_size=cfg["vocab_size"], hidden_size=h, num_layers=L,
              num_heads=heads, num_kv_heads=cfg.get("num_key_value_heads", heads),
              head_dim=cfg.get("head_dim", h // heads), rope_theta=float(cfg.get("rope_theta", 1e4)), rope_scaling=cfg.get("rope_scaling"),
              rms_eps=float(cfg.get("rms_norm_eps", cfg.get("layer_norm_epsilon", 1e-6))),
              intermediate_size=cfg.get("intermediate_size", 0),
              tie_embeddings=bool(cfg.get("tie_word_embeddings", False)),
              max_position=int(cfg.get("max_position_embeddings", 32768)),
              weight_format=detect_weight_format(cfg.get("quantization_config")),
              mtp_layers=int(cfg.get("mtp_num_hidden_layers", cfg.get("num_nextn_predict_layers", 0)) or 0))
    if arch == "dense_gqa":
        kw["qk_norm"] = mt in ("qwen3", "qwen3_moe")
        kw["attn_bias"] = bool(cfg.get("attention_bias", cfg.get("qkv_bias", mt in ("qwen2", "qwen2_moe"))))
        kw["sliding_window"] = int(cfg.get("sliding_window") or 0) if cfg.get("use_sliding_window") else 0
        if mt in ("gemma3_text", "gemma3", "gemma2"):
            if cfg.get("attn_logit_softcapping"):
                raise ValueError("attention logit soft-capping (Gemma 2) is not supported")
            act = cfg.get("hidden_activation", cfg.get("hidden_act", "gelu_pytorch_tanh"))
            if act not in ("gelu_pytorch_tanh", "gelu_tanh"):
                raise ValueError(f"unsupported Gemma activation {act!r}")
            win = int(cfg.get("sliding_window") or 0)
            lt = cfg.get("layer_types")
            if lt is None:
                pat = int(cfg.get("sliding_window_pattern", 6) or 6)
                lt = ["full_attention" if (i + 1) % pat == 0 else "sliding_attention" for i in range(L)]
            kw.update(norm_plus_one=True, post_norms=True, ffn_act="geglu", qk_norm=mt != "gemma2",
                      embed_scale=float(h) ** 0.5, tie_embeddings=bool(cfg.get("tie_word_embeddings", True)),
                      attn_scale=float(cfg.get("query_pre_attn_scalar", kw["head_dim"])) ** -0.5,
                      window_layers=[win if t == "sliding_attention" else 0 for t in lt], sliding_window=0,
                      rope_local_theta=float(cfg.get("rope_local_base_freq", 0.0) or 0.0),
                      final_logit_softcap=float(cfg.get("final_logit_softcapping") or 0.0))
        if mt == "granite":
            kw.update(embed_scale=float(cfg.get("embedding_multiplier", 1.0)), attn_scale=float(cfg.get("attention_multiplier", 0.0) or 0.0),
                      residual_multiplier=float(cfg.get("residual_multiplier", 1.0)),
                      logits_divisor=float(cfg.get("logits_scaling", 1.0) or 1.0),
                      attn_bias=bool(cfg.get("attention_bias", False)))
        if mt == "olmo2":
            kw.update(post_norms=True, post_norm_names="olmo2", pre_norms=False, qk_norm=True, qk_norm_full=True,
                      attn_bias=bool(cfg.get("attention_bias", False)))
        if mt == "minimax_m2":
            if cfg.get("shared_intermediate_size"):
                raise ValueError("MiniMax shared experts are not supported")
            kw.update(qk_norm=bool(cfg.get("use_qk_norm", True)), qk_norm_full=cfg.get("qk_norm_type", "per_layer") == "per_layer",
                      rotary_dim=int(cfg.get("rotary_dim", kw["head_dim"])), ffn_types=["moe"] * L,
                      num_experts=int(cfg.get("num_local_experts", 0)), experts_per_token=int(cfg.get("num_experts_per_tok", 8)),
                      moe_intermediate_size=cfg.get("intermediate_size", 0),
                      router="sigmoid" if cfg.get("scoring_func", "sigmoid") == "sigmoid" else "softmax",
                      router_renormalize=True, router_scaling=float(cfg.get("routed_scaling_factor", 1.0)))
        if mt == "glm4":
            kw.update(post_norms=True, post_norm_names="glm", rope_interleaved=True,
                      attn_bias=bool(cfg.get("attention_bias", True)),
                      rotary_dim=int(kw["head_dim"] * float(cfg.get("partial_rotary_factor", 0.5))))
        if mt == "phi3":
            rs = cfg.get("rope_scaling")
            if rs and str(rs.get("type", rs.get("rope_type", ""))).lower() in ("longrope", "su"):
                raise ValueError("phi3 longrope scaling is not supported")
            prf = float(cfg.get("partial_rotary_factor", 1.0))
            if prf < 1.0:
                kw["rotary_dim"] = int(kw["head_dim"] * prf)
        if mt in ("qwen3_moe", "qwen2_moe"):
            step = int(cfg.get("decoder_sparse_step", 1) or 1)
            only = set(cfg.get("mlp_only_layers") or [])
            ne = int(cfg.get("num_experts", 0))
            kw.update(ffn_types=["moe" if ne and i not in only and (i + 1) % step == 0 else "dense" for i in range(L)],
                      num_experts=ne, experts_per_token=cfg.get("num_experts_per_tok", 8),
                      moe_intermediate_size=cfg.get("moe_intermediate_size", 768), router="softmax",
                      router_renormalize=bool(cfg.get("norm_topk_prob", mt == "qwen3_moe")))
            if mt == "qwen2_moe" and cfg.get("shared_expert_intermediate_size", 0):
                mi = kw["moe_intermediate_size"]
                sh = int(cfg["shared_expert_intermediate_size"])
                if sh % mi:
                    raise ValueError("shared expert width must be a multiple of the routed expert width")
                kw.update(num_shared_experts=sh // mi, shared_expert_gate=True, shared_expert_name="shared_expert")
        if mt == "mixtral":
            kw.update(ffn_types=["moe"] * L, num_experts=int(cfg.get("num_local_experts", 8)),
                      experts_per_token=int(cfg.get("num_experts_per_tok", 2)),
                      moe_intermediate_size=cfg.get("intermediate_size", 0), router="softmax", router_renormalize=True)
    elif arch == "qwen_hybrid":
        lt = cfg.get("layer_types")
        interval = cfg.get("full_attention_interval", 4)
        if lt is None:
            lt = ["full_attention" if (i + 1) % interval == 0 else "linear_attention" for i in range(L)]
        if cfg.get("linear_conv_kernel_dim", 4) != 4:
            raise ValueError("linear_conv_kernel_dim must be 4")
        kw.update(layer_types=["attention" if t == "full_attention" else "gdn" for t in lt],
                  qk_norm=True, attn_output_gate=bool(cfg.get("attn_output_gate", True)), norm_plus_one=True,
                  rotary_dim=int(cfg.get("head_dim", h // heads) * cfg.get("partial_rotary_factor", 0.25)),
                  gdn_k_heads=cfg.get("linear_num_key_heads", 16), gdn_v_heads=cfg.get("linear_num_value_heads", 32),
                  gdn_k_dim=cfg.get("linear_key_head_dim", 128), gdn_v_dim=cfg.get("linear_value_head_dim", 128))
        ne = cfg.get("num_experts", 0)
        if ne:
            kw.update(ffn_types=["moe"] * L, num_experts=ne, experts_per_token=cfg.get("num_experts_per_tok", 8),
                      moe_intermediate_size=cfg.get("moe_intermediate_size", 512),
                      num_shared_experts=1 if cfg.get("shared_expert_intermediate_size", 0) else 0,
                      shared_expert_gate=True, router="softmax",
                      router_renormalize=bool(cfg.get("norm_topk_prob", True)))
    elif arch == "nemotron_h":
        pat = cfg.get("hybrid_override_pattern", "")
        lt, ft = [], []
        for ch in pat:
            if ch == "M":
                lt.append("mamba2"); ft.append("none")
            elif ch == "*":
                lt.append("attention"); ft.append("none")
            elif ch in "-E":
                # an MLP/MoE block: attach to the previous mixer when it has no FFN yet
                if lt and ft[-1] == "none":
                    ft[-1] = "dense" if ch == "-" else "moe"
                else:
                    lt.append("mamba2"); ft.append("dense" if ch == "-" else "moe")
        kw.update(layer_types=lt, ffn_types=ft, num_layers=len(lt), rotary_dim=-1, ffn_act="relu2",
                  mamba_heads=cfg.get("mamba_num_heads", 128), mamba_head_dim=cfg.get("mamba_head_dim", 64),
                  mamba_state=cfg.get("ssm_state_size", 128), mamba_groups=cfg.get("n_groups", 8),
                  conv_kernel=cfg.get("conv_kernel", 4))
    else:
        fd = cfg.get("first_k_dense_replace", 0)
        kw.update(layer_types=["mla"] * L, ffn_types=["dense"] * fd + ["moe"] * (L - fd), first_dense_layers=fd,
                  dense_intermediate_size=cfg.get("intermediate_size", 0),
                  q_lora_rank=cfg.get("q_lora_rank") or 0, kv_lora_rank=cfg.get("kv_lora_rank", 512),
                  qk_nope_dim=cfg.get("qk_nope_head_dim", 128), qk_rope_dim=cfg.get("qk_rope_head_dim", 64),
                  v_head_dim=cfg.get("v_head_dim", 128), head_dim=cfg.get("qk_nope_head_dim", 128) + cfg.get("qk_rope_head_dim", 64),
                  num_experts=cfg.get("n_routed_experts", 0), experts_per_token=cfg.get("num_experts_per_tok", 8),
                  moe_intermediate_size=cfg.get("moe_intermediate_size", 2048),
                  num_shared_experts=cfg.get("n_shared_experts", 0),
                  router="sigmoid" if cfg.get("scoring_func", "softmax") == "sigmoid" else "softmax",
                  router_n_group=cfg.get("n_group", 1), router_topk_group=cfg.get("topk_group", 1),
                  router_scaling=float(cfg.get("routed_scaling_factor", 1.0)),
                  router_renormalize=bool(cfg.get("norm_topk_prob", True)))
        if cfg.get("index_topk"):
            kw.update(index_topk=int(cfg["index_topk"]), index_n_heads=int(cfg.get("index_n_heads", 64)),
                      index_head_dim=int(cfg.get("index_head_dim", 128)))
        if mt == "kimi_linear":
            la = cfg.get("linear_attn_config") or {}
            kda_layers = {int(i) - 1 for i in la.get("kda_layers", [])}            # the checkpoint counts layers from 1
            if not kda_layers:
                raise ValueError("kimi_linear needs linear_attn_config.kda_layers")
            conv = int(la.get("short_conv_kernel_size", 4))
            kw.update(layer_types=["kda" if i in kda_layers else "mla" for i in range(L)],
                      kda_heads=int(la.get("num_heads", heads)), kda_head_dim=int(la.get("head_dim", 128)),
                      kda_gate_rank=int(la.get("gate_rank", 0) or 0), conv_kernel=conv,
                      kda_gate_lower_bound=float(la.get("gate_lower_bound", -5.0)),
                      rope_identity=bool(cfg.get("mla_use_nope", False)),
                      num_experts=cfg.get("num_experts", cfg.get("n_routed_experts", 0)),
                      experts_per_token=cfg.get("num_experts_per_token", cfg.get("num_experts_per_tok", 8)),
                      num_shared_experts=cfg.get("num_shared_experts", cfg.get("n_shared_experts", 0)),
                      router="sigmoid" if cfg.get("moe_router_activation_func", cfg.get("scoring_func", "sigmoid")) == "sigmoid" else "softmax",
                      router_n_group=cfg.get("num_expert_group", cfg.get("n_group", 1)),
                      router_topk_group=cfg.get("topk_group", 1),
                      router_renormalize=bool(cfg.get("moe_renormalize", cfg.get("norm_topk_prob", True))))
    kw.update(vision_kw)
    return ModelConfig(**kw)


def load_hf_config(path) -> ModelConfig:
    p = Path(path)
    return from_hf_config(json.loads((p / "config.json").read_text()), name=p.name)
