"""Architecture description for the decoder-only model families the framework trains and serves.

One dataclass covers Llama (2/3/3.1/3.2), Mistral, Qwen2/2.5, Qwen3, Qwen3-MoE and Gemma 3 (text); the differences are switches
(QKV bias, per-head q/k RMSNorm, tied embeddings, RoPE scaling, mixture-of-experts FFN; for Gemma 3: tanh-GELU gate, norms
before and after each block, scaled embeddings, sliding-window layers with their own RoPE base, a fixed attention scale). ``from_hf_dict`` reads a
HuggingFace ``config.json`` dictionary; ``PRESETS`` names the architectures used by the benchmark configs.

Models described layer by layer (Gadarax, Redarax, Kikivik, Zonidra) keep their layer list in ``mixers``: each entry names the sequence mixer, its sizes
and its MLP. ``LAYER_LISTS`` says which mixers and MLPs each architecture has and how its configuration maps to ``ModelConfig``:
Gadarax runs mixer and MLP side by side behind one norm (``layer_loop`` repeats a range of layers with the same weights), Redarax runs
them one after the other and norms what they return (``norm_place`` "post"), with an input per layer and token (``token_side``), Kikivik
runs them one after the other on norms of the residual stream, Zonidra does that and norms and scales what they return as well
(``norm_place`` "both", ``layer_scale``), its mixers read a blend with the token before (``token_shift``) and its embedding has a second
table over pairs of tokens (``bigram``). What an architecture fixes for all its mixers of a kind (biases, gates, the
layout of rotated pairs) is in ``traits`` and joins each layer's sizes (``mixer_spec``, ``mlp_spec``).
"""

from __future__ import annotations

import json
import math
import os
from dataclasses import asdict, dataclass, field
from typing import Any, Optional

import torch


@dataclass
class ModelConfig:
    model_type: str = "llama"
    vocab_size: int = 32000
    hidden_size: int = 4096
    intermediate_size: int = 11008
    num_hidden_layers: int = 32
    num_attention_heads: int = 32
    num_key_value_heads: int = 32
    head_dim: int = 128
    rms_norm_eps: float = 1e-5
    rope_theta: float = 10000.0
    rope_scaling: Optional[dict] = None
    max_position_embeddings: int = 131072
    tie_word_embeddings: bool = False
    attention_bias: bool = False       # Qwen2: bias on q/k/v projections
    qk_norm: bool = False              # Qwen3: RMSNorm over head_dim on q and k before RoPE
    # mixture of experts (Qwen3-MoE): num_experts > 0 replaces the dense FFN
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True
    router_aux_loss_coef: float = 0.0
    bos_token_id: Optional[int] = None
    eos_token_id: Optional[Any] = None
    pad_token_id: Optional[int] = None
    torch_dtype: str = "bfloat16"
    value_head: bool = False           # critic / reward model: scalar head instead of the vocabulary projection
    vision: Optional[dict] = None      # vision tower settings (models/vision.py); None: text-only model
    image_token_id: Optional[int] = None
    # Gemma 3 (nemo_rl/models/dtensor/parallelize.py:170-217 is the reference's parallel plan for this family)
    hidden_act: str = "silu"           # gate activation of the MLP: silu | gelu_pytorch_tanh
    sandwich_norm: bool = False        # RMSNorm before AND after attention / MLP (the post norms act on the block output)
    embed_scale: float = 1.0           # embeddings are multiplied by this (sqrt(hidden_size))
    norm_offset: float = 0.0           # checkpoints store RMSNorm weights as w - offset (Gemma: 1); buffers here hold w
    sliding_window: int = 0            # > 0: layers listed as "sliding_attention" see only the last `sliding_window` keys
    layer_types: Optional[list] = None  # per layer: "full_attention" | "sliding_attention"
    rope_local_theta: float = 0.0      # RoPE base of the sliding-window layers (0: same as rope_theta, scaling included)
    attn_scale: Optional[float] = None  # softmax scale when it is not head_dim ** -0.5 (query_pre_attn_scalar ** -0.5)
    final_logit_softcap: float = 0.0   # logits <- cap * tanh(logits / cap) (Gemma 2, Redarax; 0: off)

    # DeepSeek-V3: multi-head latent attention and its mixture of experts
    kv_lora_rank: int = 0              # > 0: attention is MLA (keys / values decompressed from a latent of this width)
    q_lora_rank: Optional[int] = None  # low-rank query projection (None: a plain q_proj)
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    rope_interleave: bool = True       # checkpoints store the rotary dimensions interleaved (pairs), not split in halves
    n_shared_experts: int = 0          # dense experts every token passes through, added to the routed output
    first_k_dense_replace: int = 0     # the first k layers keep a dense MLP
    scoring_func: str = "softmax"      # router scores: softmax | sigmoid (with a per-expert selection bias)
    n_group: int = 1                   # experts are split in groups; only `topk_group` groups stay eligible per token
    topk_group: int = 1
    routed_scaling_factor: float = 1.0

    # Nemotron-H (hybrid Mamba-2 / attention / MLP / MoE; nemo_rl/models/dtensor/parallelize.py:465 is the reference's plan
    # for this family): every layer is ONE mixer behind one RMSNorm, named by ``layers_block_type``
    layers_block_type: Optional[list] = None   # per layer: "mamba" | "attention" | "mlp" | "moe"
    use_rope: bool = True              # False: attention has no positional rotation (the state-space layers carry order)
    mlp_gated: bool = True             # False: down(act(up(x))) instead of down(act(gate(x)) * up(x))
    mlp_bias: bool = False
    mamba_num_heads: int = 0
    mamba_head_dim: int = 0
    ssm_state_size: int = 0
    mamba_n_groups: int = 1
    mamba_d_conv: int = 4
    mamba_chunk_size: int = 128
    mamba_conv_bias: bool = True
    mamba_proj_bias: bool = False
    mamba_dt_limit: Optional[list] = None      # [lo, hi] clamp of the step size after softplus
    moe_latent_size: Optional[int] = None      # routed experts work in a narrower space between two shared projections
    moe_shared_expert_intermediate_size: int = 0

    # models described layer by layer (Gadarax, Redarax, Kikivik, Zonidra): the layers differ in their mixers, sizes and MLPs
    mixers: Optional[list] = None      # per layer: {"type": name of the mixer, "mixer": {sizes}, "mlp": {"kind", sizes} or None}
    layer_loop: Optional[dict] = None  # {"start", "stop", "times"}: layers start .. stop - 1 run `times` times in a row with the same weights
    norm_kind: str = "rms"             # "rms" | "dyt" (dynamic tanh: w * tanh(alpha x) + b, no statistics)
    norm_place: str = "pre"            # "pre": sublayers read norm(x); "post": they read x, and norm(output) joins the residual stream; "both"
    residual_mult: float = 1.0         # what sublayer outputs are multiplied by when they join the residual stream
    token_side: Optional[dict] = None  # {"dim"}: every layer adds an input looked up by token in a table of its own (gated by the stream)
    layer_scale: bool = False          # sublayer outputs are multiplied element by element when they join the residual stream
    token_shift: bool = False          # mixers read h + (h of the token before - h) * s, element by element
    bigram: Optional[dict] = None      # {"buckets", "mul_prev", "mul_cur"}: embeddings get a row looked up by (token before, token)
    logit_scale: float = 1.0           # logits are multiplied by this (before the soft cap)
    traits: dict = field(default_factory=dict)   # kind of mixer or MLP: what the architecture fixes for it, in the words of its class

    @property
    def is_hybrid(self) -> bool:
        return self.layers_block_type is not None

    @property
    def is_mixer(self) -> bool:
        return self.mixers is not None

    @property
    def layer_form(self) -> str:
        """How the layers of a layer-list model are put together: "parallel" | "post" | "pre" (see the three block classes)."""
        return "post" if self.norm_place == "post" else "parallel" if self.norm_kind == "dyt" else "pre"

    def mixer_spec(self, i: int) -> dict:
        return {**self.traits.get(self.mixers[i]["type"], {}), **self.mixers[i]["mixer"]}

    def mlp_spec(self, i: int) -> dict:
        mlp = self.mixers[i]["mlp"]
        return {**self.traits.get(mlp.get("kind", "dense"), {}), **mlp}

    @property
    def is_recurrent(self) -> bool:
        """The model carries a per-sequence state beside (or instead of) cache pages: prefixes cannot be shared by pages."""
        return self.is_hybrid or self.token_shift or bool(self.bigram) or (self.mixers is not None and any(m["type"] in RECURRENT_MIXERS for m in self.mixers))

    @property
    def caps_logits(self) -> bool:
        """Logits are more than the product with the output weight (a scale or a soft cap follows)."""
        return self.logit_scale != 1.0 or bool(self.final_logit_softcap)

    @property
    def layer_runs(self) -> list:
        """[(layer, pass)] in execution order; pass counts from 0 inside the loop and is None outside it."""
        lp, n = self.layer_loop, self.num_hidden_layers
        if not lp:
            return [(i, None) for i in range(n)]
        body = [(i, t) for t in range(lp["times"]) for i in range(lp["start"], lp["stop"])]
        return [(i, None) for i in range(lp["start"])] + body + [(i, None) for i in range(lp["stop"], n)]

    def block_type(self, i: int) -> str:
        """"mamba" | "attention" | "mlp" | "moe" for hybrid models, "decoder" (attention + MLP in one layer) otherwise."""
        return self.layers_block_type[i] if self.layers_block_type is not None else "decoder"

    @property
    def mamba_inner(self) -> int:
        return self.mamba_num_heads * self.mamba_head_dim

    @property
    def mamba_conv_dim(self) -> int:
        return self.mamba_inner + 2 * self.mamba_n_groups * self.ssm_state_size

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0

    def layer_is_moe(self, i: int) -> bool:
        if self.layers_block_type is not None:
            return self.layers_block_type[i] == "moe"
        return self.is_moe and i >= self.first_k_dense_replace

    def layer_is_sliding(self, i: int) -> bool:
        return bool(self.sliding_window) and self.layer_types is not None and self.layer_types[i] == "sliding_attention"

    @property
    def q_size(self) -> int:
        return self.num_attention_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_key_value_heads * self.head_dim

    @property
    def qkv_size(self) -> int:
        return self.q_size + 2 * self.kv_size

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    def num_parameters(self) -> int:
        d, L = self.hidden_size, self.num_hidden_layers
        if self.model_type == "redarax":
            sd = self.token_side["dim"] if self.token_side else 0
            n = 2 * self.vocab_size * d + d + self.vocab_size * L * sd
            for e in self.mixers:
                m, mlp = e["mixer"], e.get("mlp")
                H, vd = m["heads"], m["vdim"]
                if e["type"] == "attention":
                    G, kd = m["kv_heads"], m["dim"]
                    n += (d + 1) * (H * kd + G * kd + G * vd) + 2 * kd + (H * vd + 1) * d
                elif e["type"] == "mamba2":
                    C = H * vd + 2 * m["groups"] * m["state"]
                    n += d * (H * vd + C + H) + C * (m["conv"] + 1) + 3 * H + H * vd + H * vd * d
                else:
                    C = 2 * m["kv_heads"] * m["dim"] + H * vd
                    n += d * (C + 2 * H + 2 * H * vd) + C * m["conv"] + 2 * H + vd
                n += d
                if mlp:
                    r = mlp.get("router")
                    n += d + (r["experts"] * (3 * d * mlp["expert"]["ff"] + d + 1) if r else 3 * d * mlp["ff"])
                n += 2 * d * sd + (d if sd else 0)
            return n
        if self.model_type == "kikivik":
            n = 2 * self.vocab_size * d + d
            for e in self.mixers:
                m, mlp = e["mixer"], e.get("mlp")
                H, kd, vd = m["heads"], m["dim"], m["vdim"]
                if e["type"] == "attention":
                    n += d * (H * kd + m["kv_heads"] * (kd + vd)) + 2 * kd + (1 if m.get("v_mix") else 0)
                else:
                    R, Q, rd = m["kv_rank"], m["q_rank"], m["rot_dim"]
                    n += d * (Q + R + rd) + Q + R + H * (kd + rd) * Q + H * (kd + vd) * R
                n += d + H * vd * d
                if mlp and mlp["kind"] == "moe":
                    n += d + mlp["router"]["experts"] * (3 * d * mlp["expert"]["ff"] + d) + (3 * d * mlp["shared"]["ff"] if mlp.get("shared") else 0)
                elif mlp:
                    n += d + 3 * d * mlp["ff"]
            return n
        if self.model_type == "zonidra":
            n = 2 * self.vocab_size * d + d + ((self.bigram["buckets"] + 1) * d if self.bigram else 0)
            for e in self.mixers:
                m, mlp = e["mixer"], e.get("mlp")
                H, kd, vd = m["heads"], m["dim"], m["vdim"]
                n += d * (H * kd + 2 * H * vd + (m["kv_heads"] * (kd + vd) if m.get("kv_from") is None else 0)) + H + 4 * d
                if mlp and mlp["kind"] == "moe":
                    r, sh = mlp["router"], mlp.get("shared")
                    n += r["experts"] * 3 * d * mlp["expert"]["ff"] + (r["experts"] + r.get("identity", 0)) * (d + 1) + (3 * d * sh["ff"] + d if sh else 0)
                elif mlp:
                    n += 2 * d * mlp["ff"] + 4
                n += 3 * d if mlp else 0
            return n
        if self.mixers is not None:
            n = self.vocab_size * d + 2 * d + 1 + (self.layer_loop["times"] * d if self.layer_loop else 0)
            for e in self.mixers:
                m = e["mixer"]
                H, kd, vd = m["heads"], m["dim"], m["vdim"]
                if e["type"] == "latent_attention":
                    R, rd = m["kv_rank"], m["rot_dim"]
                    n += d * (H * (kd + rd) + R + rd + 2 * H * vd) + R + H * (kd + vd) * R
                else:
                    n += d * (2 * H * kd + 3 * H * vd)
                n += 2 * d * (e["mlp"]["ff"] if e.get("mlp") else 0) + 2 * d + 1
            return n
        if self.layers_block_type is not None:
            I, C, H = self.mamba_inner, self.mamba_conv_dim, self.mamba_num_heads
            din = self.moe_latent_size or d
            per = {"mamba": (I + C + H) * d + C * (self.mamba_d_conv + 1) + 3 * H + I + d * I,
                   "attention": d * self.qkv_size + self.q_size * d,
                   "mlp": 2 * d * self.intermediate_size,
                   "moe": self.num_experts * (2 * din * self.moe_intermediate_size + d) + 2 * d * self.moe_shared_expert_intermediate_size
                          + (2 * d * din if self.moe_latent_size else 0)}
            return sum(per[t] + d for t in self.layers_block_type) + self.vocab_size * d * (1 if self.tie_word_embeddings else 2) + d
        attn = d * self.qkv_size + self.q_size * d + (self.qkv_size if self.attention_bias else 0)
        if self.is_moe:
            ffn = self.num_experts * 3 * d * self.moe_intermediate_size + self.num_experts * d
        else:
            ffn = 3 * d * self.intermediate_size
        norms = 2 * d + (2 * self.head_dim if self.qk_norm else 0)
        emb = self.vocab_size * d * (1 if self.tie_word_embeddings else 2)
        return L * (attn + ffn + norms) + emb + d

    def to_hf_dict(self) -> dict:
        if self.model_type == "kikivik":
            return {"architecture": "Kikivik", "vocab": self.vocab_size, "width": self.hidden_size, "embedding": {"scale": self.embed_scale},
                    "norm": {"eps": self.rms_norm_eps}, "layers": self.mixers, "torch_dtype": self.torch_dtype}
        if self.model_type == "zonidra":
            emb = {"scale": self.embed_scale, **({"bigram": self.bigram} if self.bigram else {})}
            return {"architecture": "Zonidra", "vocab": self.vocab_size, "width": self.hidden_size, "embedding": emb,
                    "norm": {"eps": self.rms_norm_eps}, "layers": self.mixers, "torch_dtype": self.torch_dtype}
        if self.model_type == "redarax":
            out = {"architecture": "Redarax", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.rms_norm_eps},
                   "residual_mult": self.residual_mult, "logit_scale": self.logit_scale, "layers": self.mixers, "torch_dtype": self.torch_dtype}
            if self.token_side:
                out["token_side"] = self.token_side
            return dict(out, logit_softcap=self.final_logit_softcap) if self.final_logit_softcap else out
        if self.is_mixer:
            out = {"architecture": "Gadarax", "vocab": self.vocab_size, "width": self.hidden_size, "embedding": {"scale": self.embed_scale},
                   "norm": {"eps": self.rms_norm_eps}, "layers": self.mixers, "torch_dtype": self.torch_dtype}
            return dict(out, loop=self.layer_loop) if self.layer_loop else out
        arch = {"llama": "LlamaForCausalLM", "mistral": "MistralForCausalLM", "qwen2": "Qwen2ForCausalLM",
                "qwen3": "Qwen3ForCausalLM", "qwen3_moe": "Qwen3MoeForCausalLM",
                "gemma3_text": "Gemma3ForCausalLM", "deepseek_v3": "DeepseekV3ForCausalLM",
                "nemotron_h": "NemotronHForCausalLM"}.get(self.model_type, "LlamaForCausalLM")
        d = asdict(self)
        for k in ("mixers", "layer_loop", "norm_kind", "norm_place", "residual_mult", "token_side", "layer_scale", "token_shift", "bigram", "logit_scale", "traits"):
            d.pop(k)
        nh = {k: d.pop(k) for k in ("layers_block_type", "use_rope", "mlp_gated", "mlp_bias", "mamba_num_heads", "mamba_head_dim", "ssm_state_size",
                                    "mamba_n_groups", "mamba_d_conv", "mamba_chunk_size", "mamba_conv_bias", "mamba_proj_bias", "mamba_dt_limit",
                                    "moe_latent_size", "moe_shared_expert_intermediate_size")}
        if self.model_type == "nemotron_h":
            pat = "".join({"mamba": "M", "attention": "*", "mlp": "-", "moe": "E"}[t] for t in nh["layers_block_type"])
            d.update(hybrid_override_pattern=pat, layers_block_type=nh["layers_block_type"], mamba_num_heads=nh["mamba_num_heads"],
                     mamba_head_dim=nh["mamba_head_dim"], ssm_state_size=nh["ssm_state_size"], n_groups=nh["mamba_n_groups"],
                     conv_kernel=nh["mamba_d_conv"], chunk_size=nh["mamba_chunk_size"], use_conv_bias=nh["mamba_conv_bias"],
                     use_bias=nh["mamba_proj_bias"], mlp_bias=nh["mlp_bias"], mlp_hidden_act=d["hidden_act"], layer_norm_epsilon=d["rms_norm_eps"],
                     time_step_limit=nh["mamba_dt_limit"] or [0.0, float("inf")], moe_latent_size=nh["moe_latent_size"],
                     moe_shared_expert_intermediate_size=nh["moe_shared_expert_intermediate_size"], n_routed_experts=self.num_experts,
                     n_shared_experts=self.n_shared_experts, n_group=self.n_group, topk_group=self.topk_group,
                     routed_scaling_factor=self.routed_scaling_factor)
        d.pop("value_head")
        d.pop("qk_norm")
        gem = {k: d.pop(k) for k in ("hidden_act", "sandwich_norm", "embed_scale", "norm_offset", "sliding_window", "layer_types",
                                     "rope_local_theta", "attn_scale", "final_logit_softcap")}
        if self.model_type == "gemma3_text":
            d.update(hidden_activation=gem["hidden_act"], sliding_window=gem["sliding_window"], layer_types=gem["layer_types"],
                     rope_local_base_freq=gem["rope_local_theta"], query_pre_attn_scalar=round(gem["attn_scale"] ** -2) if gem["attn_scale"] else self.head_dim,
                     final_logit_softcapping=gem["final_logit_softcap"] or None)
        d["architectures"] = [arch]
        if self.vision is None:
            d.pop("vision")
            d.pop("image_token_id")
        ds = {k: d.pop(k) for k in ("kv_lora_rank", "q_lora_rank", "qk_nope_head_dim", "qk_rope_head_dim", "v_head_dim", "rope_interleave",
                                    "n_shared_experts", "first_k_dense_replace", "scoring_func", "n_group", "topk_group", "routed_scaling_factor")}
        if self.model_type == "nemotron_h":
            d.update({k: ds[k] for k in ("n_shared_experts", "n_group", "topk_group", "routed_scaling_factor")})
        if self.model_type == "deepseek_v3":
            d.update(ds, n_routed_experts=self.num_experts)
            d.pop("num_experts")
            d.pop("head_dim")
        if not self.is_moe:
            for k in ("num_experts", "num_experts_per_tok", "moe_intermediate_size", "norm_topk_prob", "router_aux_loss_coef"):
                d.pop(k, None)
        return d

    @classmethod
    def from_hf_dict(cls, hf: dict, **overrides) -> "ModelConfig":
        if hf.get("architecture") in LAYER_LISTS:
            return cls._from_layer_list(hf, **overrides)
        mt = hf.get("model_type", "llama")
        if mt == "gemma3" and "text_config" in hf:      # the multimodal wrapper: the language model's settings are nested
            hf = dict(hf["text_config"], model_type="gemma3_text")
            mt = "gemma3_text"
        n_heads = hf["num_attention_heads"]
        if mt == "nemotron_h":
            hf = dict(hf)
            types = hf.get("layers_block_type")
            if types is None:    # older configs: one character per layer (M mamba, * attention, - MLP, E mixture of experts)
                types = [{"M": "mamba", "*": "attention", "-": "mlp", "E": "moe"}[ch] for ch in hf["hybrid_override_pattern"]]
            hf["layers_block_type"] = list(types)
            hf["num_hidden_layers"] = len(types)
            hf.setdefault("rms_norm_eps", hf.get("layer_norm_epsilon", 1e-5))
        cfg = cls(
            model_type=mt,
            vocab_size=hf["vocab_size"],
            hidden_size=hf["hidden_size"],
            intermediate_size=hf.get("intermediate_size", 0),
            num_hidden_layers=hf["num_hidden_layers"],
            num_attention_heads=n_heads,
            num_key_value_heads=hf.get("num_key_value_heads", n_heads),
            head_dim=hf.get("head_dim") or hf["hidden_size"] // n_heads,
            rms_norm_eps=hf.get("rms_norm_eps", 1e-5),
            rope_theta=float(hf.get("rope_theta", 10000.0)),
            rope_scaling=hf.get("rope_scaling"),
            max_position_embeddings=hf.get("max_position_embeddings", 131072),
            tie_word_embeddings=bool(hf.get("tie_word_embeddings", False)),
            attention_bias=bool(hf.get("attention_bias", mt == "qwen2")),
            qk_norm=mt in ("qwen3", "qwen3_moe", "gemma3_text"),
            num_experts=((hf.get("num_experts") or hf.get("num_local_experts") or 0) if mt.endswith("_moe")     # (newer HF configs: num_local_experts)
                         else (hf.get("n_routed_experts") or 0) if mt == "deepseek_v3"
                         else (hf.get("n_routed_experts") or 0) if (mt == "nemotron_h" and "moe" in hf["layers_block_type"]) else 0),
            num_experts_per_tok=hf.get("num_experts_per_tok", 0),
            moe_intermediate_size=hf.get("moe_intermediate_size", 0),
            norm_topk_prob=bool(hf.get("norm_topk_prob", True)),
            router_aux_loss_coef=float(hf.get("router_aux_loss_coef", 0.0)),
            bos_token_id=hf.get("bos_token_id"),
            eos_token_id=hf.get("eos_token_id"),
            pad_token_id=hf.get("pad_token_id"),
            torch_dtype=str(hf.get("torch_dtype") or hf.get("dtype") or "bfloat16").replace("torch.", ""),
            vision=hf.get("vision"),
            image_token_id=hf.get("image_token_id"),
        )
        if mt == "deepseek_v3":
            for k in ("kv_lora_rank", "q_lora_rank", "qk_nope_head_dim", "qk_rope_head_dim", "v_head_dim", "n_shared_experts",
                      "first_k_dense_replace", "n_group", "topk_group", "routed_scaling_factor"):
                if hf.get(k) is not None or k == "q_lora_rank":
                    setattr(cfg, k, hf.get(k))
            cfg.rope_interleave = bool(hf.get("rope_interleave", True))
            cfg.scoring_func = hf.get("scoring_func", "sigmoid")
            cfg.num_key_value_heads = cfg.num_attention_heads       # after decompression every head has its own keys and values
            cfg.head_dim = cfg.qk_nope_head_dim + cfg.qk_rope_head_dim   # what the attention kernels and the KV cache see (V is padded to it)
            rp = hf.get("rope_parameters") or hf.get("rope_scaling") or {}
            if isinstance(rp, dict) and rp.get("rope_type", rp.get("type", "default")) != "default":
                cfg.rope_scaling = {k: v for k, v in rp.items() if k != "rope_theta"}
                cfg.rope_theta = float(rp.get("rope_theta", cfg.rope_theta))
                m_all = float(rp.get("mscale_all_dim", 0) or 0)
                if m_all and float(rp["factor"]) > 1:      # the long-context recipe also sharpens the soft-max
                    ms = 0.1 * m_all * math.log(float(rp["factor"])) + 1.0
                    cfg.attn_scale = cfg.head_dim ** -0.5 * ms * ms
            elif isinstance(rp, dict) and rp.get("rope_theta"):
                cfg.rope_theta = float(rp["rope_theta"])
        if mt == "nemotron_h":
            cfg.layers_block_type = hf["layers_block_type"]
            cfg.use_rope, cfg.mlp_gated = False, False
            cfg.hidden_act = hf.get("mlp_hidden_act", "relu2")
            cfg.mlp_bias = bool(hf.get("mlp_bias", False))
            cfg.mamba_num_heads, cfg.mamba_head_dim = hf["mamba_num_heads"], hf["mamba_head_dim"]
            cfg.ssm_state_size = hf.get("ssm_state_size", 128)
            cfg.mamba_n_groups = hf.get("mamba_n_groups", hf.get("n_groups", 8))
            cfg.mamba_d_conv = hf.get("mamba_d_conv", hf.get("conv_kernel", 4))
            cfg.mamba_chunk_size = hf.get("mamba_chunk_size", hf.get("chunk_size", 128))
            cfg.mamba_conv_bias = bool(hf.get("mamba_conv_bias", hf.get("use_conv_bias", True)))
            cfg.mamba_proj_bias = bool(hf.get("mamba_proj_bias", hf.get("use_bias", False)))
            lim = hf.get("mamba_dt_limit", hf.get("time_step_limit"))
            cfg.mamba_dt_limit = [float(lim[0]), float(lim[1])] if lim is not None else None
            if cfg.is_moe:
                for k in ("n_shared_experts", "n_group", "topk_group", "routed_scaling_factor", "moe_latent_size"):
                    if hf.get(k) is not None:
                        setattr(cfg, k, hf[k])
                cfg.scoring_func = "sigmoid"
                cfg.moe_shared_expert_intermediate_size = hf.get("moe_shared_expert_intermediate_size", 0) or 0
        if mt == "gemma3_text":
            L = cfg.num_hidden_layers
            pattern = int(hf.get("sliding_window_pattern", 6) or 6)
            cfg.hidden_act = hf.get("hidden_activation", "gelu_pytorch_tanh")
            cfg.sandwich_norm, cfg.norm_offset = True, 1.0
            cfg.embed_scale = float(cfg.hidden_size) ** 0.5
            cfg.sliding_window = int(hf.get("sliding_window") or 0)
            cfg.layer_types = list(hf.get("layer_types") or ["sliding_attention" if (i + 1) % pattern else "full_attention" for i in range(L)])
            cfg.rope_local_theta = float(hf.get("rope_local_base_freq", 10000.0))
            cfg.attn_scale = float(hf.get("query_pre_attn_scalar", cfg.head_dim)) ** -0.5
            cfg.final_logit_softcap = float(hf.get("final_logit_softcapping") or 0.0)
            cfg.tie_word_embeddings = bool(hf.get("tie_word_embeddings", True))
            cfg.rms_norm_eps = hf.get("rms_norm_eps", 1e-6)
            rp = hf.get("rope_parameters")    # newer configs nest the RoPE settings per layer type
            if isinstance(rp, dict) and "full_attention" in rp:
                full, loc = rp["full_attention"], rp.get("sliding_attention", {})
                cfg.rope_theta = float(full.get("rope_theta", cfg.rope_theta))
                cfg.rope_scaling = {k: v for k, v in full.items() if k != "rope_theta"} if full.get("rope_type", "default") != "default" else None
                cfg.rope_local_theta = float(loc.get("rope_theta", cfg.rope_local_theta))
        for k, v in overrides.items():
            setattr(cfg, k, v)
        return cfg

    @classmethod
    def _from_layer_list(cls, hf: dict, **overrides) -> "ModelConfig":
        """Configurations that describe the model layer by layer (``LAYER_LISTS``)."""
        layers, (mixers, mlps, settings) = hf["layers"], LAYER_LISTS[hf["architecture"]]
        for i, e in enumerate(layers):
            need = MIXER_SIZES[e["type"]] if e["type"] in mixers else None
            if need is None:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            need = need + (("q_rank",) if hf["architecture"] == "Kikivik" and e["type"] == "latent_attention" else ())
            missing = [k for k in need if k not in e["mixer"]]
            if missing:
                raise ValueError(f"layer {i}: the {e['type']} mixer lacks {missing}")
            if e.get("mlp") and e["mlp"].get("kind", "dense") not in mlps:
                raise ValueError(f"layer {i}: unknown MLP kind {e['mlp']['kind']!r}")
            _check_mixer(i, e["type"], e["mixer"])
            if e.get("mlp") and e["mlp"].get("kind") == "moe":
                r = e["mlp"]["router"]
                g = r.get("groups") or {"count": 1, "keep": 1}
                n = r["experts"] + r.get("identity", 0)
                if n % g["count"] or not 1 <= g["keep"] <= g["count"] or not 1 <= r["top"] <= g["keep"] * (n // g["count"]):
                    raise ValueError(f"layer {i}: router {r} does not fit its groups")
            _check_source(i, layers)
        mixing = {(e["mixer"]["kv_heads"], e["mixer"]["vdim"]) for e in layers if e["type"] == "attention" and e["mixer"].get("v_mix")}
        if len(mixing) > 1:
            raise ValueError(f"layers that mix their values have unequal (key / value heads, value sizes): {sorted(mixing)}")
        lp = hf.get("loop")
        if lp and not (0 <= lp["start"] < lp["stop"] <= len(layers) and lp["times"] >= 1):
            raise ValueError(f"layer loop {lp} does not fit {len(layers)} layers")
        m0 = layers[0]["mixer"]
        cfg = cls(vocab_size=hf["vocab"], hidden_size=hf["width"], num_hidden_layers=len(layers),
                  intermediate_size=max([_ff_width(e["mlp"]) for e in layers if e.get("mlp")] or [0]), num_attention_heads=m0["heads"],
                  num_key_value_heads=m0["heads"], head_dim=m0.get("dim", m0["vdim"]), rms_norm_eps=float(hf["norm"]["eps"]), mixers=layers,
                  layer_loop=dict(lp) if lp else None, torch_dtype=str(hf.get("torch_dtype", "bfloat16")).replace("torch.", ""), **settings(hf))
        for k, v in overrides.items():
            setattr(cfg, k, v)
        return cfg

    @classmethod
    def from_pretrained(cls, path: str, **overrides) -> "ModelConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls.from_hf_dict(json.load(f), **overrides)

    def save_pretrained(self, path: str) -> None:
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.to_hf_dict(), f, indent=2)


# what a mixer's description must name
MIXER_SIZES = {
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot"),
    "retention": ("heads", "dim", "vdim", "decay", "rot"),
    "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "rot"),
    "mamba2": ("heads", "vdim", "state", "groups", "norm_groups", "conv"),
    "delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
}
RECURRENT_MIXERS = ("retention", "mamba2", "delta")


def _check_mixer(i: int, kind: str, m: dict) -> None:
    if kind == "retention" and len(m["decay"]) != m["heads"]:
        raise ValueError(f"layer {i}: {len(m['decay'])} decays for {m['heads']} heads")
    if "rot" in m:
        limit = m["rot_dim"] if kind == "latent_attention" else m["dim"]
        if m["rot"]["dims"] > limit or m["rot"]["dims"] % 2:
            raise ValueError(f"layer {i}: {m['rot']['dims']} rotated dimensions in a part of {limit}")
    for part in ("kv_heads", "groups"):
        if part in m and m["heads"] % m[part]:
            raise ValueError(f"layer {i}: {m['heads']} heads do not divide into {m[part]} {part}")
    if "norm_groups" in m and (m["heads"] * m["vdim"]) % m["norm_groups"]:
        raise ValueError(f"layer {i}: {m['heads'] * m['vdim']} channels do not divide into {m['norm_groups']} norm groups")
    if m.get("conv", 1) < 1:
        raise ValueError(f"layer {i}: a convolution needs at least one tap")
    if m.get("mask") and (m["mask"]["size"] < 1 or m["mask"].get("keep_first", 0) < 0):
        raise ValueError(f"layer {i}: mask {m['mask']}")


def _check_source(i: int, layers: list) -> None:
    """A layer that reads another layer's keys and values comes behind it and has its key / value heads and sizes."""
    m = layers[i]["mixer"]
    j = m.get("kv_from")
    if j is None:
        return
    if not 0 <= j < i or layers[j]["type"] != "attention" or layers[j]["mixer"].get("kv_from") is not None:
        raise ValueError(f"layer {i}: layer {j} has no keys and values to share")
    unequal = [k for k in ("kv_heads", "dim", "vdim") if m.get(k) != layers[j]["mixer"].get(k)]
    if unequal:
        raise ValueError(f"layer {i}: {unequal} differ from those of layer {j}, whose keys and values it reads")


def _ff_width(mlp: dict) -> int:
    return mlp["expert"]["ff"] if mlp.get("kind") == "moe" else mlp["ff"]


def _gadarax(hf: dict) -> dict:
    return dict(model_type="gadarax", tie_word_embeddings=True, mlp_gated=False, hidden_act="relu2", embed_scale=float(hf["embedding"]["scale"]), norm_kind="dyt")


def _redarax(hf: dict) -> dict:
    return dict(model_type="redarax", norm_place="post", residual_mult=float(hf["residual_mult"]), logit_scale=float(hf["logit_scale"]),
                final_logit_softcap=float(hf.get("logit_softcap") or 0.0), token_side=dict(hf["token_side"]) if hf.get("token_side") else None)


KIKIVIK_TRAITS = {"latent_attention": {"gate": False, "interleaved": False}, "attention": {"bias": False, "interleaved": False},
                  "moe": {"weigh_input": True, "corrected": False}}


def _kikivik(hf: dict) -> dict:
    return dict(model_type="kikivik", embed_scale=float(hf["embedding"]["scale"]), traits=KIKIVIK_TRAITS)


ZONIDRA_TRAITS = {"attention": {"bias": False, "qk_norm": False, "interleaved": False, "gate": True, "weights": "sigmoid", "mask_kind": "window"},
                  "dense": {"act": "poly"}, "moe": {"score": "softmax", "shared_gate": True}}


def _zonidra(hf: dict) -> dict:
    big = hf["embedding"].get("bigram")
    return dict(model_type="zonidra", embed_scale=float(hf["embedding"]["scale"]), norm_place="both", layer_scale=True, token_shift=True,
                bigram={k: int(big[k]) for k in ("buckets", "mul_prev", "mul_cur")} if big else None, traits=ZONIDRA_TRAITS)


# architecture -> (its mixers, its kinds of MLP, configuration -> further ModelConfig fields)
LAYER_LISTS = {"Gadarax": (("latent_attention", "retention"), ("dense",), _gadarax),
               "Redarax": (("attention", "mamba2", "delta"), ("dense", "moe"), _redarax),
               "Kikivik": (("latent_attention", "attention"), ("dense", "moe"), _kikivik),
               "Zonidra": (("attention",), ("dense", "moe"), _zonidra)}


def rope_inv_freq(cfg: ModelConfig, device=None) -> torch.Tensor:
    """Inverse frequencies [head_dim/2] including the ``llama3`` / ``linear`` / ``yarn`` scaling rules."""
    D = cfg.qk_rope_head_dim if cfg.is_mla else cfg.head_dim     # MLA rotates only the decoupled rotary part of each head
    if not cfg.use_rope:   # a rotation by angle zero: the attention code paths stay the same
        z = torch.zeros(D // 2, dtype=torch.float32)
        return z.to(device) if device is not None else z
    inv = 1.0 / (cfg.rope_theta ** (torch.arange(0, D, 2, dtype=torch.float32) / D))
    rs = cfg.rope_scaling or {}
    kind = rs.get("rope_type", rs.get("type", "default"))
    if kind == "linear":
        inv = inv / float(rs["factor"])
    elif kind == "llama3":
        factor, lo_f, hi_f = rs["factor"], rs.get("low_freq_factor", 1.0), rs.get("high_freq_factor", 4.0)
        old = rs.get("original_max_position_embeddings", 8192)
        wavelen = 2 * math.pi / inv
        smooth = ((old / wavelen) - lo_f) / (hi_f - lo_f)
        scaled = torch.where(wavelen > old / lo_f, inv / factor, inv)
        mid = (1 - smooth) * inv / factor + smooth * inv
        is_mid = (wavelen <= old / lo_f) & (wavelen >= old / hi_f)
        inv = torch.where(is_mid, mid, scaled)
    elif kind == "yarn":
        factor = float(rs["factor"])
        old = rs.get("original_max_position_embeddings", cfg.max_position_embeddings)
        beta_fast, beta_slow = rs.get("beta_fast", 32.0), rs.get("beta_slow", 1.0)

        def corr_dim(rot):
            return (D * math.log(old / (rot * 2 * math.pi))) / (2 * math.log(cfg.rope_theta))

        lo = max(math.floor(corr_dim(beta_fast)), 0)
        hi = min(math.ceil(corr_dim(beta_slow)), D // 2 - 1)
        ramp = ((torch.arange(D // 2, dtype=torch.float32) - lo) / max(hi - lo, 1e-3)).clamp(0, 1)
        inv = inv / factor * ramp + inv * (1 - ramp)
    return inv.to(device) if device is not None else inv


def rotary_table(rot: dict) -> tuple[torch.Tensor, float]:
    """Angle per position of each rotated pair [dims / 2] (fp32) and the factor on cosine and sine, for a rotation described by
    ``{"dims", "base"}`` and optionally ``"scaling"``: ``{"factor"}`` alone slows every pair down by ``factor``, Llama 3.1's ``{"factor",
    "original", "low", "high"}`` keeps pairs that turn more than ``high`` times within the original context, slows down by ``factor`` those that
    turn less than ``low`` times and mixes the two linearly in the turns between them, YaRN's ``{"factor",
    "original", "fast", "slow"}`` keeps the frequency of pairs that turn more than ``fast`` times within the original context and slows
    down by ``factor`` those that turn less than ``slow`` times, with a linear ramp between the two (upper end clamped at the last
    dimension)."""
    n, base = int(rot["dims"]), float(rot["base"])
    f = base ** (-2.0 * torch.arange(n // 2, dtype=torch.float64) / n) if n else torch.zeros(0, dtype=torch.float64)
    s = rot.get("scaling")
    if not s:
        return f.float(), 1.0
    factor = float(s["factor"])
    if "original" not in s:
        return (f / factor).float(), 1.0

    if "low" in s:
        turns, lo, hi = float(s["original"]) * f / (2 * math.pi), float(s["low"]), float(s["high"])
        t = ((turns - lo) / (hi - lo)).clamp(0, 1) if hi > lo else (turns >= lo).double()
        return ((1 - t) * f / factor + t * f).float(), 1.0

    def dim_of(turns):
        return n * math.log(float(s["original"]) / (2 * math.pi * float(turns))) / (2 * math.log(base))

    lo, hi = max(math.floor(dim_of(s["fast"])), 0), min(math.ceil(dim_of(s["slow"])), n - 1)
    ramp = ((torch.arange(n // 2, dtype=torch.float64) - lo) / max(hi - lo, 1e-3)).clamp(0, 1)
    return (f / factor * ramp + f * (1 - ramp)).float(), 0.1 * math.log(factor) + 1.0


def _layer_list(width: int, ff: int, latent: dict, retention: dict, kinds: str, loop: Optional[dict], vocab: int) -> dict:
    """Preset of a layer-list model: ``kinds`` has one letter per layer (A latent attention, R retention)."""
    rot = {"dims": latent["rot_dim"], "base": 500000.0, "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}}
    att = dict(latent, scale=(latent["dim"] + latent["rot_dim"]) ** -0.5, rot=rot)
    ret = dict(retention, rot={"dims": retention["dim"], "base": 10000.0},
               decay=[1.0 - 2.0 ** -(5 + 7 * i / max(1, retention["heads"] - 1)) for i in range(retention["heads"])])
    layers = [{"type": "latent_attention" if k == "A" else "retention", "mixer": att if k == "A" else ret, "mlp": {"kind": "dense", "ff": ff}} for k in kinds]
    return dict(model_type="gadarax", vocab_size=vocab, hidden_size=width, intermediate_size=ff, num_hidden_layers=len(layers),
                num_attention_heads=latent["heads"], num_key_value_heads=latent["heads"], head_dim=latent["dim"], rms_norm_eps=1e-6,
                tie_word_embeddings=True, mlp_gated=False, hidden_act="relu2", embed_scale=float(width) ** 0.5, norm_kind="dyt", mixers=layers,
                layer_loop=loop)


def _redarax_preset(width: int, kinds: str, attention: dict, mamba2: dict, delta: dict, ff: int, moe: dict, side: int, vocab: int) -> dict:
    """Preset of a post-norm layer-list model: ``kinds`` has two letters per layer, the mixer (A attention, M Mamba-2, D delta rule) and the
    feed-forward (d dense, e experts, - none)."""
    mix = {"A": ("attention", dict(attention, scale=attention["dim"] ** -0.5)), "M": ("mamba2", mamba2), "D": ("delta", delta)}
    mlp = {"d": {"kind": "dense", "ff": ff, "limit": 7.0}, "e": dict(moe, kind="moe"), "-": None}
    layers = [{"type": mix[k][0], "mixer": mix[k][1], "mlp": mlp[f]} for k, f in zip(kinds[::2], kinds[1::2])]
    m0 = layers[0]["mixer"]
    return dict(model_type="redarax", vocab_size=vocab, hidden_size=width, num_hidden_layers=len(layers), intermediate_size=max(ff, moe["expert"]["ff"]),
                num_attention_heads=m0["heads"], num_key_value_heads=m0["heads"], head_dim=m0.get("dim", m0["vdim"]), rms_norm_eps=1e-6, mixers=layers,
                norm_place="post", residual_mult=0.5, logit_scale=0.5, final_logit_softcap=30.0, token_side={"dim": side} if side else None)


def _kikivik_preset(width: int, kinds: str, latent: dict, attention: dict, ff: int, moe: dict, vocab: int) -> dict:
    """Preset of a pre-norm layer-list model: ``kinds`` has two letters per layer, the mixer (L latent attention, A chunked attention) and the
    feed-forward (d dense, e experts, - none)."""
    mix = {"L": ("latent_attention", dict(latent, scale=(latent["dim"] + latent["rot_dim"]) ** -0.5, rot={"dims": latent["rot_dim"], "base": 5e5})),
           "A": ("attention", dict(attention, scale=attention["dim"] ** -0.5, v_mix=True))}
    mlp = {"d": {"kind": "dense", "ff": ff, "limit": 7.0}, "e": dict(moe, kind="moe"), "-": None}
    layers = [{"type": mix[k][0], "mixer": mix[k][1], "mlp": mlp[f]} for k, f in zip(kinds[::2], kinds[1::2])]
    m0 = layers[0]["mixer"]
    return dict(model_type="kikivik", vocab_size=vocab, hidden_size=width, num_hidden_layers=len(layers), intermediate_size=max(ff, moe["expert"]["ff"]),
                num_attention_heads=m0["heads"], num_key_value_heads=m0["heads"], head_dim=m0["dim"], rms_norm_eps=1e-6, mixers=layers,
                embed_scale=2.0, traits=KIKIVIK_TRAITS)


def _zonidra_preset(width: int, kinds: str, attention: dict, ff: int, moe: dict, bigram: dict, vocab: int) -> dict:
    """Preset of a layer-list model with norms on both sides of its sublayers: ``kinds`` has two letters per layer, the attention (A with keys and
    values of its own, S with those of the layer before it that has some) and the feed-forward (d dense, e experts, - none)."""
    rot = {"dims": attention["dim"], "base": 5e5, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    att = dict(attention, scale=attention["dim"] ** -0.5, rot=attention.get("rot", rot))
    mlp = {"d": {"kind": "dense", "ff": ff}, "e": dict(moe, kind="moe"), "-": None}
    layers, source = [], 0
    for i, (k, f) in enumerate(zip(kinds[::2], kinds[1::2])):
        source = i if k == "A" else source
        layers.append({"type": "attention", "mixer": dict(att, kv_from=source) if k == "S" else att, "mlp": mlp[f]})
    return dict(model_type="zonidra", vocab_size=vocab, hidden_size=width, num_hidden_layers=len(layers), intermediate_size=max(ff, moe["expert"]["ff"]),
                num_attention_heads=att["heads"], num_key_value_heads=att["heads"], head_dim=att["dim"], rms_norm_eps=1e-6, mixers=layers,
                embed_scale=float(width) ** 0.5, norm_place="both", layer_scale=True, token_shift=True, bigram=bigram, traits=ZONIDRA_TRAITS)


PRESETS: dict[str, dict] = {
    # Zonidra at the size of small production models: windowed sigmoid attention, every second layer on another's keys and values
    "zonidra-2b": _zonidra_preset(2048, "AdSeAeSeAdSeAeSe", dict(heads=16, kv_heads=4, dim=128, vdim=128, mask={"size": 1024, "keep_first": 64}), 8192,
                                  dict(expert={"ff": 768}, router={"experts": 64, "identity": 8, "top": 8, "scale": 2.5}, shared={"ff": 768}),
                                  {"buckets": 65521, "mul_prev": 40503, "mul_cur": 1}, 65536),
    "zonidra-7b": _zonidra_preset(4096, "AdSeAeSeAdSeAeSe", dict(heads=32, kv_heads=8, dim=128, vdim=128, mask={"size": 1024, "keep_first": 64}), 16384,
                                  dict(expert={"ff": 1536}, router={"experts": 64, "identity": 8, "top": 8, "scale": 2.5}, shared={"ff": 1536}),
                                  {"buckets": 65521, "mul_prev": 40503, "mul_cur": 1}, 65536),
    "tiny-zonidra": _zonidra_preset(96, "AeSdAdS-", dict(heads=4, kv_heads=2, dim=24, vdim=16, mask={"size": 20, "keep_first": 3},
                                                         rot={"dims": 16, "base": 1e4, "scaling": {"factor": 2.0, "low": 1.0, "high": 3.0, "original": 64}}),
                                    160, dict(expert={"ff": 48}, router={"experts": 6, "identity": 2, "top": 3, "scale": 1.5}, shared={"ff": 40}),
                                    {"buckets": 97, "mul_prev": 31, "mul_cur": 5}, 264),
    # Kikivik at the size of small production models: latent and chunked attention layers, dense and expert feed-forwards
    "kikivik-2b": _kikivik_preset(2048, "AdLeLdAeLeLdAeLe", dict(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=768),
                                  dict(heads=16, kv_heads=4, dim=128, vdim=128, mask={"size": 1024}, rot={"dims": 128, "base": 1e6, "scaling": {"factor": 4.0}}),
                                  6144, dict(expert={"ff": 768}, router={"experts": 64, "top": 8}, shared={"ff": 768}), 65536),
    "kikivik-7b": _kikivik_preset(4096, "AdLeLdAeLeLdAeLe", dict(heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=1536),
                                  dict(heads=32, kv_heads=8, dim=128, vdim=128, mask={"size": 1024}, rot={"dims": 128, "base": 1e6, "scaling": {"factor": 4.0}}),
                                  12288, dict(expert={"ff": 1536}, router={"experts": 64, "top": 8}, shared={"ff": 1536}), 65536),
    "tiny-kikivik": _kikivik_preset(96, "AeLdAdL-", dict(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, q_rank=48),
                                    dict(heads=4, kv_heads=2, dim=24, vdim=16, mask={"size": 20}, rot={"dims": 16, "base": 1e4, "scaling": {"factor": 2.0}}),
                                    160, dict(expert={"ff": 48}, router={"experts": 8, "top": 2}, shared={"ff": 40}), 264),
    # Redarax at the size of small production models: delta-rule, Mamba-2 and grouped-query attention layers, dense and expert feed-forwards
    "redarax-2b": _redarax_preset(2048, "DdDeMeAeDdDeMeAe", dict(heads=16, kv_heads=4, dim=128, vdim=128, rot={"dims": 64, "base": 1e6}),
                                  dict(heads=32, vdim=128, state=128, groups=4, norm_groups=4, conv=4), dict(heads=16, kv_heads=8, dim=128, vdim=128, conv=4),
                                  6144, dict(expert={"ff": 768, "limit": 7.0}, router={"experts": 64, "top": 8, "groups": {"count": 8, "keep": 4}}), 256, 65536),
    "redarax-7b": _redarax_preset(4096, "DdDeMeAeDdDeMeAe", dict(heads=32, kv_heads=8, dim=128, vdim=128, rot={"dims": 64, "base": 1e6}),
                                  dict(heads=64, vdim=128, state=128, groups=8, norm_groups=8, conv=4), dict(heads=32, kv_heads=16, dim=128, vdim=128, conv=4),
                                  12288, dict(expert={"ff": 1536, "limit": 7.0}, router={"experts": 64, "top": 8, "groups": {"count": 8, "keep": 4}}), 256, 65536),
    "tiny-redarax": _redarax_preset(96, "MeDdAeD-", dict(heads=4, kv_heads=2, dim=24, vdim=16, rot={"dims": 16, "base": 1e4}),
                                    dict(heads=6, vdim=16, state=24, groups=2, norm_groups=3, conv=3), dict(heads=4, kv_heads=2, dim=16, vdim=24, conv=4),
                                    160, dict(expert={"ff": 48, "limit": 2.0}, router={"experts": 8, "top": 2, "groups": {"count": 4, "keep": 2}}), 8, 264),
    # Gadarax at the size of small production models: latent attention and retention layers, three of them looped twice
    "gadarax-1b": _layer_list(2048, 8192, dict(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512), dict(heads=16, dim=128, vdim=128),
                              "AARARARARARA", dict(start=1, stop=4, times=2), 65536),
    "gadarax-4b": _layer_list(4096, 16384, dict(heads=32, dim=128, rot_dim=64, vdim=128, kv_rank=512), dict(heads=16, dim=256, vdim=256),
                              "AARARARARARA", dict(start=1, stop=4, times=2), 65536),
    "tiny-gadarax": _layer_list(96, 160, dict(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40), dict(heads=4, dim=24, vdim=16), "ARAR",
                                dict(start=1, stop=3, times=2), 264),
    # Llama-3.1-8B: 32 layers, d 4096, GQA 32q/8kv, SwiGLU 14336, vocab 128256, RoPE theta 5e5 (llama3 scaling)
    "llama3.1-8b": dict(model_type="llama", vocab_size=128256, hidden_size=4096, intermediate_size=14336,
                        num_hidden_layers=32, num_attention_heads=32, num_key_value_heads=8, head_dim=128,
                        rms_norm_eps=1e-5, rope_theta=500000.0,
                        rope_scaling=dict(rope_type="llama3", factor=8.0, low_freq_factor=1.0, high_freq_factor=4.0,
                                          original_max_position_embeddings=8192),
                        bos_token_id=128000, eos_token_id=128001),
    "llama3.2-1b": dict(model_type="llama", vocab_size=128256, hidden_size=2048, intermediate_size=8192,
                        num_hidden_layers=16, num_attention_heads=32, num_key_value_heads=8, head_dim=64,
                        rms_norm_eps=1e-5, rope_theta=500000.0, tie_word_embeddings=True,
                        rope_scaling=dict(rope_type="llama3", factor=32.0, low_freq_factor=1.0, high_freq_factor=4.0,
                                          original_max_position_embeddings=8192)),
    "qwen3-32b": dict(model_type="qwen3", vocab_size=151936, hidden_size=5120, intermediate_size=25600,
                      num_hidden_layers=64, num_attention_heads=64, num_key_value_heads=8, head_dim=128,
                      rms_norm_eps=1e-6, rope_theta=1000000.0, qk_norm=True),
    "qwen3-30b-a3b": dict(model_type="qwen3_moe", vocab_size=151936, hidden_size=2048, intermediate_size=6144,
                          num_hidden_layers=48, num_attention_heads=32, num_key_value_heads=4, head_dim=128,
                          rms_norm_eps=1e-6, rope_theta=1000000.0, qk_norm=True, num_experts=128,
                          num_experts_per_tok=8, moe_intermediate_size=768, norm_topk_prob=True),
    "qwen2.5-0.5b": dict(model_type="qwen2", vocab_size=151936, hidden_size=896, intermediate_size=4864,
                         num_hidden_layers=24, num_attention_heads=14, num_key_value_heads=2, head_dim=64,
                         rms_norm_eps=1e-6, rope_theta=1000000.0, attention_bias=True, tie_word_embeddings=True),
    # the CPU/gloo oracle model: 4 layers, d 256, 4 heads, SwiGLU 688, vocab 2048
    # Gemma-3-1B (text): 26 layers, d 1152, 4 q / 1 kv heads of 256, GeGLU 6912, five sliding-window (512) layers per global one
    "gemma3-1b": dict(model_type="gemma3_text", vocab_size=262144, hidden_size=1152, intermediate_size=6912, num_hidden_layers=26,
                      num_attention_heads=4, num_key_value_heads=1, head_dim=256, rms_norm_eps=1e-6, rope_theta=1000000.0,
                      tie_word_embeddings=True, qk_norm=True, hidden_act="gelu_pytorch_tanh", sandwich_norm=True, embed_scale=1152 ** 0.5,
                      norm_offset=1.0, sliding_window=512, rope_local_theta=10000.0, attn_scale=256 ** -0.5,
                      layer_types=["full_attention" if (i + 1) % 6 == 0 else "sliding_attention" for i in range(26)]),
    "tiny-llama-oracle": dict(model_type="llama", vocab_size=2048, hidden_size=256, intermediate_size=688,
                              num_hidden_layers=4, num_attention_heads=4, num_key_value_heads=4, head_dim=64,
                              rms_norm_eps=1e-5, rope_theta=10000.0),
    # tiny hybrid model for offline recipes and tests: Mamba-2, MLP, attention and expert blocks
    "tiny-nemotron-h": dict(model_type="nemotron_h", vocab_size=2048, hidden_size=256, intermediate_size=512, num_hidden_layers=6,
                            layers_block_type=["mamba", "mlp", "mamba", "attention", "mamba", "moe"], num_attention_heads=4,
                            num_key_value_heads=2, head_dim=64, rms_norm_eps=1e-5, use_rope=False, mlp_gated=False, hidden_act="relu2",
                            mamba_num_heads=8, mamba_head_dim=64, ssm_state_size=32, mamba_n_groups=2, mamba_chunk_size=64,
                            num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128, n_shared_experts=1,
                            moe_shared_expert_intermediate_size=256, scoring_func="sigmoid"),
    # Nemotron-Nano-12B-v2-shaped (Mamba-2 / MLP blocks with six attention blocks; the reference's grpo-nano-v2-12b recipes)
    "nemotron-nano-12b-v2": dict(model_type="nemotron_h", vocab_size=131072, hidden_size=5120, intermediate_size=20480, num_hidden_layers=62,
                                 layers_block_type=[{"M": "mamba", "-": "mlp", "*": "attention"}[ch] for ch in
                                                    "M-M-M-M*-M-M-M-M*-M-M-M-M*-M-M-M-M*-M-M-M-M*-M-M-M-M*-M-M-M-M-"],
                                 num_attention_heads=40, num_key_value_heads=8, head_dim=128, rms_norm_eps=1e-5, use_rope=False,
                                 mlp_gated=False, hidden_act="relu2", mamba_num_heads=128, mamba_head_dim=80, ssm_state_size=128,
                                 mamba_n_groups=8, mamba_chunk_size=128),
    # Nemotron-3-Nano-30B-A3B-shaped (Mamba-2 / expert blocks with six attention blocks; the reference's grpo-nanov3 recipes)
    "nemotron-nano-30b-a3b-v3": dict(model_type="nemotron_h", vocab_size=131072, hidden_size=2688, intermediate_size=1856, num_hidden_layers=52,
                                     layers_block_type=[{"M": "mamba", "E": "moe", "*": "attention"}[ch] for ch in
                                                        "MEMEM*EMEMEM*EMEMEM*EMEMEM*EMEMEM*EMEMEMEM*EMEMEMEME"],
                                     num_attention_heads=32, num_key_value_heads=2, head_dim=128, rms_norm_eps=1e-5, use_rope=False,
                                     mlp_gated=False, hidden_act="relu2", mamba_num_heads=64, mamba_head_dim=64, ssm_state_size=128,
                                     mamba_n_groups=8, mamba_chunk_size=128, num_experts=128, num_experts_per_tok=6,
                                     moe_intermediate_size=1856, n_shared_experts=1, moe_shared_expert_intermediate_size=3712,
                                     scoring_func="sigmoid", routed_scaling_factor=2.5),
    # tiny vision-language model for offline recipes and tests: the oracle language model behind a 2-layer ViT
    "tiny-vlm": dict(model_type="llama", vocab_size=2048, hidden_size=256, intermediate_size=688,
                     num_hidden_layers=4, num_attention_heads=4, num_key_value_heads=4, head_dim=64,
                     rms_norm_eps=1e-5, rope_theta=10000.0, image_token_id=511,
                     vision=dict(patch_size=4, channels=3, hidden_size=64, intermediate_size=128, num_layers=2, num_heads=4, max_patches=256)),
    # Qwen2-VL-7B-shaped: Qwen2-7B language model, 32-layer ViT of width 1280 on 14 x 14 patches
    "qwen2-vl-7b": dict(model_type="qwen2", vocab_size=152064, hidden_size=3584, intermediate_size=18944,
                        num_hidden_layers=28, num_attention_heads=28, num_key_value_heads=4, head_dim=128,
                        rms_norm_eps=1e-6, rope_theta=1000000.0, attention_bias=True, image_token_id=151655,
                        vision=dict(patch_size=14, channels=3, hidden_size=1280, intermediate_size=5120, num_layers=32, num_heads=16,
                                    max_patches=16384)),
}


def preset(name: str, **overrides) -> ModelConfig:
    cfg = ModelConfig(**PRESETS[name])
    for k, v in overrides.items():
        setattr(cfg, k, v)
    return cfg
