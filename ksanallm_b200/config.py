"""Configuration: the serving YAML (same schema and defaults as the reference) and the model
hyper-parameters read from a Hugging Face ``config.json`` / ``generation_config.json``.

Reference behaviour: src/ksana_llm/utils/environment.cpp:275-438 (YAML), :527-620 (model config),
:121-192 (max length / rope scaling), :194-227 (EOS ids), :229-273 (KV scale files), :640-675
(block sizes); defaults from src/ksana_llm/utils/environment.h:139-260 and examples/ksana_llm.yaml.
Unknown keys are accepted with a warning. New keys: ``expert_para_size``, ``attn_data_para_size``,
``quant_method: fp8_block|nvfp4``, ``comm_backend: fused|nccl``.
"""
from __future__ import annotations

import json
import logging
import math
import os
from dataclasses import dataclass, field, fields
from typing import Any, Dict, List, Optional, Union

import yaml

log = logging.getLogger("ksana_llm")


@dataclass
class GlobalConfig:
    tensor_para_size: int = 1
    pipeline_para_size: int = 1
    pipeline_micro_batches: int = 2      # micro-batches of one step in flight across the pipeline stages
    expert_para_size: int = 1
    attn_data_para_size: int = 1
    enable_lora_adapter: bool = False
    embed_tokens_use_cpu: bool = False
    enable_cuda_graph: bool = False
    is_version_report: bool = True
    comm_backend: str = "fused"          # fused | nccl


@dataclass
class BatchSchedulerConfig:
    schedule_strategy: int = 0
    waiting_timeout_in_ms: int = 600000
    max_waiting_queue_len: int = 256
    max_token_len: int = 2048
    max_step_tokens: int = 4096
    max_batch_size: int = 8
    swapout_block_threshold: float = 1.0
    swapin_block_threshold: float = 2.0
    launch_block_threshold: float = 2.0
    preempt_mode: int = 0
    split_fuse_token_num: int = 0
    swap_threadpool_size: int = 2
    min_flexible_cache_num: int = 0
    enable_auto_prefix_cache: bool = False


@dataclass
class BlockManagerConfig:
    block_token_num: int = 16
    reserved_device_memory_ratio: float = 0.05
    lora_deivce_memory_ratio: float = 0.0     # (sic) key spelling of the reference YAML
    block_device_memory_ratio: float = -1.0
    lora_host_memory_factor: float = 10.0
    block_host_memory_factor: float = 10.0
    # optional explicit block counts (tests, CPU runs)
    device_blocks_num: int = 0
    host_blocks_num: int = 0


@dataclass
class QuantConfig:
    gptq_backend: str = "cutlass"
    kv_cache_dtype: str = "auto"              # auto | fp8_e5m2 | fp8_e4m3
    weight_quant_method: str = "auto"         # auto | fp8_e4m3 | fp8_block | nvfp4 | w4a16 (gptq / awq select w4a16)
    # scales of weights quantised at load time: "ue8m0" = powers of two (applied by the tensor cores through the
    # block-scaled MMA), "fp32" = amax / 448 exactly (served by the register-promotion GEMM)
    fp8_scale_mode: str = "ue8m0"


@dataclass
class ProfilerConfig:
    trace_export_url: str = ""
    metrics_export_url: str = ""
    export_interval_millis: int = 60000
    export_timeout_millis: int = 1000
    attributes: Dict[str, str] = field(default_factory=dict)


@dataclass
class PluginModelConfig:
    enable_tensorrt: bool = True
    plugin_thread_pool_size: int = 1


@dataclass
class EngineConfig:
    global_: GlobalConfig = field(default_factory=GlobalConfig)
    batch_scheduler: BatchSchedulerConfig = field(default_factory=BatchSchedulerConfig)
    block_manager: BlockManagerConfig = field(default_factory=BlockManagerConfig)
    quantization: QuantConfig = field(default_factory=QuantConfig)
    profiler: ProfilerConfig = field(default_factory=ProfilerConfig)
    plugin_model: PluginModelConfig = field(default_factory=PluginModelConfig)
    endpoint_type: str = "python"
    model_dir: str = ""
    tokenizer_dir: str = ""
    lora_models: List[Dict[str, Any]] = field(default_factory=list)
    # pipeline (multi-node) settings come from the process environment
    master_host: str = ""
    master_port: int = 0
    world_size: int = 1
    node_rank: int = 0


def _fill(dc, section: Optional[dict], where: str):
    if not section:
        return
    names = {f.name for f in fields(dc)}
    for k, v in section.items():
        if k in names:
            cur = getattr(dc, k)
            try:
                if isinstance(cur, bool):
                    v = bool(v)
                elif isinstance(cur, int) and not isinstance(v, bool):
                    v = int(v)
                elif isinstance(cur, float):
                    v = float(v)
            except (TypeError, ValueError):
                raise ValueError(f"bad value for {where}.{k}: {v!r}")
            setattr(dc, k, v)
        elif isinstance(v, dict):
            continue
        else:
            log.warning("unknown config key %s.%s ignored", where, k)


def load_yaml_config(path_or_dict) -> EngineConfig:
    """Parse the serving YAML (a path, a YAML string's dict, or an already-loaded dict)."""
    if isinstance(path_or_dict, dict):
        doc = path_or_dict
        base_dir = os.getcwd()
    else:
        with open(path_or_dict, "r", encoding="utf-8") as f:
            doc = yaml.safe_load(f) or {}
        base_dir = os.path.dirname(os.path.abspath(path_or_dict))
    cfg = EngineConfig()
    setting = doc.get("setting", {}) or {}
    _fill(cfg.global_, setting.get("global"), "setting.global")
    _fill(cfg.batch_scheduler, setting.get("batch_scheduler"), "setting.batch_scheduler")
    _fill(cfg.block_manager, setting.get("block_manager"), "setting.block_manager")
    q = setting.get("quantization_config", {}) or {}
    cfg.quantization.gptq_backend = str(q.get("gptq_backend", cfg.quantization.gptq_backend))
    cfg.quantization.kv_cache_dtype = str((q.get("kv_cache") or {}).get("dtype", "auto"))
    cfg.quantization.weight_quant_method = str((q.get("weight") or {}).get("quant_method", "auto"))
    cfg.quantization.fp8_scale_mode = str((q.get("weight") or {}).get("scale_mode", cfg.quantization.fp8_scale_mode))
    if cfg.quantization.fp8_scale_mode not in ("ue8m0", "fp32"):
        raise ValueError(f"unsupported weight.scale_mode {cfg.quantization.fp8_scale_mode}")
    if cfg.quantization.kv_cache_dtype not in ("auto", "fp8_e5m2", "fp8_e4m3"):
        raise ValueError(f"unsupported kv_cache.dtype {cfg.quantization.kv_cache_dtype}")
    if cfg.quantization.weight_quant_method not in ("auto", "fp8_e4m3", "fp8_block", "nvfp4", "w4a16", "gptq", "awq"):
        raise ValueError(f"unsupported weight.quant_method {cfg.quantization.weight_quant_method}")
    prof = setting.get("profiler", {}) or {}
    for k in ("trace_export_url", "metrics_export_url"):
        if k in prof:
            setattr(cfg.profiler, k, str(prof[k]))
    for k in ("export_interval_millis", "export_timeout_millis"):
        if k in prof:
            setattr(cfg.profiler, k, int(prof[k]))
    cfg.profiler.attributes = {str(k): str(v) for k, v in (prof.get("attributes") or {}).items()}
    cfg.endpoint_type = str(setting.get("endpoint_type", "python"))
    spec = doc.get("model_spec", {}) or {}
    base = spec.get("base_model", {}) or {}
    model_dir = str(base.get("model_dir", ""))
    if model_dir and not os.path.isabs(model_dir):
        model_dir = os.path.normpath(os.path.join(base_dir, model_dir))
    cfg.model_dir = model_dir
    cfg.tokenizer_dir = str(base.get("tokenizer_dir", "")) or model_dir
    _fill(cfg.plugin_model, spec.get("plugin_model"), "model_spec.plugin_model")
    cfg.lora_models = list(spec.get("lora_models") or [])
    # prefix caching is implied by the flexible cache, as in the reference
    if cfg.batch_scheduler.min_flexible_cache_num > 0:
        cfg.batch_scheduler.enable_auto_prefix_cache = True
    if cfg.global_.pipeline_para_size < 1 or cfg.global_.tensor_para_size < 1:
        raise ValueError("tensor_para_size and pipeline_para_size must be >= 1")
    if cfg.batch_scheduler.preempt_mode not in (0, 1):
        raise ValueError("preempt_mode must be 0 (SWAP) or 1 (RECOMPUTE)")
    # multi-node pipeline environment (src/ksana_llm/service/inference_server.cpp:43-67)
    cfg.master_host = os.environ.get("MASTER_HOST", "")
    cfg.master_port = int(os.environ.get("MASTER_PORT", "0") or 0)
    cfg.world_size = int(os.environ.get("WORLD_SIZE_NODES", os.environ.get("KSANA_WORLD_SIZE", "1")) or 1)
    cfg.node_rank = int(os.environ.get("NODE_RANK", "0") or 0)
    return cfg


# --------------------------------------------------------------------------------- model config
# Descriptions of layers that are configured one by one (families whose config.json lists its layers)
@dataclass
class RotarySpec:
    dims: int                             # leading dimensions of a head that rotate
    base: float
    scaling: Optional[dict] = None        # Hugging Face style rope_scaling dict
    interleaved: bool = False             # pairs (2i, 2i + 1) instead of halves (i, i + dims/2)


@dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int                              # query / key head size
    vdim: int                             # value head size
    scale: float
    window: int = 0                       # sliding window in tokens, 0: full causal attention
    keep_first: int = 0                   # first tokens that stay visible behind the window
    sink: bool = False                    # learned per-head logit in the softmax denominator
    rotary: Optional[RotarySpec] = None
    qk_norm: bool = False                 # root-mean-square norm of all of q (and of k) at once, before the rotation
    sigmoid: bool = False                 # a key's weight is the sigmoid of its score; weights are not normalised over keys
    bias_far: int = 0                     # > 0: learned biases by distance, logarithmic buckets that end at this distance


@dataclass
class StateSpaceSpec:
    """Selective state space: per head a state of ``state`` x ``vdim`` with one decay, ``groups`` of heads share input and output
    vectors; a short convolution in front, a gated norm of ``norm_groups`` parts behind."""
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int                             # of the short convolution
    norm_groups: int = 1


@dataclass
class DeltaRuleSpec:
    """Gated delta rule: per head a state of ``dim`` x ``vdim`` with a decay per key channel."""
    heads: int
    kv_heads: int                         # heads of q and k
    dim: int
    vdim: int
    taps: int


@dataclass
class ParallelSpec:
    """Attention and a recurrence that read the same input; their results are added with a factor each."""
    attention: AttentionSpec
    recurrence: DeltaRuleSpec
    attention_scale: float
    recurrence_scale: float


@dataclass
class MlpSpec:
    size: int
    limit: float                          # clamp of the gate (from above) and of the linear part (both sides)
    alpha: float = 1.702                  # slope inside the gate's sigmoid
    offset: float = 1.0                   # added to the linear part


@dataclass
class LatentAttentionSpec:
    """Attention over cached latents: per head ``dim`` plain and ``rot_dim`` rotated (pairs 2i, 2i + 1) query and key
    dimensions and ``vdim`` value dimensions, a sigmoid gate on the output."""
    heads: int
    dim: int
    rot_dim: int                          # 0: no rotated part
    vdim: int
    kv_rank: int                          # latent size
    scale: float
    rotary: Optional[RotarySpec] = None
    window: int = 0                       # sliding window in tokens, 0: full causal attention
    kv_from: Optional[int] = None         # layer whose cached latents are read; None: the layer's own
    q_rank: int = 0                       # size of the normed latent that the queries go through; 0: straight from the input
    sink: bool = False                    # learned per-head logit in the softmax denominator
    head_gate: bool = False               # one gate per head instead of one per output element


@dataclass
class GatedRecurrenceSpec:
    """Element-wise recurrence that is linear in its state: the gates do not see the state."""
    width: int


@dataclass
class PlainMlpSpec:
    """up, piecewise unit, down."""
    size: int


@dataclass
class GatedMlpSpec:
    """down(act(gate) * up)."""
    size: int
    act: str = "silu"                     # silu | gelu (tanh form)


@dataclass
class RouterSpec:
    experts: int
    top: int
    scoring: str = "softmax"              # softmax | sigmoid
    renorm: bool = False                  # the chosen weights are divided by their sum
    scale: float = 1.0
    correction: bool = False              # learned per-expert offset that enters the choice, not the weights
    groups: int = 1                       # equal groups of neighbouring experts ...
    keep_groups: int = 1                  # ... of which the best by the sum of their largest choice scores stay:
    group_top: int = 2                    # ... of how many


@dataclass
class MoeSpec:
    """Mixture of gated feed-forwards, and optionally one (``shared``) that every token goes through, with a gate."""
    router: RouterSpec
    expert: Union[GatedMlpSpec, MlpSpec]
    shared: Optional[GatedMlpSpec] = None


@dataclass
class LayerSpec:
    mixer: Union[AttentionSpec, LatentAttentionSpec, GatedRecurrenceSpec, StateSpaceSpec, ParallelSpec]
    mlp: Optional[Union[MlpSpec, PlainMlpSpec, GatedMlpSpec, MoeSpec]]


@dataclass
class LoopSpec:
    """Layers start .. stop-1 run ``times`` times with the same weights and a cache per pass."""
    start: int
    stop: int
    times: int


@dataclass
class PairEmbeddingSpec:
    """Hashed embedding of (previous token, token): row (prev * mul_prev + token * mul_cur) mod buckets."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class ModelConfig:
    model_type: str = "llama"
    hf_model_type: str = ""        # model_type as config.json spells it (names the optional weight map file)
    hidden_size: int = 4096
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 32
    head_dim: int = 128
    intermediate_size: int = 11008
    vocab_size: int = 32000
    rms_norm_eps: float = 1e-6
    rope_theta: float = 10000.0
    rope_scaling: Optional[dict] = None
    rotary_dim: int = 0                   # 0 -> head_dim
    rope_neox: bool = True
    max_position_embeddings: int = 2048
    max_token_len: int = 2048             # after rope-scaling extension
    tie_word_embeddings: bool = False
    qkv_bias: bool = False
    o_bias: bool = False
    mlp_bias: bool = False
    activation: str = "silu"
    gated_mlp: bool = True
    norm_type: str = "rmsnorm"            # rmsnorm | layernorm
    post_norm: bool = False               # GPT-1 / fairseq style
    position_embedding: str = "rope"      # rope | alibi | learned | sinusoidal | mrope | per_layer (layer_specs)
    mrope_section: Optional[List[int]] = None
    emb_scale: float = 1.0
    lm_head_norm: bool = False            # Baichuan2 normalised lm_head
    eos_token_ids: List[int] = field(default_factory=list)
    pad_token_id: int = 0
    dtype: str = "bfloat16"
    # MoE
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    shared_expert_intermediate_size: int = 0
    num_shared_experts: int = 0
    norm_topk_prob: bool = True
    moe_scoring: str = "softmax"          # softmax | sigmoid
    routed_scaling_factor: float = 1.0
    n_group: int = 1
    topk_group: int = 1
    first_k_dense_replace: int = 0
    moe_layer_freq: int = 1
    shared_expert_gate: bool = False
    expert_para_size: int = 1             # > 1: whole experts per rank of the tensor-parallel group (set by the engine)
    # MLA
    q_lora_rank: int = 0
    kv_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    # quantisation found in the checkpoint
    quant_method: str = ""                # "", fp8, gptq, awq
    quant_bits: int = 0
    quant_group_size: int = 0
    quant_desc_act: bool = False
    fp8_checkpoint: bool = False
    weight_block_size: Optional[List[int]] = None
    is_visual: bool = False
    kv_scales: Optional[List[List[float]]] = None     # per layer (k_scale, v_scale)
    # layers configured one by one
    layer_specs: Optional[List[LayerSpec]] = None
    loop: Optional[LoopSpec] = None
    pair_embedding: Optional[PairEmbeddingSpec] = None
    norm_groups: int = 1                  # equal parts of a row that the norms treat one by one
    residual_mult: float = 1.0            # factor of every sublayer's result
    logit_scale: float = 1.0
    logit_softcap: float = 0.0            # > 0: logits are cap * tanh(logits / cap)

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0


_ARCH_ALIASES = {
    "llama": "llama", "mistral": "llama", "qwen2": "qwen", "qwen": "qwen", "qwen2_vl": "qwen2_vl", "baichuan": "baichuan",
    "chatglm": "chatglm", "glm": "chatglm", "gpt2": "gpt", "openai-gpt": "gpt", "fairseq-transformer": "gpt", "mixtral": "mixtral",
    "qwen2_moe": "qwen2_moe", "deepseek_v3": "deepseek_v3", "deepseek_v2": "deepseek_v3", "internlm2": "llama",
    "yi": "llama", "lenolix": "lenolix", "rasizen": "rasizen", "fidevik": "fidevik", "fapudra": "fapudra",
}
# No position limit is part of the Lenolix, Rasizen and Fidevik designs: the serving configuration's max_token_len decides
_UNBOUNDED_POSITIONS = 1 << 20


def parse_model_max_length(hf: dict, max_pos: int) -> int:
    """Extend the position range by the rope-scaling factor the way the reference does
    (environment.cpp:121-192): su/longrope use original_max*factor when given, llama3/yarn/linear/dynamic
    multiply max_position_embeddings."""
    rs = hf.get("rope_scaling") or {}
    if not rs:
        return max_pos
    kind = rs.get("rope_type", rs.get("type", "default"))
    factor = float(rs.get("factor", 1.0))
    if kind in ("su", "longrope"):
        return int(hf.get("max_position_embeddings", max_pos))
    if kind in ("yarn",):
        orig = int(rs.get("original_max_position_embeddings", max_pos))
        return int(orig * factor)
    if kind in ("llama3",):
        return max_pos           # HF already lists the extended length
    if kind in ("linear", "dynamic"):
        return int(max_pos * factor)
    return max_pos


def resolve_architecture(model_type: str, model_dir: Optional[str] = None) -> str:
    """Model family that serves a config.json ``model_type``: a known name, else a family whose name the type
    contains (case-insensitive, e.g. "codellama" -> llama), else Llama when a weight map
    ``<model_type>_weight_map.json`` exists for it (next to the checkpoint or in the package: a Llama-shaped model
    whose tensors only carry other names), else an error (src/ksana_llm/runtime/model_instance.cpp:42-86)."""
    if model_type in _ARCH_ALIASES:
        return _ARCH_ALIASES[model_type]
    low = model_type.lower()
    for part, arch in (("llama", "llama"), ("qwen2_moe", "qwen2_moe"), ("qwen2_vl", "qwen2_vl"), ("qwen", "qwen"),
                       ("baichuan", "baichuan"), ("chatglm", "chatglm"), ("gpt", "gpt"), ("fairseq-transformer", "gpt"),
                       ("mixtral", "mixtral"), ("deepseek", "deepseek_v3")):
        if part in low:
            return arch
    if find_weight_map(low, model_dir) or find_weight_map(model_type, model_dir):
        return "llama"
    raise ValueError(f"Model type {model_type} is not supported (no <model_type>_weight_map.json found for it either).")


def find_weight_map(model_type: str, model_dir: Optional[str] = None) -> Optional[str]:
    """Path of ``<model_type>_weight_map.json``: the checkpoint directory first, then the package's weight_map folder
    (src/ksana_llm/utils/optional_file.h:23-61)."""
    name = f"{model_type}_weight_map.json"
    for folder in ([model_dir] if model_dir else []) + [os.path.join(os.path.dirname(os.path.abspath(__file__)), "weight_map")]:
        path = os.path.join(folder, name)
        if os.path.exists(path):
            return path
    return None


def model_config_from_hf(hf: dict, generation: Optional[dict] = None, model_dir: Optional[str] = None) -> ModelConfig:
    tc = hf.get("text_config")
    if isinstance(tc, dict):
        # multimodal config.json files of newer exports keep the language model's fields under text_config
        merged = dict(tc)
        merged.update({k: v for k, v in hf.items() if k not in ("text_config",) and (v is not None or k not in merged)})
        merged["model_type"] = hf.get("model_type", tc.get("model_type", "llama"))
        for k in ("tie_word_embeddings",):
            if hf.get(k) is None and tc.get(k) is not None:
                merged[k] = tc[k]
        hf = merged
    rp = hf.get("rope_parameters")
    if isinstance(rp, dict):
        # newer config.json files keep rope_theta and the scaling description together under rope_parameters
        hf = dict(hf)
        if rp.get("rope_theta") is not None and hf.get("rope_theta") is None:
            hf["rope_theta"] = rp["rope_theta"]
        if hf.get("rope_scaling") is None and rp.get("rope_type", rp.get("type", "default")) != "default":
            hf["rope_scaling"] = {k: v for k, v in rp.items() if k != "rope_theta"}
        elif hf.get("rope_scaling") is None and rp.get("mrope_section"):
            hf["rope_scaling"] = {"mrope_section": rp["mrope_section"]}
    # families with a configuration format of their own name themselves in "architecture"
    mt = hf.get("model_type") or str(hf.get("architecture", "llama")).lower()
    arch = resolve_architecture(mt, model_dir)
    if arch == "lenolix":
        return lenolix_config(hf, generation)
    if arch == "rasizen":
        return rasizen_config(hf, generation)
    if arch == "fidevik":
        return fidevik_config(hf, generation)
    if arch == "fapudra":
        return fapudra_config(hf, generation)
    c = ModelConfig(model_type=arch, hf_model_type=mt)
    if arch == "gpt":
        c.hidden_size = hf.get("n_embd", hf.get("hidden_size", hf.get("decoder_embed_dim", 768)))
        c.num_layers = hf.get("n_layer", hf.get("num_hidden_layers", hf.get("decoder_layers", 12)))
        c.num_heads = hf.get("n_head", hf.get("num_attention_heads", hf.get("decoder_attention_heads", 12)))
        c.num_kv_heads = c.num_heads
        c.intermediate_size = hf.get("n_inner") or hf.get("decoder_ffn_embed_dim") or 4 * c.hidden_size
        c.vocab_size = hf.get("vocab_size", 50257)
        c.max_position_embeddings = hf.get("n_positions", hf.get("max_position_embeddings", hf.get("max_target_positions", 1024)))
        c.rms_norm_eps = hf.get("layer_norm_epsilon", 1e-5)
        c.norm_type, c.gated_mlp = "layernorm", False
        c.activation = {"gelu_new": "gelu", "gelu": "gelu", "relu": "relu"}.get(hf.get("activation_function", hf.get("afn", "gelu")), "gelu")
        c.qkv_bias = c.o_bias = c.mlp_bias = True
        c.position_embedding = "sinusoidal" if mt == "fairseq-transformer" else "learned"
        c.post_norm = mt in ("openai-gpt", "fairseq-transformer") and not hf.get("decoder_normalize_before", False)
        c.tie_word_embeddings = hf.get("tie_word_embeddings", True)
        if mt == "fairseq-transformer" and not hf.get("no_scale_embedding", False):
            c.emb_scale = float(c.hidden_size) ** 0.5
    else:
        c.hidden_size = hf.get("hidden_size", 4096)
        c.num_layers = hf.get("num_hidden_layers", hf.get("num_layers", 32))
        c.num_heads = hf.get("num_attention_heads", 32)
        c.num_kv_heads = hf.get("num_key_value_heads", hf.get("multi_query_group_num", c.num_heads)) or c.num_heads
        c.intermediate_size = hf.get("intermediate_size", hf.get("ffn_hidden_size", 11008))
        c.vocab_size = hf.get("vocab_size", hf.get("padded_vocab_size", 32000))
        c.max_position_embeddings = hf.get("max_position_embeddings", hf.get("seq_length", 2048))
        c.rms_norm_eps = hf.get("rms_norm_eps", hf.get("layernorm_epsilon", 1e-6))
        c.rope_theta = float(hf.get("rope_theta", hf.get("rotary_emb_base", 10000.0)))
        c.tie_word_embeddings = bool(hf.get("tie_word_embeddings", False))
        c.activation = {"silu": "silu", "swiglu": "silu", "gelu": "gelu", "relu": "relu"}.get(hf.get("hidden_act", "silu"), "silu")
    c.head_dim = hf.get("head_dim") or hf.get("kv_channels") or c.hidden_size // c.num_heads
    c.rope_scaling = hf.get("rope_scaling")
    c.max_token_len = parse_model_max_length(hf, c.max_position_embeddings)
    if arch == "qwen" or arch == "qwen2_vl" or arch == "qwen2_moe":
        c.qkv_bias = True
    if mt == "qwen":
        # first-generation Qwen: config.json counts gate and up together (w1 and w2 are intermediate_size / 2 wide each)
        c.intermediate_size //= 2
        c.rms_norm_eps = hf.get("layer_norm_epsilon", c.rms_norm_eps)
    if arch == "qwen2_vl":
        c.position_embedding, c.is_visual = "mrope", True
        c.mrope_section = list((hf.get("rope_scaling") or {}).get("mrope_section", [16, 24, 24]))
        c.rope_scaling = None
    if arch == "baichuan":
        # 13B-class checkpoints (hidden != 4096) use ALiBi; Baichuan2 normalises lm_head rows
        if c.hidden_size != 4096:
            c.position_embedding = "alibi"
        c.lm_head_norm = hf.get("vocab_size", 0) == 125696
    if arch == "chatglm":
        # ChatGLM2/3 (THUDM config names) and GLM-4 in the Hugging Face layout (model_type "glm"): rotary pairs are
        # interleaved and cover only part of the head, QKV carries a bias, gate and up are one fused matrix
        c.rope_neox = False
        prf = hf.get("partial_rotary_factor", (hf.get("rope_parameters") or {}).get("partial_rotary_factor", 0.5))
        c.rotary_dim = int(c.head_dim * float(prf))
        c.qkv_bias = bool(hf.get("attention_bias", hf.get("add_qkv_bias", True)))
        if mt == "glm":
            c.num_kv_heads = hf.get("num_key_value_heads", c.num_heads) or c.num_heads
        else:
            c.num_kv_heads = hf.get("multi_query_group_num", c.num_kv_heads) if hf.get("multi_query_attention", True) else c.num_heads
    if arch in ("mixtral", "qwen2_moe", "deepseek_v3"):
        c.num_experts = hf.get("num_local_experts", hf.get("num_experts", hf.get("n_routed_experts", 8)))
        c.num_experts_per_tok = hf.get("num_experts_per_tok", 2)
        c.moe_intermediate_size = hf.get("moe_intermediate_size", c.intermediate_size)
        c.norm_topk_prob = bool(hf.get("norm_topk_prob", arch != "qwen2_moe"))
    if arch == "qwen2_moe":
        c.shared_expert_intermediate_size = hf.get("shared_expert_intermediate_size", 0)
        c.shared_expert_gate = True
    if arch == "deepseek_v3":
        c.num_shared_experts = hf.get("n_shared_experts", 1)
        c.shared_expert_intermediate_size = c.moe_intermediate_size * c.num_shared_experts
        c.moe_scoring = hf.get("scoring_func", "sigmoid")
        c.routed_scaling_factor = float(hf.get("routed_scaling_factor", 2.5))
        c.n_group, c.topk_group = hf.get("n_group", 8), hf.get("topk_group", 4)
        c.first_k_dense_replace = hf.get("first_k_dense_replace", 3)
        c.moe_layer_freq = hf.get("moe_layer_freq", 1)
        c.q_lora_rank = hf.get("q_lora_rank") or 0
        c.kv_lora_rank = hf.get("kv_lora_rank", 512)
        c.qk_nope_head_dim = hf.get("qk_nope_head_dim", 128)
        c.qk_rope_head_dim = hf.get("qk_rope_head_dim", 64)
        c.v_head_dim = hf.get("v_head_dim", 128)
        c.head_dim = c.qk_nope_head_dim + c.qk_rope_head_dim
        c.rope_neox = False
    q = hf.get("quantization_config") or {}
    if q:
        c.quant_method = str(q.get("quant_method", ""))
        c.quant_bits = int(q.get("bits", 0) or 0)
        c.quant_group_size = int(q.get("group_size", 0) or 0)
        c.quant_desc_act = bool(q.get("desc_act", False))
        if c.quant_method == "fp8":
            c.fp8_checkpoint = True
            c.weight_block_size = q.get("weight_block_size")
    td = hf.get("torch_dtype") or hf.get("dtype") or "bfloat16"          # newer exports write "dtype"
    c.dtype = {"float16": "float16", "bfloat16": "bfloat16", "float32": "float32"}.get(str(td).replace("torch.", ""), "bfloat16")
    c.eos_token_ids = _eos_ids(hf, generation)
    pad = hf.get("pad_token_id")
    c.pad_token_id = int(pad) if pad is not None else (1 if mt == "fairseq-transformer" else 0)   # fairseq dictionaries put <pad> at 1
    if c.num_heads % max(c.num_kv_heads, 1):
        raise ValueError("num_attention_heads must be a multiple of num_key_value_heads")
    return c


def _eos_ids(hf: dict, generation: Optional[dict]) -> List[int]:
    eos = (generation or {}).get("eos_token_id", hf.get("eos_token_id"))
    return [] if eos is None else [int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos])]


def _positive(d: dict, key: str, where: str) -> int:
    v = int(d[key])
    if v <= 0:
        raise ValueError(f"{where}.{key} must be positive, not {v}")
    return v


def _lenolix_attention(m: dict, where: str) -> AttentionSpec:
    a = AttentionSpec(_positive(m, "heads", where), _positive(m, "kv_heads", where), _positive(m, "dim", where),
                      _positive(m, "vdim", where), float(m["scale"]), sink=True)
    if a.heads % a.kv_heads:
        raise ValueError(f"{where}: heads must be a multiple of kv_heads")
    mask = m.get("mask")
    if mask:
        a.window, a.keep_first = _positive(mask, "size", where + ".mask"), int(mask.get("keep_first", 0))
    a.rotary = _rotary(m, where)
    return a


def lenolix_config(hf: dict, generation: Optional[dict] = None) -> ModelConfig:
    """config.json of a Lenolix model: ``vocab``, ``width``, ``norm.eps``, ``embedding`` (``scale``, ``bigram``), ``layers``
    (``type``, ``mixer``, ``mlp``) and ``loop``."""
    layers = []
    for i, e in enumerate(hf["layers"]):
        where = f"layers[{i}]"
        if e.get("type", "attention") != "attention":
            raise ValueError(f"{where}: unknown mixer type {e['type']!r}")
        mlp = e.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"{where}: unknown feed-forward kind {mlp['kind']!r}")
        layers.append(LayerSpec(_lenolix_attention(e["mixer"], where + ".mixer"),
                                MlpSpec(_positive(mlp, "ff", where + ".mlp"), float(mlp["limit"])) if mlp else None))
    if not layers:
        raise ValueError("layers is empty")
    emb = hf.get("embedding") or {}
    first = layers[0].mixer
    c = ModelConfig(model_type="lenolix", hf_model_type="lenolix", hidden_size=_positive(hf, "width", "config"), num_layers=len(layers),
                    num_heads=first.heads, num_kv_heads=first.kv_heads, head_dim=first.dim, v_head_dim=first.vdim,
                    intermediate_size=max([s.mlp.size for s in layers if s.mlp] or [0]), vocab_size=_positive(hf, "vocab", "config"),
                    rms_norm_eps=float(hf["norm"]["eps"]), norm_type="layernorm", tie_word_embeddings=True,
                    position_embedding="per_layer",
                    emb_scale=float(emb.get("scale", 1.0)), layer_specs=layers)
    c.max_position_embeddings = c.max_token_len = int(hf.get("max_position_embeddings", _UNBOUNDED_POSITIONS))
    if emb.get("bigram"):
        b = emb["bigram"]
        c.pair_embedding = PairEmbeddingSpec(_positive(b, "buckets", "embedding.bigram"), int(b["mul_prev"]), int(b["mul_cur"]))
    c.loop = _loop(hf, len(layers))
    c.eos_token_ids = _eos_ids(hf, generation)
    return c


def _loop(hf: dict, layers: int) -> Optional[LoopSpec]:
    d = hf.get("loop")
    if not d:
        return None
    loop = LoopSpec(int(d["start"]), int(d["stop"]), _positive(d, "times", "loop"))
    if not 0 <= loop.start < loop.stop <= layers:
        raise ValueError("loop must cover at least one of the layers")
    return loop


def _rotary(m: dict, where: str, interleaved: bool = False) -> Optional[RotarySpec]:
    rot = m.get("rot")
    if not rot or int(rot["dims"]) <= 0:
        return None
    dims = int(rot["dims"])
    if dims % 2 or dims > int(m["dim"]):
        raise ValueError(f"{where}.rot.dims must be even and at most dim")
    sc = rot.get("scaling")
    return RotarySpec(dims, float(rot["base"]), {
        "rope_type": "llama3", "factor": float(sc["factor"]), "low_freq_factor": float(sc["low"]),
        "high_freq_factor": float(sc["high"]), "original_max_position_embeddings": float(sc["original"])} if sc else None, interleaved)


def _latent_attention(m: dict, where: str) -> LatentAttentionSpec:
    rot = m["rot"]
    a = LatentAttentionSpec(*(_positive(m, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")), float(m["scale"]),
                            RotarySpec(_positive(rot, "dims", where + ".rot"), float(rot["base"])))
    if a.rotary.dims != a.rot_dim or a.rot_dim % 2:
        raise ValueError(f"{where}: rot.dims must equal rot_dim and be even")
    if m.get("mask"):
        a.window = _positive(m["mask"], "size", where + ".mask")
    if m.get("kv_from") is not None:
        a.kv_from = int(m["kv_from"])
    return a


def rasizen_config(hf: dict, generation: Optional[dict] = None) -> ModelConfig:
    """config.json of a Rasizen model: ``vocab``, ``width``, ``norm`` (``eps``, ``groups``), ``residual_mult`` and ``layers``
    (``type``, ``mixer``, ``mlp``)."""
    layers = []
    for i, e in enumerate(hf["layers"]):
        where = f"layers[{i}]"
        mlp = e.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"{where}: unknown feed-forward kind {mlp['kind']!r}")
        if e["type"] == "mingru":
            mixer = GatedRecurrenceSpec(_positive(e["mixer"], "width", where + ".mixer"))
        elif e["type"] == "latent_attention":
            mixer = _latent_attention(e["mixer"], where + ".mixer")
            if mixer.kv_from is not None:
                src = layers[mixer.kv_from].mixer if 0 <= mixer.kv_from < i else None
                if not isinstance(src, LatentAttentionSpec) or src.kv_from is not None:
                    raise ValueError(f"{where}.mixer.kv_from must name an earlier layer with latents of its own")
                if (src.kv_rank, src.rot_dim, src.rotary) != (mixer.kv_rank, mixer.rot_dim, mixer.rotary):
                    raise ValueError(f"{where}.mixer: kv_rank, rot_dim and rot must equal those of layer {mixer.kv_from}")
        else:
            raise ValueError(f"{where}: unknown mixer type {e['type']!r}")
        layers.append(LayerSpec(mixer, PlainMlpSpec(_positive(mlp, "ff", where + ".mlp")) if mlp else None))
    if not layers:
        raise ValueError("layers is empty")
    attn = [s.mixer for s in layers if isinstance(s.mixer, LatentAttentionSpec)]
    heads = math.gcd(*(a.heads for a in attn)) if attn else math.gcd(*(s.mixer.width for s in layers))   # what tensor parallelism splits
    c = ModelConfig(model_type="rasizen", hf_model_type="rasizen", hidden_size=_positive(hf, "width", "config"), num_layers=len(layers),
                    num_heads=heads, num_kv_heads=heads, head_dim=attn[0].dim + attn[0].rot_dim if attn else 1,
                    v_head_dim=attn[0].vdim if attn else 0, intermediate_size=max([s.mlp.size for s in layers if s.mlp] or [0]),
                    vocab_size=_positive(hf, "vocab", "config"), rms_norm_eps=float(hf["norm"]["eps"]), tie_word_embeddings=True,
                    position_embedding="per_layer", gated_mlp=False, activation="xielu", layer_specs=layers,
                    norm_groups=int(hf["norm"].get("groups", 1)), residual_mult=float(hf.get("residual_mult", 1.0)))
    if c.norm_groups < 1 or c.hidden_size % c.norm_groups:
        raise ValueError(f"width {c.hidden_size} does not divide into {c.norm_groups} norm groups")
    c.max_position_embeddings = c.max_token_len = int(hf.get("max_position_embeddings", _UNBOUNDED_POSITIONS))
    c.eos_token_ids = _eos_ids(hf, generation)
    return c


def _gated_mlp(m: dict, where: str, act: str) -> GatedMlpSpec:
    return GatedMlpSpec(_positive(m, "ff", where), act)


def _router(r: dict, at: str, **fixed) -> RouterSpec:
    groups = r.get("groups") or {"count": 1, "keep": 1}
    router = RouterSpec(_positive(r, "experts", at), _positive(r, "top", at), groups=_positive(groups, "count", at + ".groups"),
                        keep_groups=_positive(groups, "keep", at + ".groups"), **fixed)
    if router.experts % router.groups or router.keep_groups > router.groups:
        raise ValueError(f"{at}: {router.experts} experts, {router.keep_groups} of {router.groups} groups")
    if router.top > router.experts // router.groups * router.keep_groups:
        raise ValueError(f"{at}: {router.top} of the kept groups' experts cannot be chosen")
    return router


def _moe(m: dict, where: str) -> MoeSpec:
    router = _router(m["router"], where + ".router", scoring="sigmoid", correction=True)
    return MoeSpec(router, _gated_mlp(m["expert"], where + ".expert", "silu"),
                   _gated_mlp(m["shared"], where + ".shared", "silu") if m.get("shared") else None)


def fidevik_config(hf: dict, generation: Optional[dict] = None) -> ModelConfig:
    """config.json of a Fidevik model: ``vocab``, ``width``, ``norm.eps``, ``logit_scale``, ``layers`` (``type``, ``mixer``,
    ``mlp``) and ``loop``."""
    layers = []
    for i, e in enumerate(hf["layers"]):
        where = f"layers[{i}]"
        m, mlp, at = e["mixer"], e.get("mlp"), where + ".mixer"
        if e["type"] == "attention":
            mixer = AttentionSpec(*(_positive(m, k, at) for k in ("heads", "kv_heads", "dim", "vdim")), float(m["scale"]),
                                  rotary=_rotary(m, at, interleaved=True), qk_norm=True)
            if mixer.heads % mixer.kv_heads:
                raise ValueError(f"{at}: heads must be a multiple of kv_heads")
        elif e["type"] == "latent_attention":
            mixer = LatentAttentionSpec(_positive(m, "heads", at), _positive(m, "dim", at), 0, _positive(m, "vdim", at),
                                        _positive(m, "kv_rank", at), float(m["scale"]), q_rank=_positive(m, "q_rank", at), sink=True,
                                        head_gate=True)
        else:
            raise ValueError(f"{where}: unknown mixer type {e['type']!r}")
        if mlp and mlp.get("kind", "dense") not in ("dense", "moe"):
            raise ValueError(f"{where}: unknown feed-forward kind {mlp['kind']!r}")
        ff = None
        if mlp:
            ff = _moe(mlp, where + ".mlp") if mlp.get("kind") == "moe" else _gated_mlp(mlp, where + ".mlp", "gelu")
        layers.append(LayerSpec(mixer, ff))
    if not layers:
        raise ValueError("layers is empty")
    mixers = [s.mixer for s in layers]
    heads = math.gcd(*(a.heads for a in mixers))             # what tensor parallelism splits
    kv = math.gcd(*(a.kv_heads if isinstance(a, AttentionSpec) else a.heads for a in mixers))
    c = ModelConfig(model_type="fidevik", hf_model_type="fidevik", hidden_size=_positive(hf, "width", "config"), num_layers=len(layers),
                    num_heads=heads, num_kv_heads=math.gcd(heads, kv), head_dim=mixers[0].dim, v_head_dim=mixers[0].vdim,
                    intermediate_size=max([s.mlp.size for s in layers if isinstance(s.mlp, GatedMlpSpec)] or [0]),
                    vocab_size=_positive(hf, "vocab", "config"), rms_norm_eps=float(hf["norm"]["eps"]), norm_type="layernorm",
                    position_embedding="per_layer", layer_specs=layers, logit_scale=float(hf.get("logit_scale", 1.0)))
    c.loop = _loop(hf, len(layers))
    c.max_position_embeddings = c.max_token_len = int(hf.get("max_position_embeddings", _UNBOUNDED_POSITIONS))
    c.eos_token_ids = _eos_ids(hf, generation)
    return c


def _divides(n: int, k: int, where: str, names: str) -> None:
    if n % k:
        raise ValueError(f"{where}: {names}: {n} does not divide by {k}")


def _state_space(m: dict, where: str) -> StateSpaceSpec:
    a = StateSpaceSpec(*(_positive(m, k, where) for k in ("heads", "vdim", "state", "groups", "conv")), int(m.get("norm_groups") or 1))
    _divides(a.heads, a.groups, where, "heads and groups")
    _divides(a.heads * a.vdim, a.norm_groups, where, "heads * vdim and norm_groups")
    return a


def _parallel(m: dict, where: str) -> ParallelSpec:
    left, right, at = m["left"], m["right"], where + ".left"
    a = AttentionSpec(*(_positive(left, k, at) for k in ("heads", "kv_heads", "dim", "vdim")), float(left["scale"]), sigmoid=True,
                      bias_far=_positive(left, "bias_max", at))
    _divides(a.heads, a.kv_heads, at, "heads and kv_heads")
    if a.dim != a.vdim:
        raise ValueError(f"{at}: the values are the keys, dim {a.dim} and vdim {a.vdim} must be equal")
    mask = left.get("mask")
    if mask:
        a.window, a.keep_first = _positive(mask, "size", at + ".mask"), int(mask.get("keep_first") or 0)
    at = where + ".right"
    r = DeltaRuleSpec(*(_positive(right, k, at) for k in ("heads", "kv_heads", "dim", "vdim", "conv")))
    _divides(r.heads, r.kv_heads, at, "heads and kv_heads")
    return ParallelSpec(a, r, float(m["left_scale"]), float(m["right_scale"]))


def fapudra_config(hf: dict, generation: Optional[dict] = None) -> ModelConfig:
    """config.json of a Fapudra model: ``vocab``, ``width``, ``max_positions``, ``norm.eps``, ``embedding.scale``, ``logit_softcap``
    and ``layers`` (``type``, ``mixer``, ``mlp``)."""
    layers = []
    for i, e in enumerate(hf["layers"]):
        where = f"layers[{i}]"
        parse = {"mamba2": _state_space, "parallel": _parallel}.get(e["type"])
        if parse is None:
            raise ValueError(f"{where}: unknown mixer type {e['type']!r}")
        mixer, mlp, ff = parse(e["mixer"], where + ".mixer"), e.get("mlp"), None
        if mlp:
            if mlp.get("kind", "moe") != "moe":
                raise ValueError(f"{where}: unknown feed-forward kind {mlp['kind']!r}")
            at = where + ".mlp"
            ff = MoeSpec(_router(mlp["router"], at + ".router", renorm=True, group_top=1),
                         MlpSpec(_positive(mlp["expert"], "ff", at + ".expert"), float(mlp["expert"]["limit"])))
        layers.append(LayerSpec(mixer, ff))
    if not layers:
        raise ValueError("layers is empty")
    attn = [s.mixer.attention for s in layers if isinstance(s.mixer, ParallelSpec)]
    first = attn[0] if attn else None
    c = ModelConfig(model_type="fapudra", hf_model_type="fapudra", hidden_size=_positive(hf, "width", "config"), num_layers=len(layers),
                    num_heads=first.heads if first else 1, num_kv_heads=first.kv_heads if first else 1,
                    head_dim=first.dim if first else 1, v_head_dim=first.vdim if first else 0, intermediate_size=0,
                    vocab_size=_positive(hf, "vocab", "config"), rms_norm_eps=float(hf["norm"]["eps"]), position_embedding="per_layer",
                    emb_scale=float((hf.get("embedding") or {}).get("scale", 1.0)), layer_specs=layers,
                    logit_softcap=float(hf.get("logit_softcap") or 0.0))
    c.max_position_embeddings = c.max_token_len = _positive(hf, "max_positions", "config")
    c.eos_token_ids = _eos_ids(hf, generation)
    return c


def load_model_config(model_dir: str) -> ModelConfig:
    with open(os.path.join(model_dir, "config.json"), "r", encoding="utf-8") as f:
        hf = json.load(f)
    gen = None
    gpath = os.path.join(model_dir, "generation_config.json")
    if os.path.exists(gpath):
        with open(gpath, "r", encoding="utf-8") as f:
            gen = json.load(f)
    return model_config_from_hf(hf, gen, model_dir)


def load_kv_scales(path: str, num_layers: int) -> List[List[float]]:
    """``kv_cache_scales.json``: {"kv_cache": {"scaling_factor": {"0": {"<layer>": scale}}}} (one scale
    used for both K and V of a layer)."""
    with open(path, "r", encoding="utf-8") as f:
        doc = json.load(f)
    table = doc["kv_cache"]["scaling_factor"]["0"]
    return [[float(table[str(i)]), float(table[str(i)])] for i in range(num_layers)]


def check_tp(model: ModelConfig, tp: int) -> None:
    if model.num_heads % tp:
        raise ValueError(f"num_heads {model.num_heads} is not divisible by tensor_para_size {tp}")
    if model.num_kv_heads % tp and tp % model.num_kv_heads:
        raise ValueError(f"num_kv_heads {model.num_kv_heads} incompatible with tensor_para_size {tp}")


def kv_block_bytes(model: ModelConfig, block_token_num: int, tp: int, pp: int, kv_dtype_bytes: int) -> int:
    """Bytes of one KV block on one rank: layers/pp x kv_heads/tp x head_dim x block_tokens x 2 (K,V)."""
    layers = (model.num_layers + pp - 1) // pp
    if model.is_mla:
        return layers * block_token_num * (model.kv_lora_rank + model.qk_rope_head_dim) * kv_dtype_bytes
    kvh = max(1, model.num_kv_heads // tp)
    return layers * kvh * model.head_dim * block_token_num * 2 * kv_dtype_bytes
