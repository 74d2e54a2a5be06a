"""Registry of model families: which configuration class reads a model's JSON, which native library part runs it, and how
its weights reach the backend.  `CudaInference.load_weights` goes through `family_of(config)`; a new design adds its
architecture name here and, if it is not a combination of existing blocks, its blocks in csrc/.
"""
from __future__ import annotations

import ctypes as C

import numpy as np

from ._lib import IM_DTYPE_BF16, IM_DTYPE_F16, IM_DTYPE_F32, check, lib, vp
from .bundle import GpuBundleError, ModelConfig
from .stack_config import DESIGNS, GatedLinearAttention, GroupedAttention, LatentAttention, LinearAttention, StackConfig


class _CModelConfig(C.Structure):
    _fields_ = [("num_layers", C.c_int), ("hidden_size", C.c_int), ("intermediate_size", C.c_int), ("num_heads", C.c_int),
                ("num_kv_heads", C.c_int), ("head_dim", C.c_int), ("vocab_size", C.c_int), ("max_seq_len", C.c_int),
                ("max_batch", C.c_int), ("rms_eps", C.c_float), ("attn_scale", C.c_float), ("embed_scale", C.c_float),
                ("rope_theta", C.c_double), ("rotary_dim", C.c_int), ("qk_norm", C.c_int), ("tie_word_embeddings", C.c_int),
                ("tq_bits", C.c_int), ("rotation_seed", C.c_uint64), ("tp_world", C.c_int), ("tp_rank", C.c_int),
                ("prefill_chunk_size", C.c_int), ("decode_schedule", C.c_int), ("tp_collective", C.c_int),
                ("wait_limit_ms", C.c_int)]


class _CStackLayer(C.Structure):
    _fields_ = [("mixer", C.c_int), ("heads", C.c_int), ("dim", C.c_int), ("vdim", C.c_int), ("ff", C.c_int), ("kv_rank", C.c_int),
                ("rot_dim", C.c_int), ("rot_dims", C.c_int), ("scale", C.c_float), ("rot_base", C.c_double), ("yarn_factor", C.c_double),
                ("yarn_original", C.c_double), ("yarn_fast", C.c_double), ("yarn_slow", C.c_double), ("decay", C.POINTER(C.c_double)),
                ("kv_heads", C.c_int), ("chunk", C.c_int), ("kv_from", C.c_int), ("rot_divide", C.c_double), ("gate_rank", C.c_int), ("tau", C.c_float)]


class _CStackConfig(C.Structure):
    _fields_ = [("vocab", C.c_int), ("width", C.c_int), ("num_layers", C.c_int), ("layers", C.POINTER(_CStackLayer)),
                ("loop_start", C.c_int), ("loop_stop", C.c_int), ("loop_times", C.c_int), ("norm_eps", C.c_float),
                ("logit_softcap", C.c_float), ("block", C.c_int), ("ff_act", C.c_int), ("embed_scale", C.c_float), ("tied_head", C.c_int),
                ("max_seq_len", C.c_int), ("max_batch", C.c_int), ("prefill_chunk_size", C.c_int), ("compute_f32", C.c_int)]


class QuantizedBlocks:
    """Llama / Qwen3 blocks with affine-quantized projections (csrc/model.cu)."""
    native = "quantized"
    library = None           # part of the complete library only
    config = ModelConfig

    @staticmethod
    def complete(mc: ModelConfig, provider) -> None:
        """Sizes that only the tensors give: none."""

    @staticmethod
    def create(engine, mc: ModelConfig) -> C.c_void_p:
        cfg = engine.config
        cc = _CModelConfig(mc.num_hidden_layers, mc.hidden_size, mc.intermediate_size, mc.num_attention_heads,
                           mc.num_key_value_heads, mc.head_dim, mc.vocab_size, cfg.max_seq_len, cfg.max_batch,
                           mc.rms_norm_eps, mc.attn_scale, float(mc.extra.get("embed_scale", 0.0) or 0.0), mc.rope_theta,
                           int(mc.extra.get("rotary_dim", 0) or 0), int(mc.has_qk_norm), int(mc.tie_word_embeddings),
                           cfg.n_bits if cfg.enable_turboquant else 16, cfg.rotation_seed, cfg.tp_world, cfg.tp_rank,
                           int(cfg.prefill_chunk_size or 0),
                           {"auto": 0, "per_kernel": 1, "tagged": 2}[cfg.decode_schedule],
                           {"auto": 0, "nccl": 1}[cfg.tp_collective], int(cfg.wait_limit_ms))
        model = C.c_void_p()
        check(lib().im_cuda_model_create(engine._dev, C.byref(cc), C.byref(model)))
        return model

    @staticmethod
    def tensor_names(mc: ModelConfig, provider) -> list:
        """The Hugging Face tensor names (weight_loading.rs:163-426)."""
        names = ["model.embed_tokens.weight", "model.norm.weight"]
        if provider.has_tensor("lm_head.weight"):
            names.append("lm_head.weight")
        for i in range(mc.num_hidden_layers):
            p = f"model.layers.{i}"
            names += [f"{p}.input_layernorm.weight", f"{p}.post_attention_layernorm.weight"]
            if mc.has_qk_norm:
                names += [f"{p}.self_attn.q_norm.weight", f"{p}.self_attn.k_norm.weight"]
            names += [f"{p}.self_attn.{x}_proj.weight" for x in "qkvo"] + [f"{p}.mlp.{x}_proj.weight" for x in ("gate", "up", "down")]
        return names

    @staticmethod
    def load_tensor(model, name: str, t) -> None:
        if not t.quantized:
            data = np.ascontiguousarray(t.data)
            if data.dtype != np.float16:
                data = data.astype(np.float16)   # dense tensors live in fp16 on the GPU (metal/weights.rs:928-953)
            check(lib().im_cuda_model_load_dense(model, name.encode(), vp(data), C.c_size_t(data.size)))
            return
        if len(t.shape) != 2:
            raise GpuBundleError(f"{name}: quantized tensor must be 2-D, got shape {t.shape}")
        N, K = t.shape
        sc, zp = np.ascontiguousarray(t.scale), np.ascontiguousarray(t.zero_point)
        if sc.dtype != zp.dtype:
            sc, zp = sc.astype(np.float32), zp.astype(np.float32)
        pd = IM_DTYPE_F32 if sc.dtype == np.float32 else IM_DTYPE_F16
        awq = None if t.awq_scales is None else np.ascontiguousarray(t.awq_scales, dtype=np.float16)
        codes = np.ascontiguousarray(t.data, dtype=np.uint8)
        check(lib().im_cuda_model_load_affine(model, name.encode(), vp(codes), vp(sc), vp(zp), C.c_int(pd), vp(awq),
                                              C.c_int(N), C.c_int(K), C.c_int(t.group_size), C.c_int(t.bit_width)))


class LayerStack:
    """Models given as a list of layers (csrc/stack.cu); weights dense, in bf16 or f32 (CudaConfig.dtype)."""
    native = "stack"
    library = "stack"
    config = StackConfig

    @staticmethod
    def complete(mc: StackConfig, provider) -> None:
        """Sizes that only the tensors' shapes give."""
        mc.complete(lambda name: tuple(provider.tensor(name).shape) if provider.has_tensor(name) else None)

    @staticmethod
    def create(engine, mc: StackConfig) -> C.c_void_p:
        cfg = engine.config
        if cfg.tp_world != 1:
            raise GpuBundleError("models given as a list of layers run on one GPU")
        layers = (_CStackLayer * len(mc.layers))()
        keep = []
        for c, L in zip(layers, mc.layers):
            m = L.mixer
            c.heads, c.dim, c.vdim, c.ff = m.heads, m.dim, m.vdim, L.ff
            if isinstance(m, LatentAttention):
                c.mixer, c.kv_rank, c.rot_dim, c.rot_dims, c.scale, c.rot_base = 1, m.kv_rank, m.rot_dim, m.rot.dims, m.scale, m.rot.base
                c.yarn_factor, c.yarn_original, c.yarn_fast, c.yarn_slow = m.rot.factor, m.rot.original, m.rot.fast, m.rot.slow
            elif isinstance(m, LinearAttention):
                c.mixer = 2
                keep.append((C.c_double * m.heads)(*m.decay))
                c.decay = C.cast(keep[-1], C.POINTER(C.c_double))
            elif isinstance(m, GroupedAttention):
                c.mixer, c.kv_heads, c.scale, c.chunk = 3, m.kv_heads, m.scale, m.chunk
                c.kv_from = 0 if m.kv_from is None else m.kv_from + 1
                c.rot_dim = c.rot_dims = m.rot.dims
                c.rot_base, c.rot_divide = m.rot.base, m.rot.divide
            elif isinstance(m, GatedLinearAttention):
                c.mixer, c.gate_rank, c.tau = 4, m.rank, m.tau
        cc = _CStackConfig(mc.vocab_size, mc.hidden_size, len(mc.layers), layers, mc.loop_start, mc.loop_stop, mc.loop_times, mc.norm_eps,
                           mc.logit_softcap, int(mc.design.post_norm), int(mc.design.silu), mc.embed_scale, int(mc.design.tied_head), cfg.max_seq_len, cfg.max_batch, int(cfg.prefill_chunk_size or 0), int(cfg.dtype == "float32"))
        model = C.c_void_p()
        check(lib().im_cuda_model_create_stack(engine._dev, C.byref(cc), C.byref(model)))
        return model

    @staticmethod
    def tensor_names(mc: StackConfig, provider) -> list:
        return list(mc.tensors())

    @staticmethod
    def load_tensor(model, name: str, t) -> None:
        if t.quantized:
            raise GpuBundleError(f"{name}: this family takes dense tensors")
        data = np.ascontiguousarray(t.data)
        if t.dtype == "bfloat16" and data.dtype == np.uint16:
            dt = IM_DTYPE_BF16
        elif data.dtype == np.float16:
            dt = IM_DTYPE_F16
        else:
            data, dt = np.ascontiguousarray(data, dtype=np.float32), IM_DTYPE_F32
        shape = (C.c_int64 * len(t.shape))(*t.shape)
        check(lib().im_cuda_model_load_tensor(model, name.encode(), vp(data), C.c_int(dt), C.c_int(len(t.shape)), shape))


def family_of_name(architecture: str):
    """The designs of stack_config.py belong to the list-of-layers family; everything else is the quantized block family."""
    return LayerStack if architecture.lower() in DESIGNS else QuantizedBlocks


def family_of(config):
    return LayerStack if isinstance(config, StackConfig) else QuantizedBlocks


def config_from_json(obj):
    """The configuration object of a model's JSON (config.json of a checkpoint, model_config of a bundle)."""
    if not isinstance(obj, dict):
        raise GpuBundleError("model_config must be an object")
    return family_of_name(str(obj.get("architecture", ""))).config.from_json(obj)
