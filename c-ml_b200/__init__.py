"""ctypes binding of lib/libcml_b200.so (the cmlb200 C-ABI plus the C-ML-compatible C11 host
API). Used by tests/ and bench.py only; the product itself is C11 + CUDA. The directory name
contains a hyphen, so import it with `__graft_entry__.load_package()`.

There is no fallback: if the shared library has not been built, importing raises."""
import ctypes as C
from pathlib import Path

PKG_DIR = Path(__file__).resolve().parent
LIB_PATH = PKG_DIR / "lib" / "libcml_b200.so"

Q4_0, Q8_0, NF4 = 2, 7, 100

if not LIB_PATH.exists():
    raise ImportError(f"{LIB_PATH} is missing: run `python c-ml_b200/build.py` (needs nvcc). "
                      "There is no CPU or PyTorch fallback for this path.")
lib = C.CDLL(str(LIB_PATH))


class QMat(C.Structure):
    """cmlb200_qmat (include/cmlb200.h)."""
    _fields_ = [("type", C.c_int), ("rows", C.c_int), ("cols", C.c_int), ("block", C.c_int),
                ("qs", C.c_void_p), ("scales", C.c_void_p), ("flags", C.c_int), ("tiles", C.c_void_p)]


def _sig(name, restype, *argtypes):
    fn = getattr(lib, name)
    fn.restype = restype
    fn.argtypes = list(argtypes)
    return fn


vp, sz, ci = C.c_void_p, C.c_size_t, C.c_int
last_error = _sig("cmlb200_last_error", C.c_char_p)
_sig("cmlb200_device_count", ci, C.POINTER(ci))
_sig("cmlb200_set_device", ci, ci)
_sig("cmlb200_malloc", ci, C.POINTER(vp), sz)
_sig("cmlb200_free", ci, vp)
_sig("cmlb200_host_alloc_pinned", ci, C.POINTER(vp), sz)
_sig("cmlb200_host_free_pinned", ci, vp)
_sig("cmlb200_memcpy_h2d", ci, vp, vp, sz, vp)
_sig("cmlb200_memcpy_d2h", ci, vp, vp, sz, vp)
_sig("cmlb200_memcpy_d2d", ci, vp, vp, sz, vp)
_sig("cmlb200_memset", ci, vp, ci, sz, vp)
_sig("cmlb200_stream_create", ci, C.POINTER(vp))
_sig("cmlb200_stream_destroy", ci, vp)
_sig("cmlb200_stream_sync", ci, vp)
_sig("cmlb200_device_sync", ci)
_sig("cmlb200_qs_bytes", sz, ci, ci, ci, ci)
_sig("cmlb200_scale_bytes", sz, ci, ci, ci, ci)
_sig("cmlb200_repack_gguf", ci, ci, vp, ci, ci, vp, vp)
_sig("cmlb200_scales_have_subnormals", ci, vp, sz)
_sig("cmlb200_unrepack_gguf", ci, ci, vp, vp, ci, ci, vp)
_sig("cmlb200_gguf_dequantize", ci, ci, vp, vp, sz, vp)
_sig("cmlb200_dequant_qmat", ci, C.POINTER(QMat), vp, vp)
_sig("cmlb200_dequantize_nf4", ci, vp, vp, ci, ci, sz, vp, vp)
_sig("cmlb200_gemv", ci, C.POINTER(QMat), vp, vp, ci, vp)
_sig("cmlb200_gemv_noalloc", ci, C.POINTER(QMat), vp, vp, ci, vp)
_sig("cmlb200_gemv_accum", ci, C.POINTER(QMat), vp, vp, ci, vp)
_sig("cmlb200_gemv_host", ci, C.POINTER(QMat), vp, vp, ci, vp)
_sig("cmlb200_gemv_swiglu", ci, C.POINTER(QMat), C.POINTER(QMat), vp, vp, ci, vp)
_sig("cmlb200_xq_bytes", sz, ci, ci)
_sig("cmlb200_x_digits", ci, vp, ci, ci, vp, vp)
_sig("cmlb200_rmsnorm_digits", ci, vp, vp, ci, ci, C.c_float, vp, vp, vp)
_sig("cmlb200_gemv_xq", ci, C.POINTER(QMat), C.POINTER(QMat), vp, vp, ci, ci, vp)
_sig("cmlb200_gemv_rmsnorm", ci, C.POINTER(QMat), C.POINTER(QMat), vp, vp, C.c_float, vp, ci, ci, vp)
_sig("cmlb200_attention_scratch_floats", sz, ci, ci, ci, ci)
_sig("cmlb200_attention_ex", ci, vp, ci, vp, vp, vp, vp, ci, ci, ci, ci, ci, ci, ci, vp, vp, vp, ci, vp)
_sig("cmlb200_qkv_rope_append", ci, vp, ci, vp, vp, ci, ci, ci, ci, C.c_float, ci, vp, vp, ci, ci, vp)
_sig("cmlb200_attention_decode_scratch_bytes", sz, ci, ci, ci, ci)
_sig("cmlb200_attention_decode", ci, vp, ci, vp, vp, vp, vp, vp, ci, ci, ci, ci, ci, ci, ci, vp, vp, vp, ci, vp)
_sig("cmlb200_rope_table", ci, vp, ci, ci, C.c_float, vp, vp)
_sig("cmlb200_attention_prefill", ci, vp, ci, vp, vp, ci, vp, ci, ci, ci, ci, ci, vp, vp, vp)
_sig("cmlb200_argmax", ci, vp, ci, ci, vp, vp)
_sig("cmlb200_embed_f16", ci, vp, vp, ci, ci, ci, vp, vp)
_sig("cmlb200_rmsnorm", ci, vp, vp, ci, ci, C.c_float, vp, vp, vp)
_sig("cmlb200_tiles_bytes", sz, ci, ci, ci)
_sig("cmlb200_repack_tiles", ci, ci, vp, ci, ci, vp)
_sig("cmlb200_unrepack_tiles", ci, ci, vp, ci, ci, vp)
_sig("cmlb200_gemv_tiles", ci, C.POINTER(QMat), vp, vp, ci, ci, vp)
_sig("cmlb200_gemv_tiles_status", ci, C.POINTER(ci), ci)
_sig("cmlb200_gemm_bf16", ci, C.POINTER(QMat), vp, vp, ci, vp)
_sig("cmlb200_gemm_bf16_splitk", ci, C.POINTER(QMat), vp, vp, ci, ci, vp)
_sig("cmlb200_gemm_bf16_ex", ci, C.POINTER(QMat), vp, ci, ci, vp, vp, vp)
_sig("cmlb200_gemm_status", ci, C.POINTER(ci), ci)
_sig("cmlb200_linear_nf4_general", ci, vp, vp, ci, ci, ci, ci, vp, ci, vp, vp)
_sig("cmlb200_tp_ar_workspace_bytes", sz, sz)
_sig("cmlb200_tp_allreduce_add", ci, vp, vp, sz, ci, ci, C.POINTER(vp), sz, vp)
_sig("cmlb200_gemv_tp_allreduce", ci, C.POINTER(QMat), vp, vp, ci, ci, ci, C.POINTER(vp), sz, vp)
_sig("cmlb200_gemv_tp_fused_ok", ci, C.POINTER(QMat), ci)
_sig("cmlb200_tp_ar_status", ci, vp, C.POINTER(ci))
_sig("cmlb200_tp_ar_bulk_workspace_bytes", sz, sz, ci)
_sig("cmlb200_tp_allreduce_bulk_add", ci, vp, vp, sz, ci, ci, C.POINTER(vp), sz, vp)
_sig("cmlb200_tp_allreduce_bulk_emulate", ci, C.POINTER(vp), C.POINTER(vp), sz, ci, C.POINTER(vp), sz, vp)
_sig("cmlb200_tp_ar_status_reset", ci, vp)
_sig("cmlb200_set_wait_limit", ci, ci)


class CmlB200Error(RuntimeError):
    pass


def check(rc: int, what: str = ""):
    """Raise with the library's own message when a C-ABI call failed."""
    if rc != 0:
        raise CmlB200Error(f"{what} failed ({rc}): {last_error().decode(errors='replace')}")
    return rc


def np_ptr(a):
    return a.ctypes.data_as(C.c_void_p)


def repack_gguf(qtype: int, blocks, rows: int, cols: int):
    """Host repack of a numpy uint8 array of GGUF blocks into (qs, scales) numpy planes."""
    import numpy as np
    qs = np.empty(lib.cmlb200_qs_bytes(qtype, rows, cols, 32), np.uint8)
    sc = np.empty(lib.cmlb200_scale_bytes(qtype, rows, cols, 32), np.uint8)
    check(lib.cmlb200_repack_gguf(qtype, np_ptr(blocks), rows, cols, np_ptr(qs), np_ptr(sc)), "repack")
    return qs, sc


def repack_tiles(qtype: int, blocks, rows: int, cols: int):
    """Host repack of GGUF blocks into the tile-major buffer of the tensor-core decode path."""
    import numpy as np
    out = np.empty(lib.cmlb200_tiles_bytes(qtype, rows, cols), np.uint8)
    check(lib.cmlb200_repack_tiles(qtype, np_ptr(blocks), rows, cols, np_ptr(out)), "repack_tiles")
    return out


# ---- the C-ML-compatible C11 host API (include/cml_quant_api.h) ---------------------------------
class Tensor(C.Structure):
    pass


Tensor._fields_ = [("shape", C.POINTER(C.c_int)), ("ndim", C.c_int), ("numel", C.c_size_t), ("dtype", C.c_int),
                   ("device", C.c_int), ("ir_node", C.c_void_p), ("ir_context", C.c_void_p), ("saved_ir_node", C.c_void_p),
                   ("saved_ir_context", C.c_void_p), ("is_executed", C.c_bool), ("data", C.c_void_p), ("owns_data", C.c_bool),
                   ("from_buffer_cache", C.c_bool), ("requires_grad", C.c_bool), ("grad", C.c_void_p), ("ref_count", C.c_int),
                   ("base", C.c_void_p), ("strides", C.POINTER(C.c_size_t)), ("storage_offset", C.c_size_t),
                   ("is_contiguous", C.c_bool), ("buffer_handle", C.c_void_p), ("user_data", C.c_void_p)]


class TensorConfig(C.Structure):
    _fields_ = [("dtype", C.c_int), ("device", C.c_int), ("has_dtype", C.c_bool), ("has_device", C.c_bool)]


class LlamaConfig(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("vocab_size", "hidden_size", "intermediate_size", "num_layers", "num_heads",
                                       "num_kv_heads", "max_seq_len")] + \
               [("rope_theta", C.c_float), ("rms_norm_eps", C.c_float), ("tensor_parallel_size", C.c_int),
                ("tensor_parallel_rank", C.c_int)]


class LlamaModel(C.Structure):
    _fields_ = [("config", LlamaConfig), ("embed_tokens", C.POINTER(Tensor)), ("norm", C.POINTER(Tensor)),
                ("lm_head", C.POINTER(Tensor)), ("layers", C.c_void_p), ("num_layers", C.c_int), ("tokenizer", C.c_void_p),
                ("weights_loaded", C.c_bool), ("current_seq_len", C.c_int)]


class GenerationConfig(C.Structure):
    _fields_ = [("temperature", C.c_float), ("top_p", C.c_float), ("top_k", C.c_int), ("max_new_tokens", C.c_int),
                ("eos_token_id", C.c_int), ("do_sample", C.c_bool)]


class GenerationResult(C.Structure):
    _fields_ = [("token_ids", C.POINTER(C.c_int)), ("num_tokens", C.c_int), ("text", C.c_char_p), ("total_time_ms", C.c_float),
                ("tokens_per_second", C.c_float)]


class NF4Tensor(C.Structure):
    _fields_ = [("packed_data", C.POINTER(Tensor)), ("scales", C.POINTER(C.c_float)), ("num_scales", C.c_int),
                ("block_size", C.c_int), ("original_numel", C.c_size_t), ("original_shape", C.POINTER(C.c_int)),
                ("original_ndim", C.c_int)]


class QLoRALinear(C.Structure):
    _fields_ = [("in_features", C.c_int), ("out_features", C.c_int), ("rank", C.c_int), ("alpha", C.c_float),
                ("scaling", C.c_float), ("base_weight_nf4", C.POINTER(NF4Tensor)), ("lora_A", C.POINTER(Tensor)),
                ("lora_B", C.POINTER(Tensor)), ("enable_double_quant", C.c_bool)]


class KVCache(C.Structure):
    _fields_ = [("key_cache", C.POINTER(Tensor)), ("value_cache", C.POINTER(Tensor)), ("max_seq_len", C.c_int),
                ("current_len", C.c_int), ("num_kv_heads", C.c_int), ("head_dim", C.c_int)]


class GQAConfig(C.Structure):
    _fields_ = [("num_heads", C.c_int), ("num_kv_heads", C.c_int), ("head_dim", C.c_int), ("scale", C.c_float),
                ("causal", C.c_bool), ("window_size", C.c_int)]


class PageBlock(C.Structure):
    _fields_ = [("key_data", C.POINTER(C.c_float)), ("value_data", C.POINTER(C.c_float)), ("num_tokens", C.c_int),
                ("block_id", C.c_int), ("in_use", C.c_bool)]


class BlockTable(C.Structure):
    _fields_ = [("block_ids", C.POINTER(C.c_int)), ("num_blocks", C.c_int), ("capacity", C.c_int), ("seq_len", C.c_int)]


class PagedKVCache(C.Structure):
    _fields_ = [("blocks", C.POINTER(PageBlock)), ("num_blocks", C.c_int), ("max_blocks", C.c_int),
                ("free_list", C.POINTER(C.c_int)), ("free_count", C.c_int), ("sequences", C.POINTER(BlockTable)),
                ("num_sequences", C.c_int), ("max_sequences", C.c_int), ("num_kv_heads", C.c_int), ("head_dim", C.c_int),
                ("block_size", C.c_int), ("total_allocated", C.c_size_t), ("total_freed", C.c_size_t)]


class RoPEConfig(C.Structure):
    _fields_ = [("dim", C.c_int), ("max_seq_len", C.c_int), ("base", C.c_float)]


class ParallelLinear(C.Structure):          # CMLColumnParallelLinear and CMLRowParallelLinear share the layout
    _fields_ = [("weight", C.POINTER(Tensor)), ("bias", C.POINTER(Tensor)), ("in_features", C.c_int), ("out_features", C.c_int),
                ("tp_size", C.c_int), ("tp_rank", C.c_int)]


TP = C.POINTER(Tensor)
MP = C.POINTER(LlamaModel)
KP = C.POINTER(KVCache)
PLP = C.POINTER(ParallelLinear)
_sig("cml_kv_cache_create", KP, ci, ci, ci)
_sig("cml_kv_cache_free", None, KP)
_sig("cml_kv_cache_append", ci, KP, TP, TP)
_sig("cml_kv_cache_reset", None, KP)
_sig("cml_kv_cache_get_keys", TP, KP)
_sig("cml_kv_cache_get_values", TP, KP)
_sig("cml_gqa_forward", TP, TP, TP, TP, C.POINTER(GQAConfig), TP)
_sig("cml_gqa_forward_cached", TP, TP, TP, TP, KP, C.POINTER(GQAConfig))
_sig("cml_rope_forward", TP, TP, ci, C.POINTER(RoPEConfig))
PKP = C.POINTER(PagedKVCache)
_sig("cml_paged_kv_cache_create", PKP, ci, ci, ci, ci)
_sig("cml_paged_kv_cache_free", None, PKP)
_sig("cml_paged_cache_alloc_block", ci, PKP)
_sig("cml_paged_cache_free_block", None, PKP, ci)
_sig("cml_paged_cache_init_sequence", ci, PKP)
_sig("cml_paged_cache_free_sequence", None, PKP, ci)
_sig("cml_paged_cache_append", ci, PKP, ci, vp, vp)
_sig("cml_paged_gqa_forward", TP, PKP, ci, TP, C.POINTER(GQAConfig))
class SpeculativeConfig(C.Structure):
    _fields_ = [("num_draft_tokens", C.c_int), ("temperature", C.c_float), ("top_p", C.c_float), ("top_k", C.c_int), ("do_sample", C.c_bool)]


class SpeculativeResult(C.Structure):
    _fields_ = [("accepted_tokens", C.POINTER(C.c_int)), ("num_accepted", C.c_int), ("num_drafted", C.c_int), ("num_verified", C.c_int),
                ("acceptance_rate", C.c_float), ("draft_time_ms", C.c_double), ("verify_time_ms", C.c_double), ("total_time_ms", C.c_double)]


ModelForwardFn = C.CFUNCTYPE(C.c_void_p, C.c_void_p, C.POINTER(C.c_int), C.c_int)
SampleTokenFn = C.CFUNCTYPE(C.c_int, C.c_void_p, C.c_void_p, C.c_float)


class SpeculativeDecoder(C.Structure):
    _fields_ = [("config", SpeculativeConfig), ("draft_model_ctx", C.c_void_p), ("draft_forward", ModelForwardFn), ("draft_sample", SampleTokenFn),
                ("target_model_ctx", C.c_void_p), ("target_forward", ModelForwardFn), ("target_sample", SampleTokenFn), ("vocab_size", C.c_int),
                ("total_drafted", C.c_size_t), ("total_accepted", C.c_size_t), ("total_steps", C.c_size_t)]


class SpeculativeLlama(C.Structure):
    _fields_ = [("model", MP), ("cached_tokens", C.POINTER(C.c_int)), ("cached_len", C.c_int), ("capacity", C.c_int), ("min_rows", C.c_int),
                ("rows_computed", C.c_size_t), ("calls", C.c_size_t)]


SDP, SRP, SLP = C.POINTER(SpeculativeDecoder), C.POINTER(SpeculativeResult), C.POINTER(SpeculativeLlama)
_sig("cml_speculative_default_config", SpeculativeConfig)
_sig("cml_speculative_create", SDP, C.POINTER(SpeculativeConfig), ci)
_sig("cml_speculative_free", None, SDP)
_sig("cml_speculative_set_draft_model", None, SDP, vp, vp, vp)
_sig("cml_speculative_set_target_model", None, SDP, vp, vp, vp)
_sig("cml_speculative_decode_step", SRP, SDP, vp, ci)
_sig("cml_speculative_result_free", None, SRP)
_sig("cml_speculative_acceptance_rate", C.c_float, SDP)
_sig("cml_speculative_llama_create", SLP, MP, C.c_bool)
_sig("cml_speculative_llama_free", None, SLP)
_sig("cml_speculative_llama_forward", TP, vp, vp, ci)
_sig("cml_speculative_llama_sample", ci, vp, TP, C.c_float)
_sig("cml_llama_truncate", ci, MP, ci, ci)
class SequenceRequest(C.Structure):
    _fields_ = [("request_id", C.c_int), ("prompt_tokens", C.POINTER(C.c_int)), ("num_prompt_tokens", C.c_int), ("max_new_tokens", C.c_int),
                ("temperature", C.c_float), ("top_p", C.c_float), ("status", C.c_int), ("paged_seq_id", C.c_int),
                ("generated_tokens", C.POINTER(C.c_int)), ("num_generated", C.c_int), ("gen_capacity", C.c_int), ("current_pos", C.c_int),
                ("submit_time_ms", C.c_double), ("first_token_time_ms", C.c_double), ("finish_time_ms", C.c_double)]


class ServingStats(C.Structure):
    _fields_ = [("total_requests", C.c_size_t), ("completed_requests", C.c_size_t), ("active_sequences", C.c_size_t),
                ("total_tokens_generated", C.c_size_t), ("avg_time_to_first_token_ms", C.c_double), ("avg_tokens_per_second", C.c_double),
                ("total_time_ms", C.c_double)]


class ServingConfig(C.Structure):
    _fields_ = [("max_batch_size", C.c_int), ("max_queue_size", C.c_int), ("max_seq_len", C.c_int), ("max_new_tokens_default", C.c_int),
                ("temperature_default", C.c_float), ("top_p_default", C.c_float)]


FinishFn = C.CFUNCTYPE(None, C.POINTER(SequenceRequest), C.c_void_p)
_sig("cml_serving_default_config", ServingConfig)
_sig("cml_serving_create", vp, C.POINTER(ServingConfig))
_sig("cml_serving_free", None, vp)
_sig("cml_serving_submit", ci, vp, vp, ci, ci)
_sig("cml_serving_step", ci, vp)
_sig("cml_serving_get_status", ci, vp, ci)
_sig("cml_serving_get_tokens", C.POINTER(C.c_int), vp, ci, C.POINTER(C.c_int))
_sig("cml_serving_finish_request", ci, vp, ci)
_sig("cml_serving_get_stats", ServingStats, vp)
_sig("cml_serving_run_llama", ci, vp, MP, ci, ci, vp, vp)
_sig("cml_column_parallel_create", PLP, TP, TP, ci, ci)
_sig("cml_column_parallel_free", None, PLP)
_sig("cml_column_parallel_forward", TP, PLP, TP)
_sig("cml_row_parallel_create", PLP, TP, TP, ci, ci)
_sig("cml_row_parallel_free", None, PLP)
_sig("cml_row_parallel_forward", TP, PLP, TP)
_sig("cml_tp_all_reduce_sum", TP, C.POINTER(TP), ci)
_sig("cml_tp_shard_weight", TP, TP, ci, ci, ci)
_sig("cml_llama_layer_forward", TP, MP, vp, TP, ci)
_sig("cml_set_log_level", None, ci)
_sig("tensor_from_data", TP, vp, C.POINTER(ci), ci, C.POINTER(TensorConfig))
_sig("tensor_zeros", TP, C.POINTER(ci), ci, C.POINTER(TensorConfig))
_sig("tensor_free", None, TP)
_sig("tensor_data_ptr", vp, TP)
_sig("gguf_type_is_quantized", C.c_bool, ci)
_sig("gguf_quant_block_size", ci, ci)
_sig("gguf_quant_type_size", sz, ci)
_sig("gguf_dequantize", ci, ci, vp, vp, sz)
_sig("gguf_open_read", vp, C.c_char_p)
_sig("gguf_close", None, vp)
_sig("gguf_get_num_tensors", ci, vp)
_sig("gguf_get_tensor_name", C.c_char_p, vp, ci)
_sig("gguf_read_tensor", TP, vp, C.c_char_p)
_sig("cml_quantize_nf4", TP, TP, ci, C.POINTER(C.POINTER(C.c_float)), C.POINTER(ci))
_sig("cml_dequantize_nf4", TP, TP, C.POINTER(C.c_float), ci, ci, sz)
_sig("cml_nf4_tensor_create", C.POINTER(NF4Tensor), TP, ci)
_sig("cml_nf4_tensor_free", None, C.POINTER(NF4Tensor))
_sig("cml_nf4_tensor_dequantize", TP, C.POINTER(NF4Tensor))
_sig("cml_qlora_linear_create", C.POINTER(QLoRALinear), TP, ci, C.c_float, ci)
_sig("cml_qlora_linear_free", None, C.POINTER(QLoRALinear))
_sig("cml_qlora_linear_forward", TP, C.POINTER(QLoRALinear), TP)
_sig("cml_qlora_linear_invalidate", None, C.POINTER(QLoRALinear))
_sig("cml_qlora_memory_usage", sz, C.POINTER(QLoRALinear))
_sig("cml_qlora_full_memory_usage", sz, ci, ci)
_sig("cml_llama_config_7b", LlamaConfig)
_sig("cml_llama_config_13b", LlamaConfig)
_sig("cml_llama_config_70b", LlamaConfig)
_sig("cml_generation_default_config", GenerationConfig)
_sig("cml_llama_create", MP, C.POINTER(LlamaConfig))
_sig("cml_llama_free", None, MP)
_sig("cml_llama_load_gguf", ci, MP, C.c_char_p)
_sig("cml_llama_forward", TP, MP, vp, ci)
_sig("cml_llama_forward_batch", TP, MP, vp, ci)
_sig("cml_llama_prefill_sequence", ci, MP, ci, vp, ci)
_sig("cml_llama_decode_greedy", ci, MP, vp, ci, ci, vp, C.POINTER(C.c_float))
_sig("cml_llama_generate", vp, MP, C.c_char_p, C.POINTER(GenerationConfig))
_sig("cml_generation_result_free", None, vp)
_sig("cml_llama_sample_token", ci, TP, C.POINTER(GenerationConfig))
_sig("cml_llama_reset", None, MP)
_sig("cml_llama_print_config", None, C.POINTER(LlamaConfig))
_sig("cml_llama_set_options", ci, MP, ci, ci)
_sig("cml_tp_shard_qblocks", ci, ci, vp, ci, ci, ci, ci, ci, vp)
_sig("cml_llama_tp_unique_id", ci, vp)
_sig("cml_llama_tp_init", ci, MP, vp, ci)
_sig("cml_llama_tp_prompt_allreduce", ci, MP, C.POINTER(sz), C.POINTER(C.c_float), C.POINTER(C.c_float))
class Tokenizer(C.Structure):
    _fields_ = [("vocab", C.POINTER(C.c_char_p)), ("vocab_size", C.c_int), ("merges", C.c_void_p), ("num_merges", C.c_int),
                ("token_to_id", C.c_void_p), ("hash_size", C.c_int), ("bos_token_id", C.c_int), ("eos_token_id", C.c_int),
                ("pad_token_id", C.c_int), ("unk_token_id", C.c_int)]


TKP = C.POINTER(Tokenizer)
_sig("cml_tokenizer_create", TKP, C.POINTER(C.c_char_p), ci, C.POINTER(C.c_char_p), ci)
_sig("cml_tokenizer_free", None, TKP)
_sig("cml_tokenizer_encode", C.POINTER(C.c_int), TKP, C.c_char_p, C.POINTER(C.c_int))
_sig("cml_tokenizer_decode", vp, TKP, vp, ci)
_sig("cml_tokenizer_set_special", None, TKP, ci, ci, ci, ci)
_sig("cml_tokenizer_vocab_size", ci, TKP)
_sig("gguf_get_num_metadata", ci, vp)
_sig("gguf_get_metadata_key", C.c_char_p, vp, ci)
_sig("gguf_get_metadata_type", ci, vp, C.c_char_p)
_sig("gguf_get_metadata_int", ci, vp, C.c_char_p, C.POINTER(C.c_int64))
_sig("gguf_get_metadata_float", ci, vp, C.c_char_p, C.POINTER(C.c_double))
_sig("gguf_get_metadata_string", C.c_char_p, vp, C.c_char_p)
_sig("gguf_get_metadata_array_length", C.c_int64, vp, C.c_char_p, C.POINTER(ci))
_sig("gguf_get_metadata_array_string", C.c_char_p, vp, C.c_char_p, C.c_int64)
_sig("gguf_get_metadata_array_data", vp, vp, C.c_char_p)
_sig("gguf_create_tokenizer", TKP, vp)
_sig("cml_llama_config_from_gguf", ci, C.c_char_p, C.POINTER(LlamaConfig))
_sig("cml_llama_load_gguf_tokenizer", ci, MP, C.c_char_p)
class LoRALinear(C.Structure):
    _fields_ = [("in_features", C.c_int), ("out_features", C.c_int), ("rank", C.c_int), ("alpha", C.c_float), ("scaling", C.c_float),
                ("base_weight", C.POINTER(Tensor)), ("lora_A", C.POINTER(Tensor)), ("lora_B", C.POINTER(Tensor)),
                ("frozen_base", C.POINTER(Tensor)), ("merged", C.c_bool)]


class LoRAAdapter(C.Structure):
    _fields_ = [("name", C.c_char * 64), ("rank", C.c_int), ("alpha", C.c_float), ("scaling", C.c_float), ("num_layers", C.c_int),
                ("layers", C.POINTER(C.POINTER(LoRALinear))), ("merged", C.c_bool)]


LP, AP = C.POINTER(LoRALinear), C.POINTER(LoRAAdapter)
_sig("cml_lora_linear_create", LP, TP, ci, C.c_float)
_sig("cml_lora_linear_free", None, LP)
_sig("cml_lora_linear_forward", TP, LP, TP)
_sig("cml_lora_linear_merge", ci, LP)
_sig("cml_lora_linear_unmerge", ci, LP)
_sig("cml_lora_adapter_create", AP, C.c_char_p, ci, C.c_float)
_sig("cml_lora_adapter_free", None, AP)
_sig("cml_lora_adapter_add_layer", ci, AP, LP)
_sig("cml_lora_adapter_merge_all", ci, AP)
_sig("cml_lora_adapter_unmerge_all", ci, AP)
_sig("cmlb200_lora_merge", ci, vp, vp, vp, ci, ci, ci, C.c_float, vp)
class QuantParams(C.Structure):
    _fields_ = [("scale", C.c_float), ("zero_point", C.c_int32)]


_sig("cml_quantize_compute_params", QuantParams, TP, C.c_bool)
_sig("cml_quantize_int8", TP, TP, C.POINTER(QuantParams), C.POINTER(QuantParams))
_sig("cml_dequantize_int8", TP, TP, C.POINTER(QuantParams))
_sig("cml_quantize_uint8", TP, TP, C.POINTER(QuantParams), C.POINTER(QuantParams))
_sig("cml_dequantize_uint8", TP, TP, C.POINTER(QuantParams))
_sig("gguf_open_write", vp, C.c_char_p)
_sig("gguf_write_tensor", ci, vp, C.c_char_p, TP)
_sig("gguf_write_blocks", ci, vp, C.c_char_p, ci, C.POINTER(C.c_int64), ci, vp)
_sig("gguf_write_metadata", ci, vp, C.c_char_p, ci, vp)
_sig("gguf_write_metadata_array", ci, vp, C.c_char_p, ci, vp, C.c_uint64)
_sig("cml_init", ci)
_sig("cml_cleanup", ci)
_sig("tensor_manual_seed", None, C.c_uint64)
_sig("tensor_get_seed", C.c_uint64)
REFERENCE_QUIRKS, KV_FP32, ALL_LOGITS_FP32 = 1, 2, 4


# ---- layered models (include/cml_lm.h and the kernels behind it) ---------------------------------
DT_F32, DT_BF16, DT_F16 = 0, 1, 2
ACT_SILU, ACT_GELU_TANH, ACT_CLAMPED, ACT_GELU_ERF = 0, 1, 2, 3
DTYPE_FLOAT32, DTYPE_BFLOAT16 = 0, 6


class Dense(C.Structure):
    """cmlb200_dense."""
    _fields_ = [("dtype", ci), ("rows", ci), ("cols", ci), ("ld", ci), ("w", vp), ("bias", vp), ("cap", C.c_float)]


class Attn(C.Structure):
    """cmlb200_attn."""
    _fields_ = [("heads", ci), ("kv_heads", ci), ("dim", ci), ("vdim", ci), ("dim_ld", ci), ("vdim_ld", ci), ("scale", C.c_float),
                ("window", ci), ("slopes", vp), ("sink", ci), ("q_norm", vp), ("k_norm", vp), ("eps", C.c_float), ("temp_coef", C.c_float),
                ("temp_every", C.c_float), ("gate_col", ci), ("cache_dtype", ci), ("k_pool", vp), ("v_pool", vp), ("block_size", ci),
                ("block_table", vp), ("table_ld", ci), ("gate_wide", ci), ("keep", ci), ("chunk", ci), ("sinks", vp), ("head_norm", ci), ("keys_as_values", ci),
                ("out_scale", C.c_float), ("freq", vp), ("rot_dims", ci), ("taps", ci), ("conv", vp), ("ring", vp), ("cap", C.c_float), ("talk", vp),
                ("scores", vp), ("scores_ld", ci)]


class Latent(C.Structure):
    """cmlb200_latent."""
    _fields_ = [("heads", ci), ("dim", ci), ("rot_dim", ci), ("vdim", ci), ("rank", ci), ("ld", ci), ("ld_rank", ci), ("scale", C.c_float), ("window", ci),
                ("c_norm", vp), ("eps", C.c_float), ("freq", vp), ("rot_mul", C.c_float), ("kv_col", ci), ("gate_col", ci), ("cache_dtype", ci), ("pool", vp),
                ("block_size", ci), ("block_table", vp), ("table_ld", ci), ("pool_blocks", ci), ("gate_heads", ci), ("sinks", vp)]


class Moe(C.Structure):
    """cmlb200_moe."""
    _fields_ = [("experts", ci), ("top", ci)] + [(n, vp) for n in ("ids", "weight", "pos", "src", "expert", "start", "count", "active", "num_active", "tiles",
                                                                     "num_tiles")] + \
               [("sigmoid", ci), ("group_best", ci), ("identity", ci), ("groups", ci), ("keep", ci), ("correction", vp), ("normalize", ci), ("scale", C.c_float), ("self", vp)]


class Streams(C.Structure):
    """cmlb200_streams."""
    _fields_ = [("streams", ci), ("mix", vp), ("out", vp), ("read", vp)]


class Join(C.Structure):
    """cmlb200_join."""
    _fields_ = [("parts", C.POINTER(Moe)), ("h", vp), ("add", vp), ("ld_add", ci)]


class Delta(C.Structure):
    """cmlb200_delta."""
    _fields_ = [("heads", ci), ("kv_heads", ci), ("dim", ci), ("vdim", ci), ("taps", ci), ("vdim_ld", ci), ("col", ci), ("conv", vp), ("rate", vp),
                ("dt_bias", vp), ("norm", vp), ("eps", C.c_float), ("out_scale", C.c_float), ("state", vp), ("ring", vp)]


class Gru(C.Structure):
    """cmlb200_gru."""
    _fields_ = [("width", ci), ("col", ci), ("state", vp)]


class GatedJoin(C.Structure):
    """cmlb200_gated_join."""
    _fields_ = [("a", vp), ("b", vp), ("ldm", ci), ("a_norm", vp), ("b_norm", vp), ("f", vp), ("ldf", ci), ("parts", C.POINTER(Moe)), ("ga", vp), ("gf", vp), ("ldg", ci),
                ("table", vp), ("table_dtype", ci), ("vocab", ci), ("tokens", vp)]


class LMOptions(C.Structure):
    _fields_ = [("dtype", ci), ("max_tokens", ci), ("max_sequences", ci), ("max_step_rows", ci)]


class LMEntry(C.Structure):
    _fields_ = [("seq", ci), ("tokens", vp), ("num_tokens", ci), ("want", vp), ("num_want", ci)]


_sig("cmlb200_embed_rows", ci, vp, ci, vp, vp, vp, ci, ci, ci, vp, vp)
_sig("cmlb200_residual_norm", ci, vp, vp, ci, vp, vp, C.c_float, ci, ci, vp, vp, ci, ci, vp)
_sig("cmlb200_qk_norm_append", ci, C.POINTER(Attn), vp, ci, vp, vp, ci, vp)
_sig("cmlb200_attention_tiles", ci, C.POINTER(Attn), vp, ci, vp, ci, vp, ci, vp)
_sig("cmlb200_attention_one", ci, C.POINTER(Attn), vp, ci, vp, vp, ci, ci, vp, ci, vp)
_sig("cmlb200_attention_rows_f32", ci, C.POINTER(Attn), vp, ci, vp, vp, ci, vp, ci, vp)
for _n in ("cmlb200_gemv_dense", "cmlb200_gemm_dense", "cmlb200_linear_dense_f32"):
    _sig(_n, ci, C.POINTER(Dense), vp, ci, ci, vp, ci, vp)
for _n in ("cmlb200_gemv_dense_glu", "cmlb200_gemm_dense_glu"):
    _sig(_n, ci, C.POINTER(Dense), vp, ci, ci, ci, ci, vp, ci, vp)
_sig("cmlb200_gemm_dense_status", ci, C.POINTER(ci), ci)
_sig("cmlb200_glu_rows_f32", ci, vp, ci, ci, ci, ci, vp, ci, vp)
_LAT, _MOE, _DENSE, _cf = C.POINTER(Latent), C.POINTER(Moe), C.POINTER(Dense), C.c_float
_sig("cmlb200_residual_add", ci, vp, vp, ci, _MOE, vp, _cf, ci, ci, vp, ci, ci, vp)
_sig("cmlb200_poly_norm", ci, vp, ci, ci, ci, vp, _cf, vp, ci, ci, vp)
_sig("cmlb200_embed_streams", ci, vp, ci, vp, _cf, ci, ci, ci, ci, vp, vp)
_sig("cmlb200_stream_join", ci, C.POINTER(Streams), vp, vp, ci, C.POINTER(Join), vp, _cf, ci, ci, vp, vp, ci, ci, vp)
_sig("cmlb200_delta_one", ci, C.POINTER(Delta), vp, ci, vp, ci, vp, ci, vp, vp, ci, vp, ci, ci, vp)
_sig("cmlb200_delta_rows", ci, C.POINTER(Delta), vp, ci, vp, ci, vp, ci, vp, vp, ci, ci, vp, ci, vp, vp, ci, ci, vp)
_sig("cmlb200_delta_work_floats", C.c_long, C.POINTER(Delta), ci, ci)
_sig("cmlb200_gru_one", ci, C.POINTER(Gru), vp, ci, vp, vp, ci, vp, ci, ci, vp)
_sig("cmlb200_gru_rows", ci, C.POINTER(Gru), vp, ci, vp, ci, vp, ci, ci, vp)
_sig("cmlb200_rotate_append", ci, C.POINTER(Attn), vp, ci, vp, vp, ci, ci, ci, vp, vp)
_sig("cmlb200_ring_rows", ci, C.POINTER(Attn), vp, ci, vp, ci, vp)
_sig("cmlb200_talk_scores_tiles", ci, C.POINTER(Attn), vp, vp, ci, ci, vp, ci, vp)
_sig("cmlb200_talk_scores_rows", ci, C.POINTER(Attn), vp, vp, vp, ci, ci, vp, ci, vp)
_sig("cmlb200_talk_scores_heads", ci)
_sig("cmlb200_gated_join_rows", ci, C.POINTER(GatedJoin), vp, vp, _cf, ci, ci, vp, ci, ci, vp)
_sig("cmlb200_norm_columns", ci, vp, ci, ci, ci, vp, _cf, ci, vp, ci, ci, vp)
_sig("cmlb200_moe_gemv_act", ci, _MOE, _DENSE, vp, ci, ci, ci, ci, ci, vp, ci, vp)
_sig("cmlb200_moe_gemm_act", ci, _MOE, _DENSE, vp, ci, ci, ci, ci, vp, ci, vp)
_sig("cmlb200_act_rows_f32", ci, vp, ci, ci, ci, ci, vp, ci, vp)
_sig("cmlb200_pack_columns", ci, vp, ci, ci, ci, ci, ci, ci, vp, ci, vp)
_sig("cmlb200_latent_append", ci, _LAT, vp, ci, vp, vp, ci, vp)
for _n in ("cmlb200_latent_query", "cmlb200_latent_query_f32"):
    _sig(_n, ci, _LAT, vp, vp, ci, vp, vp, ci, vp, vp)
_sig("cmlb200_attention_latent", ci, _LAT, vp, ci, vp, vp, ci, ci, vp, ci, vp, vp)
_sig("cmlb200_set_attention_latent_form", ci, ci)
_sig("cmlb200_attention_latent_tc_fits", ci, _LAT)
_sig("cmlb200_attention_latent_status", ci, C.POINTER(ci), ci)
for _n in ("cmlb200_latent_output", "cmlb200_latent_output_f32"):
    _sig(_n, ci, _LAT, vp, vp, vp, ci, ci, vp, ci, vp)
_sig("cmlb200_latent_gather", ci, _LAT, vp, ci, vp, C.POINTER(Attn), vp)
_sig("cmlb200_latent_expand", ci, _LAT, _DENSE, vp, ci, C.POINTER(Attn), vp)
_sig("cmlb200_moe_positions", C.c_long, ci, ci, ci, ci)
_sig("cmlb200_moe_route", ci, _MOE, vp, ci, ci, ci, vp)
_sig("cmlb200_moe_gather", ci, _MOE, vp, ci, ci, ci, vp, ci, vp)
_sig("cmlb200_moe_gemv", ci, _MOE, _DENSE, vp, ci, ci, ci, ci, vp, ci, vp)
_sig("cmlb200_moe_gemv_glu", ci, _MOE, _DENSE, vp, ci, ci, ci, ci, ci, _cf, vp, ci, vp)
_sig("cmlb200_moe_gemm", ci, _MOE, _DENSE, vp, ci, ci, ci, vp, ci, vp)
_sig("cmlb200_moe_gemm_glu", ci, _MOE, _DENSE, vp, ci, ci, ci, ci, _cf, vp, ci, vp)
_sig("cmlb200_moe_linear_f32", ci, _MOE, _DENSE, vp, ci, ci, ci, ci, vp, ci, vp)
_sig("cmlb200_moe_glu_rows_f32", ci, vp, ci, ci, ci, ci, _cf, vp, ci, vp)
_sig("cml_lm_default_options", LMOptions)
_sig("cml_lm_known", ci, C.c_char_p)
_sig("cml_lm_load", vp, C.c_char_p, C.POINTER(LMOptions))
_sig("cml_lm_free", None, vp)
_sig("cml_lm_architecture", C.c_char_p, vp)
for _n in ("cml_lm_vocab_size", "cml_lm_sequence_open", "cml_lm_block_size", "cml_lm_blocks_total", "cml_lm_blocks_free"):
    _sig(_n, ci, vp)
_sig("cml_lm_sequence_close", ci, vp, ci)
_sig("cml_lm_sequence_length", ci, vp, ci)
_sig("cml_lm_step", ci, vp, C.POINTER(LMEntry), ci, vp)
_sig("cml_lm_step_greedy", ci, vp, C.POINTER(LMEntry), ci, vp)
_sig("cml_lm_decode_greedy", ci, vp, vp, vp, ci, ci, vp, C.POINTER(C.c_float))
_sig("cml_serving_run_lm", ci, vp, vp, C.POINTER(GenerationConfig), ci, vp, vp)
_sig("cml_lm_generate", C.POINTER(GenerationResult), vp, vp, ci, C.POINTER(GenerationConfig))
_sig("cml_paged_kv_cache_create_device", C.POINTER(PagedKVCache), ci, ci, ci)
_sig("cml_paged_cache_blocks_for", ci, C.POINTER(PagedKVCache), ci, ci)
_sig("cml_paged_cache_extend", ci, C.POINTER(PagedKVCache), ci, ci)
_sig("cml_paged_cache_release_before", None, C.POINTER(PagedKVCache), ci, ci)
_sig("cml_paged_cache_release_between", None, C.POINTER(PagedKVCache), ci, ci, ci)


class LanguageModel:
    """A model loaded through cml_lm_load, with numpy arrays in and out."""

    def __init__(self, path, dtype=DTYPE_BFLOAT16, max_tokens=2048, max_sequences=8, max_step_rows=0):
        self.h = lib.cml_lm_load(str(path).encode(), C.byref(LMOptions(dtype, max_tokens, max_sequences, max_step_rows)))
        if not self.h:
            raise CmlB200Error(f"cml_lm_load({path}) failed")
        self.vocab = lib.cml_lm_vocab_size(self.h)

    def close(self):
        if self.h:
            lib.cml_lm_free(self.h)
            self.h = None

    def open(self):
        s = lib.cml_lm_sequence_open(self.h)
        if s < 0:
            raise CmlB200Error("no free sequence")
        return s

    def end(self, seq):
        check(lib.cml_lm_sequence_close(self.h, seq), "cml_lm_sequence_close")

    def step(self, entries, greedy=False):
        """entries: (seq, tokens, wanted places or None for all). One list item of logits [n, vocab] (or picks [n]) per entry."""
        import numpy as np
        keep, arr = [], (LMEntry * len(entries))()
        for i, (seq, tokens, want) in enumerate(entries):
            t = np.ascontiguousarray(tokens, np.int32)
            w = np.arange(len(t), dtype=np.int32) if want is None else np.ascontiguousarray(want, np.int32)
            keep += [t, w]
            arr[i] = LMEntry(seq, np_ptr(t), len(t), np_ptr(w), len(w))
        counts = [arr[i].num_want for i in range(len(entries))]
        out = np.zeros(max(1, sum(counts)), np.int32) if greedy else np.zeros((max(1, sum(counts)), self.vocab), np.float32)
        check((lib.cml_lm_step_greedy if greedy else lib.cml_lm_step)(self.h, arr, len(entries), np_ptr(out)), "cml_lm_step")
        return np.split(out[:sum(counts)], np.cumsum(counts)[:-1])

    def decode_greedy(self, seqs, first, steps):
        import numpy as np
        s, f, ms = np.ascontiguousarray(seqs, np.int32), np.ascontiguousarray(first, np.int32), C.c_float(0)
        out = np.zeros((steps, len(s)), np.int32)
        check(lib.cml_lm_decode_greedy(self.h, np_ptr(s), np_ptr(f), len(s), steps, np_ptr(out), C.byref(ms)), "cml_lm_decode_greedy")
        return out, ms.value


def tensor_to_numpy(tp, free=True):
    """Copy a host Tensor* returned by the library into a numpy array (fp32 / uint8 / fp16)."""
    import numpy as np
    t = tp.contents
    shape = [t.shape[i] for i in range(t.ndim)]
    np_dtype = {0: np.float32, 8: np.uint8, 7: np.int8, 5: np.float16, 2: np.int32}[t.dtype]
    n = int(np.prod(shape))
    arr = np.frombuffer((C.c_char * (n * np.dtype(np_dtype).itemsize)).from_address(t.data), dtype=np_dtype).reshape(shape).copy()
    if free:
        lib.tensor_free(tp)
    return arr


def numpy_to_tensor(a):
    """A host Tensor* owning a copy of `a` (fp32, fp16, int32, uint8 or int8); release with lib.tensor_free."""
    import numpy as np
    a = np.ascontiguousarray(a)
    dt = {np.dtype(np.float32): 0, np.dtype(np.uint8): 8, np.dtype(np.int8): 7, np.dtype(np.int32): 2, np.dtype(np.float16): 5}[a.dtype]
    cfg = TensorConfig(dt, 0, True, True)
    shape = (C.c_int * a.ndim)(*a.shape)
    return lib.tensor_from_data(np_ptr(a), shape, a.ndim, C.byref(cfg))
