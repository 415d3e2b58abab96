"""ctypes mirrors of the structs in include/zq.h."""
import ctypes as C


class Epilogue(C.Structure):
    _fields_ = [
        ("d_bias", C.c_void_p),
        ("gelu", C.c_int),
        ("d_mul", C.c_void_p),
        ("d_residual", C.c_void_p),
    ]


class TensorRef(C.Structure):
    _fields_ = [
        ("data", C.c_void_p),
        ("type", C.c_int32),
        ("out_dim", C.c_uint32),
        ("in_dim", C.c_uint32),
    ]


class Gpt2Config(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("vocab", "embed", "head", "layer", "ctx", "ffn")]


class Gpt2Block(C.Structure):
    _fields_ = [
        ("ln1_weight", C.c_void_p),
        ("ln1_bias", C.c_void_p),
        ("attn_qkv_weight", TensorRef),
        ("attn_qkv_bias", C.c_void_p),
        ("attn_proj_weight", TensorRef),
        ("attn_proj_bias", C.c_void_p),
        ("ln2_weight", C.c_void_p),
        ("ln2_bias", C.c_void_p),
        ("mlp_fc_weight", TensorRef),
        ("mlp_fc_bias", C.c_void_p),
        ("mlp_proj_weight", TensorRef),
        ("mlp_proj_bias", C.c_void_p),
    ]


class Gpt2Weights(C.Structure):
    _fields_ = [
        ("wte", C.c_void_p),
        ("wpe", C.c_void_p),
        ("ln_f_weight", C.c_void_p),
        ("ln_f_bias", C.c_void_p),
        ("blocks", C.POINTER(Gpt2Block)),
    ]


class Gemma3Config(C.Structure):
    _fields_ = [
        ("vocab", C.c_uint32),
        ("embed", C.c_uint32),
        ("head", C.c_uint32),
        ("head_kv", C.c_uint32),
        ("head_dim", C.c_uint32),
        ("layer", C.c_uint32),
        ("ctx", C.c_uint32),
        ("ffn", C.c_uint32),
        ("rope_base", C.c_float),
        ("sliding_window", C.c_uint32),
        ("rms_eps", C.c_float),
        ("global_every", C.c_uint32),
    ]


class Gemma3Block(C.Structure):
    _fields_ = [
        ("attn_norm_weight", C.c_void_p),
        ("post_attention_norm_weight", C.c_void_p),
        ("attn_q_weight", TensorRef),
        ("attn_k_weight", TensorRef),
        ("attn_v_weight", TensorRef),
        ("attn_output_weight", TensorRef),
        ("attn_q_norm_weight", C.c_void_p),
        ("attn_k_norm_weight", C.c_void_p),
        ("ffn_norm_weight", C.c_void_p),
        ("post_ffw_norm_weight", C.c_void_p),
        ("ffn_gate_weight", TensorRef),
        ("ffn_up_weight", TensorRef),
        ("ffn_down_weight", TensorRef),
    ]


class Gemma3Weights(C.Structure):
    _fields_ = [
        ("token_embd", TensorRef),
        ("output_norm_weight", C.c_void_p),
        ("blocks", C.POINTER(Gemma3Block)),
    ]


class Bf16Ref(C.Structure):
    _fields_ = [("data", C.c_void_p), ("rows", C.c_uint32), ("cols", C.c_uint32)]


class Gqa(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "ctx", "slots")] + [
        (n, C.c_float) for n in ("scale", "norm_eps", "temp_coef", "temp_every")]


class DecoderConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("vocab", "width", "layers", "ctx", "n_seq")] + [
        ("precision", C.c_int32), ("embed_scale", C.c_float), ("norm_eps", C.c_float)]


class DecoderLayer(C.Structure):
    _fields_ = (
        [(n, C.c_uint32) for n in ("mixer", "parallel", "heads", "kv_heads", "dim", "vdim", "v_mix", "decay_rank", "rot_dim",
                                   "kv_rank", "taps")]
        + [("kv_from", C.c_int32)]
        + [(n, C.c_uint32) for n in ("mlp", "mlp_glu", "ff", "experts", "top", "route", "expert_ff", "expert_glu", "shared_ff",
                                     "shared_glu")]
        + [(n, C.c_float) for n in ("scale", "q_temp_coef", "q_temp_every", "vmix", "gate_cap", "rot_base", "limit",
                                    "expert_limit", "shared_limit")]
        + [(n, C.c_void_p) for n in ("norm1", "norm1b", "norm2", "norm2b")]
        + [(n, Bf16Ref) for n in ("q", "k", "v", "o")]
        + [(n, C.c_void_p) for n in ("q_norm", "k_norm")]
        + [(n, Bf16Ref) for n in ("r", "g", "w1", "w2")]
        + [(n, C.c_void_p) for n in ("mu", "w0", "u", "mix_norm")]
        + [(n, Bf16Ref) for n in ("i", "f")]
        + [(n, C.c_void_p) for n in ("i_bias", "f_bias")]
        + [(n, Bf16Ref) for n in ("b", "a1", "a2", "g1", "g2")]
        + [(n, C.c_void_p) for n in ("conv", "A_log", "dt_bias")]
        + [(n, Bf16Ref) for n in ("dkv", "uk", "uv")]
        + [("dkv_norm", C.c_void_p)]
        + [(n, Bf16Ref) for n in ("gate", "up", "down", "router")]
        + [("router_bias", C.c_void_p)]
        + [(n, C.POINTER(Bf16Ref)) for n in ("expert_gate", "expert_up", "expert_down")]
        + [(n, Bf16Ref) for n in ("shared_gate", "shared_up", "shared_down", "shared_sg")]
    )


class DecoderWeights(C.Structure):
    _fields_ = [("embed", Bf16Ref), ("head", Bf16Ref), ("embed_norm", C.c_void_p), ("final_norm", C.c_void_p),
                ("layers", C.POINTER(DecoderLayer))]


class MemoryShape(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "dim", "vdim", "ld")] + [(n, C.c_float) for n in ("gate_cap", "eps")]


class DeltaShape(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "taps", "a_rank", "g_rank", "ld")] + [
        ("eps", C.c_float)]


class LatentShape(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "dim", "rot", "vdim", "rank", "ctx", "slots", "ld")] + [
        (n, C.c_float) for n in ("scale", "eps")]
