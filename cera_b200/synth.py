"""Seeded synthetic llama-architecture models, generated and quantized on the device.

Stands in for real GGUF checkpoints: every tensor is N(0, sigma) from the
counter-based generator behind `synth_normal`, quantized with the reference's
own quantizer rules, so any implementation that knows (seed, role, layer)
regenerates identical bytes.
"""
import numpy as np
import torch

from . import ops
from .model import CudaModel, Role
from .types import F32, Q4_K, Q6_K

# The benchmark model's tensor mix (a Q4_K_M-style GGUF): Q4_K attention / gate / up / token_embd, Q6_K ffn_down and output.
LLAMA3_8B = dict(n_layers=32, hidden_size=4096, intermediate_size=14336, n_heads=32, n_kv_heads=8, head_dim=128,
                 vocab_size=128256, rope_theta=500000.0, rms_norm_eps=1e-5, rope_type=0)
DEFAULT_TYPES = {Role.TOKEN_EMBD: Q4_K, Role.OUTPUT: Q6_K, Role.ATTN_Q: Q4_K, Role.ATTN_K: Q4_K, Role.ATTN_V: Q4_K,
                 Role.ATTN_OUTPUT: Q4_K, Role.FFN_GATE: Q4_K, Role.FFN_UP: Q4_K, Role.FFN_DOWN: Q6_K}


def tensor_seed(seed, role, layer):
    return (seed * 1000003 + int(role) * 4099 + layer + 1) & 0xFFFFFFFFFFFFFFFF


def build_llama(cfg, seed=0, sigma=0.02, types=None, sink=None, **model_kw):
    """Create, fill and finalize a CudaModel.  sink(role, layer, ggml_type, rows, cols, host_bytes)
    receives a host copy of every tensor (tests hand these to the CPU oracle)."""
    types = {**DEFAULT_TYPES, **(types or {})}
    m = CudaModel(**cfg, **model_kw)
    hs, ff = cfg["hidden_size"], cfg["intermediate_size"]
    qd, kvd = cfg["n_heads"] * cfg["head_dim"], cfg["n_kv_heads"] * cfg["head_dim"]

    def matrix(role, layer, rows, cols):
        t = types[role]
        w = ops.synth_normal(rows * cols, tensor_seed(seed, role, layer), sigma)
        raw = ops.quantize_weights(t, w)
        del w
        m.add_tensor(role, layer, t, rows, cols, raw)
        if sink:
            sink(role, layer, t, rows, cols, raw.cpu().numpy())
        del raw

    def ones(role, layer, n):
        v = np.ones(n, dtype=np.float32)
        m.add_tensor(role, layer, F32, 1, n, v)
        if sink:
            sink(role, layer, F32, 1, n, v)

    matrix(Role.TOKEN_EMBD, 0, cfg["vocab_size"], hs)
    matrix(Role.OUTPUT, 0, cfg["vocab_size"], hs)
    ones(Role.OUTPUT_NORM, 0, hs)
    for l in range(cfg["n_layers"]):
        ones(Role.ATTN_NORM, l, hs)
        ones(Role.FFN_NORM, l, hs)
        matrix(Role.ATTN_Q, l, qd, hs)
        matrix(Role.ATTN_K, l, kvd, hs)
        matrix(Role.ATTN_V, l, kvd, hs)
        matrix(Role.ATTN_OUTPUT, l, hs, qd)
        matrix(Role.FFN_GATE, l, ff, hs)
        matrix(Role.FFN_UP, l, ff, hs)
        matrix(Role.FFN_DOWN, l, hs, ff)
    torch.cuda.synchronize()
    m.finalize()
    return m


def goletar_config(width, n_layers, vocab=32768, experts=32, top=4, ff=None):
    """A Goletar configuration whose layers have the shapes of a real model of this width: minGRU and latent attention in
    turn, heads of 128 + 64, a latent of 512."""
    ff = ff or width // 2
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": 7.0}, "router": {"experts": experts, "top": top}}
    gru = {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}
    att = {"type": "latent_attention", "mlp": mlp,
           "mixer": {"heads": width // 128, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192.0 ** -0.5,
                     "rot": {"base": 10000.0, "dims": 64}}}
    return {"architecture": "Goletar", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "layers": [gru if i % 2 == 0 else att for i in range(n_layers)],
            "embedding": {"bigram": {"buckets": 100003, "mul_prev": 9973, "mul_cur": 31}}}


def build_goletar(config, seed=0, dtype="bfloat16", **model_kw):
    """A finalized Goletar model with random weights made on the device."""
    from . import goletar
    from .layered import Ff, LayeredModel, Mixer
    from .types import BF16
    kw, layers = goletar.describe(config)
    m = LayeredModel(layers, dtype=dtype, **kw, **model_kw)
    gen = torch.Generator(device="cuda").manual_seed(seed)
    W = kw["hidden_size"]

    def shape(role, d):
        if role in (Role.TOKEN_EMBD, Role.OUTPUT):
            return kw["vocab_size"], W
        if role == Role.BIGRAM_EMBD:
            return kw["bigram_buckets"] + 1, W
        if role in (Role.OUTPUT_NORM, Role.MIX_PRE_NORM, Role.MIX_POST_NORM, Role.FF_PRE_NORM, Role.FF_POST_NORM):
            return 1, 1
        latent = d.mixer == Mixer.LATENT_ATTENTION
        return {Role.MIX_OUTPUT: (W, d.n_heads * d.value_dim if latent else d.recurrent_width),
                Role.LATENT_Q: (d.n_heads * (d.head_dim + d.rot_dim), W), Role.LATENT_DOWN: (d.kv_rank + d.rot_dim, W), Role.LATENT_NORM: (1, d.kv_rank),
                Role.LATENT_UP_K: (d.n_heads * d.head_dim, d.kv_rank), Role.LATENT_UP_V: (d.n_heads * d.value_dim, d.kv_rank),
                Role.LATENT_SINK: (1, d.n_heads), Role.LATENT_GATE: (d.n_heads, W), Role.GRU_Z: (d.recurrent_width, W), Role.GRU_X: (d.recurrent_width, W),
                Role.GRU_GATE: (d.recurrent_width, W), Role.GRU_Z_BIAS: (1, d.recurrent_width), Role.GRU_X_BIAS: (1, d.recurrent_width),
                Role.ROUTER: (d.n_experts, W), Role.EXPERT_GATE: (d.ff_width, W), Role.EXPERT_UP: (d.ff_width, W), Role.EXPERT_DOWN: (W, d.ff_width)}[role]

    for _, role, layer, expert in goletar.tensor_roles(layers):
        rows, cols = shape(role, layers[layer])
        v = torch.randn(rows, cols, device="cuda", dtype=torch.bfloat16, generator=gen)
        if rows > 1 and role not in (Role.TOKEN_EMBD, Role.BIGRAM_EMBD):
            v *= cols ** -0.5
        elif rows * cols == 1 or role == Role.LATENT_NORM:
            v.fill_(1.0)
        m.add_tensor(role, layer, BF16, rows, cols, v, expert=expert)
    torch.cuda.synchronize()
    m.finalize()
    return m


def piditar_config(width, n_layers, vocab=32768, ff=None):
    """A Piditar configuration whose layers have the shapes of a real model of this width: real-gated recurrence, attention with
    heads of 128 in groups of four, real-gated recurrence, state-space recurrence with heads of 64 and a state of 128, in turn."""
    mlp = {"kind": "dense", "ff": ff or 2 * width}
    lru = {"type": "rglru", "mixer": {"width": width, "blocks": width // 256, "conv": 4}, "mlp": mlp}
    att = {"type": "attention", "mlp": mlp,
           "mixer": {"heads": width // 128, "kv_heads": width // 512, "dim": 128, "vdim": 128, "scale": 128.0 ** -0.5, "softcap": 50.0,
                     "rot": {"base": 500000.0, "dims": 128}}}
    ssm = {"type": "mamba2", "mixer": {"heads": width // 32, "vdim": 64, "state": 128, "groups": 8, "norm_groups": 8, "conv": 4}, "mlp": mlp}
    return {"architecture": "Piditar", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "layers": [(lru, att, lru, ssm)[i % 4] for i in range(n_layers)], "loop": {"start": 0, "stop": 1, "times": 1}}


def build_piditar(config, seed=0, dtype="bfloat16", **model_kw):
    """A finalized Piditar model with random weights made on the device."""
    from . import piditar
    from .layered import LayeredModel, Mixer
    from .types import BF16
    kw, layers = piditar.describe(config)
    m = LayeredModel(layers, dtype=dtype, **kw, **model_kw)
    gen = torch.Generator(device="cuda").manual_seed(seed)
    W = kw["hidden_size"]

    def shape(role, d):
        H, inner = d.n_heads, d.n_heads * d.value_dim
        w, b = d.recurrent_width, d.recurrent_width // d.n_blocks if d.n_blocks else 0
        channels = inner + 2 * d.n_groups * d.state_size if d.mixer == Mixer.SSM else w
        return {Role.TOKEN_EMBD: (kw["vocab_size"], W), Role.OUTPUT_NORM: (1, W), Role.MIX_PRE_NORM: (1, W), Role.FF_PRE_NORM: (1, W),
                Role.MIX_OUTPUT: (W, w if d.mixer == Mixer.RGLRU else inner), Role.FFN_GATE: (d.ff_width, W), Role.FFN_UP: (d.ff_width, W),
                Role.FFN_DOWN: (W, d.ff_width), Role.ATTN_Q: (H * d.head_dim, W), Role.ATTN_K: (d.n_kv_heads * d.head_dim, W),
                Role.ATTN_V: (d.n_kv_heads * d.value_dim, W), Role.ATTN_Q_BIAS: (1, H * d.head_dim), Role.ATTN_K_BIAS: (1, d.n_kv_heads * d.head_dim),
                Role.ATTN_V_BIAS: (1, d.n_kv_heads * d.value_dim), Role.CONV: (channels, d.conv_taps), Role.CONV_BIAS: (1, channels),
                Role.LRU_OUT: (w, W), Role.LRU_IN: (w, W), Role.LRU_OUT_BIAS: (1, w), Role.LRU_IN_BIAS: (1, w), Role.LRU_DECAY_GATE: (w, b),
                Role.LRU_INPUT_GATE: (w, b), Role.LRU_DECAY_GATE_BIAS: (1, w), Role.LRU_INPUT_GATE_BIAS: (1, w), Role.LRU_LAMBDA: (1, w),
                Role.SSM_IN: (inner + channels + H, W), Role.SSM_DT_BIAS: (1, H), Role.SSM_A_LOG: (1, H), Role.SSM_D: (1, H),
                Role.SSM_NORM: (1, inner)}[role]

    for _, role, layer, _ in piditar.tensor_roles(layers):
        rows, cols = shape(role, layers[layer])
        v = torch.randn(rows, cols, device="cuda", dtype=torch.bfloat16, generator=gen)
        if rows > 1 and role != Role.TOKEN_EMBD:
            v *= cols ** -0.5
        elif role in (Role.OUTPUT_NORM, Role.MIX_PRE_NORM, Role.FF_PRE_NORM):
            v.fill_(0.0)
        m.add_tensor(role, layer, BF16, rows, cols, v)
    torch.cuda.synchronize()
    m.finalize()
    return m


def prompt_tokens(n, vocab, seed):
    """Uniform-random token ids, reproducible without numpy's generator state."""
    mask = (1 << 64) - 1
    out = np.empty(n, dtype=np.uint32)
    for i in range(n):
        x = (i + seed * 0x9E3779B97F4A7C15 + 0x9E3779B97F4A7C15) & mask
        x = ((x ^ (x >> 30)) * 0xBF58476D1CE4E5B9) & mask
        x = ((x ^ (x >> 27)) * 0x94D049BB133111EB) & mask
        x ^= x >> 31
        out[i] = x % vocab
    return out
