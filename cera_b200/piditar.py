"""The Piditar design: a decoder whose layers mix tokens by attention over grouped heads with soft-capped scores, a real-gated
linear recurrence or a state-space recurrence, with a gated unit as feed-forward, zero-centred norm weights ahead of every
sublayer, a scaled embedding that is also the head, and a range of layers that runs several times.

Maps config.json and the tensor names of model.safetensors onto the layer descriptions and tensor roles of
cera_cuda_model_create_layered; everything below runs in the library.
"""
import json
import math
import os

from .layered import Ff, LayerDesc, LayeredModel, Mixer
from .model import Role

LRU_DECAY = 8.0     # log a = -LRU_DECAY * gate * softplus(lambda)
NORM_OFFSET = 1.0   # norm weights are stored around zero


def _layer(i, entry):
    d = LayerDesc()
    m = entry["mixer"]
    if entry["type"] == "attention":
        rot = m["rot"]
        d.mixer = Mixer.ATTENTION
        d.n_heads, d.n_kv_heads, d.head_dim, d.value_dim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        d.rot_dim, d.rope_base, d.attn_scale, d.softcap = rot["dims"], rot["base"], m["scale"], m.get("softcap") or 0.0
        d.qk_norm = d.attn_bias = 1
    elif entry["type"] == "rglru":
        d.mixer = Mixer.RGLRU
        d.recurrent_width, d.n_blocks, d.conv_taps, d.decay = m["width"], m["blocks"], m["conv"], LRU_DECAY
    elif entry["type"] == "mamba2":
        d.mixer = Mixer.SSM
        d.n_heads, d.value_dim, d.state_size, d.n_groups = m["heads"], m["vdim"], m["state"], m["groups"]
        d.n_norm_groups, d.conv_taps = m["norm_groups"], m["conv"]
    else:
        raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
    mlp = entry.get("mlp")
    if mlp is None:
        d.ff = Ff.NONE
    elif mlp["kind"] == "dense":
        d.ff = Ff.GATED
        d.ff_width, d.act_limit, d.act_alpha, d.act_shift = mlp["ff"], math.inf, 1.0, 0.0  # silu(gate) * up
    else:
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    return d


def describe(config):
    """config.json (parsed) -> (model keywords, layer descriptions)."""
    loop = config.get("loop") or {}
    start, stop = loop.get("start", 0), loop.get("stop", 0)
    return (dict(hidden_size=config["width"], vocab_size=config["vocab"], norm_eps=config["norm"]["eps"], embedding_scale=config["embedding"]["scale"],
                 norm_offset=NORM_OFFSET, tied_output=1, no_post_norms=1, loop_start=start, loop_stop=stop,
                 loop_times=loop["times"] if stop > start else 1),
            [_layer(i, e) for i, e in enumerate(config["layers"])])


_MIXER = {
    Mixer.ATTENTION: [("q", Role.ATTN_Q), ("q.b", Role.ATTN_Q_BIAS), ("k", Role.ATTN_K), ("k.b", Role.ATTN_K_BIAS), ("v", Role.ATTN_V),
                      ("v.b", Role.ATTN_V_BIAS), ("o", Role.MIX_OUTPUT)],
    Mixer.RGLRU: [("y", Role.LRU_OUT), ("y.b", Role.LRU_OUT_BIAS), ("x", Role.LRU_IN), ("x.b", Role.LRU_IN_BIAS), ("conv", Role.CONV),
                  ("conv.b", Role.CONV_BIAS), ("ra", Role.LRU_DECAY_GATE), ("ra.b", Role.LRU_DECAY_GATE_BIAS), ("ri", Role.LRU_INPUT_GATE),
                  ("ri.b", Role.LRU_INPUT_GATE_BIAS), ("lam", Role.LRU_LAMBDA), ("o", Role.MIX_OUTPUT)],
    Mixer.SSM: [("in", Role.SSM_IN), ("conv", Role.CONV), ("conv.b", Role.CONV_BIAS), ("dt_bias", Role.SSM_DT_BIAS), ("A_log", Role.SSM_A_LOG),
                ("D", Role.SSM_D), ("norm", Role.SSM_NORM), ("o", Role.MIX_OUTPUT)],
}
_FF = [("gate", Role.FFN_GATE), ("up", Role.FFN_UP), ("down", Role.FFN_DOWN)]


def tensor_roles(layers):
    """Every tensor of the design: (name, role, layer, None)."""
    out = [("embed", Role.TOKEN_EMBD, 0, None), ("final.norm", Role.OUTPUT_NORM, 0, None)]
    for i, d in enumerate(layers):
        out.append((f"l{i}.norm1", Role.MIX_PRE_NORM, i, None))
        out += [(f"l{i}.mix.{n}", r, i, None) for n, r in _MIXER[d.mixer]]
        if d.ff != Ff.NONE:
            out.append((f"l{i}.norm2", Role.FF_PRE_NORM, i, None))
            out += [(f"l{i}.mlp.{n}", r, i, None) for n, r in _FF]
    return out


def load_piditar(path, config=None, max_seq_len=4096, dtype="bfloat16", device=0):
    """A finalized model from a folder with config.json and model.safetensors."""
    if config is None:
        with open(os.path.join(path, "config.json")) as f:
            config = json.load(f)
    kw, layers = describe(config)
    model = LayeredModel(layers, max_seq_len=max_seq_len, dtype=dtype, device=device, **kw)
    model.load(path, tensor_roles(layers))
    return model
