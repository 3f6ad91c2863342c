"""The Goletar design: a decoder whose layers mix tokens by latent attention or a minGRU recurrence, with routed experts,
a bigram embedding and single-number norms before and after every sublayer.

Maps config.json and the tensor names of model.safetensors onto the layer descriptions and tensor roles of
cera_cuda_model_create_layered; everything below runs in the library.
"""
import json
import os

from .layered import LayerDesc, LayeredModel, Mixer, Ff
from .model import Role

# the expert unit: min(g) * sigmoid(ALPHA g) * (u + SHIFT)
ACT_ALPHA = 1.702
ACT_SHIFT = 1.0


def _layer(i, entry):
    d = LayerDesc()
    m = entry["mixer"]
    if entry["type"] == "latent_attention":
        rot = m["rot"]
        if rot["dims"] != m["rot_dim"]:
            raise ValueError(f"layer {i}: {rot['dims']} rotated dimensions in a rotated part of {m['rot_dim']}")
        d.mixer = Mixer.LATENT_ATTENTION
        d.n_heads, d.head_dim, d.rot_dim, d.value_dim, d.kv_rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        d.rope_base, d.attn_scale = rot["base"], m["scale"]
    elif entry["type"] == "mingru":
        d.mixer = Mixer.MINGRU
        d.recurrent_width = m["width"]
    else:
        raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
    mlp = entry.get("mlp")
    if mlp is None:
        d.ff = Ff.NONE
    elif mlp["kind"] == "moe":
        d.ff = Ff.MOE
        d.ff_width, d.act_limit = mlp["expert"]["ff"], mlp["expert"]["limit"]
        d.n_experts, d.n_used = mlp["router"]["experts"], mlp["router"]["top"]
        d.act_alpha, d.act_shift = ACT_ALPHA, ACT_SHIFT
        d.router_softmax, d.router_renorm, d.weight_input = 0, 0, 1
    else:
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    return d


def describe(config):
    """config.json (parsed) -> (model keywords, layer descriptions)."""
    b = config["embedding"]["bigram"]
    return (dict(hidden_size=config["width"], vocab_size=config["vocab"], norm_eps=config["norm"]["eps"], bigram_buckets=b["buckets"],
                 bigram_mul_prev=b["mul_prev"], bigram_mul_cur=b["mul_cur"]),
            [_layer(i, e) for i, e in enumerate(config["layers"])])


_LATENT = [("q", Role.LATENT_Q), ("dkv", Role.LATENT_DOWN), ("dkv.norm", Role.LATENT_NORM), ("uk", Role.LATENT_UP_K), ("uv", Role.LATENT_UP_V),
           ("sink", Role.LATENT_SINK), ("g", Role.LATENT_GATE), ("o", Role.MIX_OUTPUT)]
_MINGRU = [("z", Role.GRU_Z), ("z.b", Role.GRU_Z_BIAS), ("x", Role.GRU_X), ("x.b", Role.GRU_X_BIAS), ("g", Role.GRU_GATE), ("o", Role.MIX_OUTPUT)]
_EXPERT = [("gate", Role.EXPERT_GATE), ("up", Role.EXPERT_UP), ("down", Role.EXPERT_DOWN)]


def tensor_roles(layers):
    """Every tensor of the design: (name, role, layer, expert or None)."""
    out = [("embed", Role.TOKEN_EMBD, 0, None), ("bigram", Role.BIGRAM_EMBD, 0, None), ("final.norm", Role.OUTPUT_NORM, 0, None),
           ("head", Role.OUTPUT, 0, None)]
    for i, d in enumerate(layers):
        out += [(f"l{i}.norm1", Role.MIX_PRE_NORM, i, None), (f"l{i}.norm1b", Role.MIX_POST_NORM, i, None)]
        out += [(f"l{i}.mix.{n}", r, i, None) for n, r in (_LATENT if d.mixer == Mixer.LATENT_ATTENTION else _MINGRU)]
        if d.ff == Ff.MOE:
            out += [(f"l{i}.norm2", Role.FF_PRE_NORM, i, None), (f"l{i}.norm2b", Role.FF_POST_NORM, i, None), (f"l{i}.mlp.router", Role.ROUTER, i, None)]
            out += [(f"l{i}.mlp.e{e}.{n}", r, i, e) for e in range(d.n_experts) for n, r in _EXPERT]
    return out


def load_goletar(path, config=None, max_seq_len=4096, dtype="bfloat16", device=0):
    """A finalized model from a folder with config.json and model.safetensors."""
    if config is None:
        with open(os.path.join(path, "config.json")) as f:
            config = json.load(f)
    kw, layers = describe(config)
    model = LayeredModel(layers, max_seq_len=max_seq_len, dtype=dtype, device=device, **kw)
    model.load(path, tensor_roles(layers))
    return model
