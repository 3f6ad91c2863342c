"""Small random Piditar models for the tests: configurations and the change that makes one key stand out."""
import copy

import numpy as np

import piditar_ref as P
from goletar_util import BF16_TOL, F32_TOL, TOL, error, tokens  # noqa: F401


def attention(heads=6, kv_heads=2, dim=40, vdim=24, rot=16, base=1000.0, scale=0.2, softcap=6.0, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap,
                      "rot": {"base": base, "dims": rot}}}


def rglru(width=90, blocks=3, conv=3, mlp=None):
    return {"type": "rglru", "mlp": mlp, "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def mamba2(heads=4, vdim=24, state=20, groups=2, norm_groups=1, conv=4, mlp=None):
    return {"type": "mamba2", "mlp": mlp,
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def unit(ff=56):
    return {"kind": "dense", "ff": ff}


def config(layers, width=72, vocab=101, eps=1e-5, scale=1.5, loop=None):
    return {"architecture": "Piditar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "embedding": {"scale": scale},
            "loop": loop or {"start": 0, "stop": 1, "times": 1}}


def aim(cfg, weights, q_tok, k_tok):
    """Change layer 0 (attention whose heads have unrotated dimensions, no layer of a repeated pass) so that queries of q_tok and
    keys of k_tok point the same way in every head, wherever they stand, and what is read shows beside the embedding."""
    w, m, eps = copy.deepcopy(weights), cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    h = {t: P.norm(w["embed"][t] * cfg["embedding"]["scale"], w["l0.norm1"], eps) for t in (q_tok, k_tok)}
    way = np.zeros(m["dim"])
    way[m["rot"]["dims"]:] = np.where(np.arange(m["dim"] - m["rot"]["dims"]) % 2, -12.0, 12.0)
    for name, tok, n in (("l0.mix.q", q_tok, m["heads"]), ("l0.mix.k", k_tok, m["kv_heads"])):
        v = w[name] + np.outer(np.tile(way, n), h[tok] / (h[tok] @ h[tok]))
        w[name] = P.from_bf16(P.to_bf16(v)).astype(np.float64)
    w["l0.mix.o"] *= 4.0
    return w
