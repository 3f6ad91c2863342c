"""Small random Goletar models for the tests: configurations, the bump that makes one key stand out, error measures."""
import copy

import numpy as np

import goletar_ref as G

F32_TOL, BF16_TOL = 1e-5, 2e-2  # rms over the vocabulary of the logits' difference (mean taken off), in units of their spread
TOL = {"float32": F32_TOL, "bfloat16": BF16_TOL}


def attention(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=48, base=1000.0, scale=0.2, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def mingru(width=100, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def moe(ff=40, limit=1.5, experts=5, top=2):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(layers, width=72, vocab=101, eps=1e-5, buckets=53, mul_prev=31, mul_cur=17):
    return {"architecture": "Goletar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}


def tokens(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def error(got, want, quantile=1.0):
    """Worst position's error, or a quantile over the positions: with 16-bit rounding a token whose experts are a close call may
    go to another one, and a test that routes freely looks at most positions instead of all."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    d = got - want
    d -= d.mean(axis=-1, keepdims=True)
    return float(np.quantile(np.sqrt((d * d).mean(axis=-1)) / np.maximum(want.std(axis=-1), 1e-6), quantile))


def aim(cfg, weights, layer, q_tok, k_tok, bump):
    """Change layer `layer` (0, an attention layer; the bigram rows are cleared) so that a query of token q_tok scores `bump`
    higher on keys of token k_tok than chance would have it."""
    w = copy.deepcopy(weights)
    w["bigram"][:] = 0.0
    m, eps, p = cfg["layers"][layer]["mixer"], cfg["norm"]["eps"], f"l{layer}."
    h = {t: G.rms_norm(w["embed"][t], w[p + "norm1"], eps) for t in (q_tok, k_tok)}
    c = G.rms_norm((w[p + "mix.dkv"] @ h[k_tok])[:m["kv_rank"]], w[p + "mix.dkv.norm"], eps)
    k = (w[p + "mix.uk"] @ c).reshape(m["heads"], m["dim"])
    q = w[p + "mix.q"].reshape(m["heads"], m["dim"] + m["rot_dim"], -1)
    for i in range(m["heads"]):
        want = bump / m["scale"] / (k[i] @ k[i]) * k[i]
        q[i, :m["dim"]] += np.outer(want, h[q_tok]) / (h[q_tok] @ h[q_tok])
    w[p + "mix.q"] = G.from_bf16(G.to_bf16(q.reshape(w[p + "mix.q"].shape))).astype(np.float64)
    return w
