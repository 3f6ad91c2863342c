"""Plain CPU implementation of the Goletar design in float64 numpy, one function per mechanism.

Slow and direct: every function takes whole sequences, loops over positions where the equations do, and keeps no cache
(the recurrence apart, which is one).  It shares nothing with cera_b200: tests compare the CUDA path against it."""
import json
import struct

import numpy as np

F = np.float64


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight; weight is a number or a vector."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * weight


def embed(tokens, table, bigram, buckets, mul_prev, mul_cur):
    """Token row plus the row hashed from (previous token, token); the first token takes the spare last row."""
    out = np.empty((len(tokens), table.shape[1]), dtype=F)
    for t, tok in enumerate(tokens):
        row = buckets if t == 0 else (int(tokens[t - 1]) * mul_prev + int(tok) * mul_cur) % buckets
        out[t] = table[tok] + bigram[row]
    return out


def rotate(x, pos, base):
    """Adjacent pairs (2i, 2i+1) of the last axis turned by pos * base^(-2i/d)."""
    d = x.shape[-1]
    out = np.empty_like(x)
    for i in range(d // 2):
        a = pos * float(base) ** (-2.0 * i / d)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def sink_softmax(scores, sink):
    """Softmax over the last axis whose denominator also holds exp(sink)."""
    m = max(scores.max(), sink)
    e = np.exp(scores - m)
    return e / (e.sum() + np.exp(sink - m))


def latent_attention(h, w, c, eps):
    """h: [T, width]; w: q, dkv, dkv.norm, uk, uv, sink, g, o; c: the mixer's sizes."""
    H, d, r, dv, rank = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    T = len(h)
    q = (h @ w["q"].T).reshape(T, H, d + r)
    down = h @ w["dkv"].T
    lat = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    k_rot = np.stack([rotate(down[t, rank:], t, c["rot"]["base"]) for t in range(T)])
    q_rot = np.stack([rotate(q[t, :, d:], t, c["rot"]["base"]) for t in range(T)])
    k = (lat @ w["uk"].T).reshape(T, H, d)
    v = (lat @ w["uv"].T).reshape(T, H, dv)
    gate = sigmoid(h @ w["g"].T)
    out = np.zeros((T, H, dv), dtype=F)
    for t in range(T):
        for i in range(H):
            s = (k[:t + 1, i] @ q[t, i, :d] + k_rot[:t + 1] @ q_rot[t, i]) * c["scale"]
            out[t, i] = (sink_softmax(s, w["sink"][i]) @ v[:t + 1, i]) * gate[t, i]
    return out.reshape(T, H * dv) @ w["o"].T


def mingru(h, w, state=None):
    """State of every position: S_t = (1 - z_t) S_(t-1) + z_t * candidate_t."""
    z = sigmoid(h @ w["z"].T + w["z.b"])
    u = h @ w["x"].T + w["x.b"]
    cand = np.where(u >= 0, u + 0.5, sigmoid(u))
    gate = silu(h @ w["g"].T)
    s = np.zeros(z.shape[1], dtype=F) if state is None else state
    y = np.empty_like(z)
    for t in range(len(h)):
        s = (1.0 - z[t]) * s + z[t] * cand[t]
        y[t] = s * gate[t]
    return y @ w["o"].T, s


def clamped_glu(x, gate, up, down, limit):
    g = np.minimum(x @ gate.T, limit)
    u = np.clip(x @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, router, top):
    """Chosen experts (largest sigmoid scores, lower index first on ties) and their scores."""
    s = sigmoid(h @ router.T)
    order = np.argsort(-s, axis=-1, kind="stable")[..., :top]
    return order, np.take_along_axis(s, order, axis=-1)


def moe(h, w, c):
    ids, wt = route(h, w["router"], c["router"]["top"])
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(ids[t], wt[t]):
            out[t] += clamped_glu(s * h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], c["expert"]["limit"])
    return out


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def layers_out(tokens, config, weights):
    """Residual stream after the embedding and after every layer."""
    eps, b = config["norm"]["eps"], config["embedding"]["bigram"]
    x = embed(tokens, weights["embed"], weights["bigram"], b["buckets"], b["mul_prev"], b["mul_cur"])
    seen = [x]
    for i, layer in enumerate(config["layers"]):
        w = _sub(weights, f"l{i}.")
        h = rms_norm(x, w["norm1"], eps)
        mix = _sub(w, "mix.")
        if layer["type"] == "latent_attention":
            y = latent_attention(h, mix, layer["mixer"], eps)
        else:
            y, _ = mingru(h, mix)
        x = x + rms_norm(y, w["norm1b"], eps)
        if layer["mlp"] is not None:
            y = moe(rms_norm(x, w["norm2"], eps), _sub(w, "mlp."), layer["mlp"])
            x = x + rms_norm(y, w["norm2b"], eps)
        seen.append(x)
    return seen


def logits(tokens, config, weights):
    x = layers_out(tokens, config, weights)[-1]
    return rms_norm(x, weights["final.norm"], config["norm"]["eps"]) @ weights["head"].T


def greedy(prompt, n, config, weights):
    toks = [int(t) for t in prompt]
    for _ in range(n):
        toks.append(int(np.argmax(logits(toks, config, weights)[-1])))
    return toks[len(prompt):]


# ---- random models ------------------------------------------------------------------------------------------------

def tensor_shapes(config):
    W = config["width"]
    shapes = {"embed": (config["vocab"], W), "bigram": (config["embedding"]["bigram"]["buckets"] + 1, W), "final.norm": (),
              "head": (config["vocab"], W)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        shapes.update({p + "norm1": (), p + "norm1b": ()})
        if layer["type"] == "latent_attention":
            H = m["heads"]
            shapes.update({p + "mix.q": (H * (m["dim"] + m["rot_dim"]), W), p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], W),
                           p + "mix.dkv.norm": (m["kv_rank"],), p + "mix.uk": (H * m["dim"], m["kv_rank"]),
                           p + "mix.uv": (H * m["vdim"], m["kv_rank"]), p + "mix.sink": (H,), p + "mix.g": (H, W),
                           p + "mix.o": (W, H * m["vdim"])})
        else:
            n = m["width"]
            shapes.update({p + "mix.z": (n, W), p + "mix.z.b": (n,), p + "mix.x": (n, W), p + "mix.x.b": (n,), p + "mix.g": (n, W),
                           p + "mix.o": (W, n)})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["expert"]["ff"]
            shapes.update({p + "norm2": (), p + "norm2b": (), p + "mlp.router": (layer["mlp"]["router"]["experts"], W)})
            for e in range(layer["mlp"]["router"]["experts"]):
                shapes.update({f"{p}mlp.e{e}.gate": (ff, W), f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
    return shapes


def to_bf16(x):
    """float -> nearest bfloat16 (ties to even), as uint16 bits."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(bits):
    return (bits.astype(np.uint32) << 16).view(np.float32)


def random_weights(config, seed):
    """bf16-representable weights of a scale that keeps every branch alive, as float64."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf.startswith("norm"):
            v = 1.0 + 0.3 * rng.standard_normal(shape)
        elif leaf in ("embed", "bigram"):
            v = rng.standard_normal(shape)
        elif leaf == "sink":
            v = rng.standard_normal(shape) + 1.0
        elif leaf == "b":
            v = rng.standard_normal(shape)
        else:
            gain = {"router": 1.0, "gate": 1.5, "up": 1.5, "z": 1.5, "x": 1.5, "q": 1.5}.get(leaf, 1.0)
            v = gain * rng.standard_normal(shape) / np.sqrt(shape[-1])
        out[name] = from_bf16(to_bf16(np.asarray(v))).astype(F).reshape(shape)
    return out


def save(path, config, weights):
    """config.json and model.safetensors in folder `path` (a pathlib.Path)."""
    (path / "config.json").write_text(json.dumps(config))
    head, blobs, at = {}, [], 0
    for name, v in weights.items():
        b = to_bf16(v).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    text = json.dumps(head).encode()
    with open(path / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
