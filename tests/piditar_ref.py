"""Plain CPU implementation of the Piditar design in float64 numpy, one function per mechanism.

Slow and direct, as goletar_ref.py: whole sequences in, a loop over positions where an equation has one, no cache besides
the recurrences' own state.  It shares nothing with cera_b200: tests compare the CUDA path against it."""
import numpy as np

from goletar_ref import F, from_bf16, rms_norm, save, sigmoid, silu, to_bf16  # noqa: F401


def softplus(x):
    return np.logaddexp(0.0, x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


def causal_conv(x, taps, bias):
    """x: [T, channels]; taps: [channels, n], the last one meets the current position; positions before the start are zero."""
    T, n = len(x), taps.shape[1]
    out = np.empty_like(x)
    for t in range(T):
        out[t] = bias
        for k in range(n):
            at = t - (n - 1 - k)
            if at >= 0:
                out[t] += taps[:, k] * x[at]
    return out


def rotate_front(x, pos, dims, base):
    """The first `dims` entries of the last axis turn in adjacent pairs by pos * base^(-2i / dims); the others stay."""
    out = np.array(x, dtype=F)
    for i in range(dims // 2):
        a = pos * float(base) ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def attention(h, w, c, eps):
    """Grouped heads; queries and keys rotated, then of unit root mean square; scores soft-capped.  h: [T, width]."""
    H, G, d, dv, T = c["heads"], c["kv_heads"], c["dim"], c["vdim"], len(h)
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, d)
    k = (h @ w["k"].T + w["k.b"]).reshape(T, G, d)
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, dv)
    turn = lambda x: np.stack([rotate_front(x[t], t, c["rot"]["dims"], c["rot"]["base"]) for t in range(T)])  # noqa: E731
    q, k = rms_norm(turn(q), 1.0, eps), rms_norm(turn(k), 1.0, eps)
    out = np.zeros((T, H, dv), dtype=F)
    for t in range(T):
        for i in range(H):
            g = i // (H // G)
            s = k[:t + 1, g] @ q[t, i] * c["scale"]
            s = c["softcap"] * np.tanh(s / c["softcap"])
            e = np.exp(s - s.max())
            out[t, i] = e / e.sum() @ v[:t + 1, g]
    return out.reshape(T, H * dv) @ w["o"].T


def rglru(h, w, c, state=None):
    """Gated branch times the real-gated linear recurrence over the convolved branch.  Returns (output, last state)."""
    width, B, T = c["width"], c["blocks"], len(h)
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    n = width // B
    s = np.zeros(width) if state is None else state
    out = np.empty((T, width))
    for t in range(T):
        r, i = np.empty(width), np.empty(width)
        for b in range(B):
            part = slice(b * n, (b + 1) * n)
            r[part] = sigmoid(w["ra"][b] @ u[t, part] + w["ra.b"][b])
            i[part] = sigmoid(w["ri"][b] @ u[t, part] + w["ri.b"][b])
        log_a = -8.0 * r * softplus(w["lam"])
        s = np.exp(log_a) * s + np.sqrt(-np.expm1(2.0 * log_a)) * i * u[t]
        out[t] = s * y[t]
    return out @ w["o"].T, s


def mamba2(h, w, c, eps, state=None):
    """State-space recurrence with a matrix state per head.  Returns (output, last state [heads, N, vdim])."""
    H, P, N, G, T = c["heads"], c["vdim"], c["state"], c["groups"], len(h)
    inner = H * P
    z, xbc, dt = np.split(h @ w["in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    x, b, cc = np.split(silu(causal_conv(xbc, w["conv"], w["conv.b"])), [inner, inner + G * N], axis=1)
    x, b, cc = x.reshape(T, H, P), b.reshape(T, G, N), cc.reshape(T, G, N)
    dt = softplus(dt + w["dt_bias"])
    s = np.zeros((H, N, P)) if state is None else np.array(state)
    y = np.empty((T, H, P))
    for t in range(T):
        for i in range(H):
            g = i // (H // G)
            s[i] = np.exp(-np.exp(w["A_log"][i]) * dt[t, i]) * s[i] + dt[t, i] * np.outer(b[t, g], x[t, i])
            y[t, i] = s[i].T @ cc[t, g] + w["D"][i] * x[t, i]
    y = y.reshape(T, inner) * silu(z)
    parts = y.reshape(T, c["norm_groups"], -1)
    y = rms_norm(parts, 1.0, eps).reshape(T, inner) * w["norm"]
    return y @ w["o"].T, s


def gated_ff(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def norm(x, w, eps):
    """The weight is stored around zero."""
    return rms_norm(x, 1.0 + w, eps)


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def passes(config):
    """(layer, opens a repeated pass) of every layer run."""
    n, loop = len(config["layers"]), config.get("loop") or {"start": 0, "stop": 0, "times": 1}
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(b)]
    for _ in range(loop["times"] - 1):
        runs += [(i, i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def layer(x, kind, sizes, ff, w, eps):
    h, mix = norm(x, w["norm1"], eps), _sub(w, "mix.")
    if kind == "attention":
        x = x + attention(h, mix, sizes, eps)
    elif kind == "rglru":
        x = x + rglru(h, mix, sizes)[0]
    else:
        x = x + mamba2(h, mix, sizes, eps)[0]
    if ff is not None:
        x = x + gated_ff(norm(x, w["norm2"], eps), _sub(w, "mlp."))
    return x


def layers_out(tokens, config, weights):
    """Residual stream after the embedding and after every layer run."""
    eps = config["norm"]["eps"]
    e = weights["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    x, seen = e, [e]
    for i, again in passes(config):
        if again:
            x = x + e
        c = config["layers"][i]
        x = layer(x, c["type"], c["mixer"], c["mlp"], _sub(weights, f"l{i}."), eps)
        seen.append(x)
    return seen


def logits(tokens, config, weights):
    return norm(layers_out(tokens, config, weights)[-1], weights["final.norm"], config["norm"]["eps"]) @ weights["embed"].T


def greedy(prompt, n, config, weights):
    toks = [int(t) for t in prompt]
    for _ in range(n):
        toks.append(int(np.argmax(logits(toks, config, weights)[-1])))
    return toks[len(prompt):]


# ---- random models ------------------------------------------------------------------------------------------------

def tensor_shapes(config):
    W = config["width"]
    shapes = {"embed": (config["vocab"], W), "final.norm": (W,)}
    for i, entry in enumerate(config["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        shapes[p + "norm1"] = (W,)
        if entry["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            mix = {"q": (H * d, W), "q.b": (H * d,), "k": (G * d, W), "k.b": (G * d,), "v": (G * dv, W), "v.b": (G * dv,), "o": (W, H * dv)}
        elif entry["type"] == "rglru":
            n, B, c = m["width"], m["blocks"], m["conv"]
            b = n // B
            mix = {"y": (n, W), "y.b": (n,), "x": (n, W), "x.b": (n,), "conv": (n, c), "conv.b": (n,), "ra": (B, b, b), "ra.b": (B, b), "ri": (B, b, b),
                   "ri.b": (B, b), "lam": (n,), "o": (W, n)}
        else:
            H, inner, gn = m["heads"], m["heads"] * m["vdim"], m["groups"] * m["state"]
            mix = {"in": (2 * inner + 2 * gn + H, W), "conv": (inner + 2 * gn, m["conv"]), "conv.b": (inner + 2 * gn,), "dt_bias": (H,), "A_log": (H,),
                   "D": (H,), "norm": (inner,), "o": (W, inner)}
        shapes.update({p + "mix." + k: v for k, v in mix.items()})
        if entry["mlp"] is not None:
            ff = entry["mlp"]["ff"]
            shapes.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return shapes


def random_weights(config, seed):
    """bf16-representable weights of a scale that keeps every branch alive, as float64."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf, z = name.rsplit(".", 1)[-1], rng.standard_normal(shape)
        if leaf in ("norm1", "norm2"):
            v = 0.3 * z
        elif leaf == "norm":
            v = 0.3 * z + (0.0 if name == "final.norm" else 1.0)
        elif leaf in ("embed", "lam", "D"):
            v = z
        elif leaf == "b":
            v = 0.5 * z
        elif leaf == "dt_bias":
            v = z - 1.0
        elif leaf == "A_log":
            v = z - 1.0
        elif leaf == "conv":
            v = z / np.sqrt(shape[-1])
        else:
            gain = {"gate": 1.5, "up": 1.5, "in": 1.5, "x": 1.5, "y": 1.5}.get(leaf, 1.0)
            v = gain * z / np.sqrt(shape[-1])
        out[name] = from_bf16(to_bf16(np.asarray(v))).astype(F).reshape(shape)
    return out
