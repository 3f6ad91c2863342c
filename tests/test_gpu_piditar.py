"""Piditar on the GPU against the plain float64 implementation: mechanisms alone, cuts of a prompt, decoding, state reuse, keys
far away and at tile edges, long memories, repeated layers, greedy generation through the public entry points."""
import subprocess
import sys

import numpy as np
import pytest

import piditar_ref as P
from gpu_util import need_gpu
from piditar_util import TOL, aim, attention, config, error, mamba2, rglru, tokens, unit

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]

MECHANISMS = {
    "attention": [attention()],
    "attention_one_head": [attention(heads=1, kv_heads=1, dim=16, vdim=16, rot=16, base=50.0, softcap=2.0)],
    "attention_no_sharing": [attention(heads=5, kv_heads=5, dim=24, vdim=40, rot=2)],
    "attention_one_group": [attention(heads=7, kv_heads=1, dim=18, vdim=10, rot=18, softcap=100.0)],
    "attention_many_heads": [attention(heads=40, kv_heads=2, dim=64, vdim=72, rot=48)],
    "attention_wide": [attention(heads=8, kv_heads=2, dim=128, vdim=128, rot=64, scale=0.1, softcap=20.0)],
    "attention_beyond_tiles": [attention(heads=2, kv_heads=1, dim=300, vdim=290, rot=100, scale=0.05)],
    "rglru": [rglru()],
    "rglru_one_block": [rglru(width=130, blocks=1, conv=4)],
    "rglru_many_blocks": [rglru(width=96, blocks=12, conv=2)],
    "rglru_one_tap": [rglru(width=64, blocks=2, conv=1)],
    "rglru_wide": [rglru(width=640, blocks=2, conv=6)],
    "mamba2": [mamba2()],
    "mamba2_one_head": [mamba2(heads=1, vdim=33, state=7, groups=1, conv=2)],
    "mamba2_group_per_head": [mamba2(heads=6, vdim=16, state=16, groups=6, norm_groups=6, conv=1)],
    "mamba2_norm_across_heads": [mamba2(heads=6, vdim=20, state=48, groups=3, norm_groups=4, conv=5)],
    "mamba2_wide": [mamba2(heads=4, vdim=64, state=128, groups=1, norm_groups=1)],
    "mamba2_wide_values": [mamba2(heads=2, vdim=130, state=100, groups=2, norm_groups=2, conv=3)],
    "mamba2_state_200": [mamba2(heads=2, vdim=72, state=200, groups=1)],
    "mamba2_large_state": [mamba2(heads=2, vdim=48, state=300, groups=1)],
    "unit": [rglru(width=8, blocks=1, mlp=unit(200))],
    "unit_narrow": [rglru(width=8, blocks=1, mlp=unit(9))],
    "repeated": [rglru(), attention(mlp=unit())],
}
LOOPS = {"repeated": {"start": 0, "stop": 2, "times": 3}}
MIXED = [mamba2(), rglru(mlp=unit()), attention(mlp=unit(77)), mamba2(heads=3, groups=3, norm_groups=3, conv=2, mlp=unit())]


def mixed(loop=True):
    return config(MIXED, loop={"start": 1, "stop": 3, "times": 2} if loop else None)


def load(tmp_path, cfg, w, dtype, max_seq_len):
    need_gpu()
    from cera_b200 import load_model
    tmp_path.mkdir(exist_ok=True)
    P.save(tmp_path, cfg, w)
    return load_model(tmp_path, dtype=dtype, max_seq_len=max_seq_len)


def feed(model, toks, sizes):
    """All logits of a fresh sequence cut into portions of the given sizes (the last one repeats)."""
    model.truncate_kv(0)
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        out.append(model.forward_prefill_logits_at(toks[at:at + n], at, list(range(n))))
        at, i = at + n, i + 1
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_alone(tmp_path, name, dtype):
    cfg = config(MECHANISMS[name], width=136 if "wide" in name else 72, loop=LOOPS.get(name))
    w = P.random_weights(cfg, 11)
    toks = tokens(150, cfg["vocab"], 12)
    want = P.logits(toks, cfg, w)
    m = load(tmp_path, cfg, w, dtype, 160)
    for sizes in ([150], [40, 1], [1]):
        assert error(feed(m, toks, sizes), want) < TOL[dtype], sizes
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[2], [3, 2, 15, 16, 17, 1, 64, 63, 2], [100, 2, 7], [129, 128, 1, 1], [65, 1, 127, 2, 1, 33]])
def test_portions_of_a_prompt(tmp_path, dtype, sizes):
    cfg = mixed()
    w = P.random_weights(cfg, 21)
    toks = tokens(330, cfg["vocab"], 22)
    m = load(tmp_path, cfg, w, dtype, 330)
    assert error(feed(m, toks, sizes), P.logits(toks, cfg, w)) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("width,vocab,eps,loop", [(64, 40, 1e-6, {"start": 0, "stop": 4, "times": 2}), (65, 1000, 1e-3, {"start": 3, "stop": 4, "times": 4}),
                                                  (250, 77, 1e-2, {"start": 0, "stop": 1, "times": 5})])
def test_other_sizes(tmp_path, width, vocab, eps, loop):
    cfg = config([attention(heads=4, kv_heads=4, dim=10, rot=6, vdim=9, softcap=3.0), mamba2(heads=5, vdim=width // 5, state=9, groups=1, norm_groups=5, conv=2),
                  rglru(width=width + 5, blocks=1 if width % 2 else 3, conv=5, mlp=unit(65)), mamba2(heads=2, vdim=8, state=64, groups=2, mlp=unit(31))], width=width,
                 vocab=vocab, eps=eps, scale=0.25, loop=loop)
    w = P.random_weights(cfg, 23)
    toks = tokens(90, vocab, 24)
    want = P.logits(toks, cfg, w)
    for dtype in DTYPES:
        m = load(tmp_path / dtype, cfg, w, dtype, 90)
        got = feed(m, toks, [60, 5, 1])
        # bf16: a normed part whose numbers nearly cancel carries their rounding into the logits
        assert error(got, want, 1.0 if dtype == "float32" else 0.5) < TOL[dtype]
        assert error(got, want) < 10 * TOL[dtype]
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sequence_does_not_see_the_one_before(tmp_path, dtype):
    cfg = mixed()
    w = P.random_weights(cfg, 31)
    m = load(tmp_path, cfg, w, dtype, 256)
    for n, seed in ((256, 1), (3, 2), (1, 3), (100, 4), (17, 5), (256, 6)):
        toks = tokens(n, cfg["vocab"], seed)
        assert error(feed(m, toks, [max(n - 4, 1), 1]), P.logits(toks, cfg, w)) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_snapshots_interleave_sequences(tmp_path, dtype):
    cfg = mixed()
    w = P.random_weights(cfg, 32)
    m = load(tmp_path, cfg, w, dtype, 96)
    seqs = [tokens(n, cfg["vocab"], 40 + n) for n in (70, 33, 96)]
    want = [P.logits(t, cfg, w) for t in seqs]
    m.truncate_kv(0)
    states, at, got = [m.snapshot()] * 3, [0, 0, 0], [[], [], []]
    step = [17, 3, 30]
    while any(a < len(t) for a, t in zip(at, seqs)):
        for i, t in enumerate(seqs):
            if at[i] == len(t):
                continue
            m.truncate_kv(0)
            m.restore(states[i])
            n = min(step[i], len(t) - at[i])
            got[i].append(m.forward_prefill_logits_at(t[at[i]:at[i] + n], at[i], list(range(n))))
            at[i] += n
            states[i] = m.snapshot()
            step[i] = 1 if step[i] > 1 else 5
    for g, x in zip(got, want):
        assert error(np.concatenate(g), x) < TOL[dtype]
    m.close()


EDGES = [0, 1, 15, 16, 31, 32, 63, 64, 65, 127, 128, 129, 255, 256, 300]


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_key_at_every_edge(tmp_path, dtype):
    """One key stands out for the queries of one token; the oracle without that key (a mistake planted there) is far off, so a
    key lost at a tile's or split's edge shows."""
    cfg = config([attention(heads=4, kv_heads=2, dim=32, rot=16, vdim=32, base=10000.0, scale=0.6, softcap=30.0)])
    q_tok, k_tok = 7, 9
    w = aim(cfg, P.random_weights(cfg, 41), q_tok, k_tok)
    m = load(tmp_path, cfg, w, dtype, 340)
    base = [t if t not in (q_tok, k_tok) else 11 for t in tokens(330, 101, 42)]
    for edge in EDGES:
        toks = list(base)
        toks[edge] = k_tok
        asks = [p for p in (edge + 1, edge + 2, edge + 63, edge + 64, edge + 65, 200, 329) if edge < p < 330]
        for p in asks:
            toks[p] = q_tok
        want = P.logits(toks, cfg, w)
        lost = list(toks)
        lost[edge] = 11
        wrong = P.logits(lost, cfg, w)
        rows = np.array(asks)
        assert min(error(wrong[[r]], want[[r]]) for r in rows) > 5 * TOL[dtype], "the planted mistake must show"
        for sizes in ([330], [edge + 1, 64, 2, 1], [max(edge, 1), 1]):
            assert error(feed(m, toks, sizes)[rows], want[rows]) < TOL[dtype], (edge, sizes)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_across_prompt_chunks(tmp_path, dtype):
    """A prompt longer than one internal chunk (2048 tokens): a key at its start, at the chunk's edge, and queries beyond."""
    cfg = config([attention(heads=2, kv_heads=1, dim=32, rot=16, vdim=16, base=10000.0, scale=0.6, softcap=30.0), rglru(width=40, blocks=2),
                  mamba2(heads=2, vdim=16, state=16, groups=1)])
    q_tok, k_tok = 7, 9
    w = aim(cfg, P.random_weights(cfg, 43), q_tok, k_tok)
    base = [t if t not in (q_tok, k_tok) else 11 for t in tokens(2200, 101, 44)]
    m = load(tmp_path, cfg, w, dtype, 2200)
    for edge in (0, 2047, 2048):
        toks = list(base)
        toks[edge] = k_tok
        asks = [2049, 2111, 2112, 2199]
        for p in asks:
            toks[p] = q_tok
        want = P.logits(toks, cfg, w)[asks]
        m.truncate_kv(0)
        assert error(m.forward_prefill_logits_at(toks, 0, asks), want) < TOL[dtype]
        m.truncate_kv(0)
        m.forward_prefill(toks[:2198], 0, want_logits=False)
        m.forward(toks[2198], 2198)
        assert error(m.forward(toks[2199], 2199)[None], want[-1:]) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_soft_cap_bites(tmp_path, dtype):
    """Scores far above the cap, and far below it."""
    for k, (scale, cap) in enumerate(((2.0, 1.5), (0.3, 500.0))):
        cfg = config([attention(scale=scale, softcap=cap)])
        w = P.random_weights(cfg, 51)
        w["l0.mix.o"] *= 4.0
        toks = tokens(70, cfg["vocab"], 52)
        want = P.logits(toks, cfg, w)
        other = config([attention(scale=scale, softcap=20.0 if k else 1e6)])
        if k == 0:
            assert error(P.logits(toks, other, w), want) > 0.1
        m = load(tmp_path / str(k), cfg, w, dtype, 70)
        for sizes in ([70], [1]):
            assert error(feed(m, toks, sizes), want) < TOL[dtype]
        m.close()


@pytest.mark.parametrize("kind", ["rglru", "mamba2"])
def test_state_survives_a_long_memory(tmp_path, kind):
    """Decays next to 1: what the first tokens wrote is still there hundreds of tokens later."""
    cfg = config([rglru(width=96) if kind == "rglru" else mamba2(state=32)])
    w = P.random_weights(cfg, 61)
    if kind == "rglru":
        w["l0.mix.lam"][:] = -9.0
    else:
        w["l0.mix.A_log"][:] = -7.0
    w["l0.mix.o"] *= 4.0
    toks = tokens(600, cfg["vocab"], 62)
    want = P.logits(toks, cfg, w)
    other = [t + 1 if i < 40 and t < 100 else t for i, t in enumerate(toks)]
    assert error(P.logits(other, cfg, w)[-1:], want[-1:]) > 5e-3
    for dtype in DTYPES:
        m = load(tmp_path / dtype, cfg, w, dtype, 600)
        for sizes in ([600], [500, 1], [31, 33, 2]):
            assert error(feed(m, toks, sizes), want) < TOL[dtype]
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["rglru", "mamba2"])
def test_a_past_that_is_forgotten_at_once(tmp_path, kind, dtype):
    """Decays next to 0 (their logarithms sum to thousands over a portion), and the convolution's reach alone crosses a cut."""
    cfg = config([rglru(conv=4) if kind == "rglru" else mamba2(conv=4)])
    w = P.random_weights(cfg, 63)
    if kind == "rglru":
        w["l0.mix.lam"][:] = 9.0
    else:
        w["l0.mix.A_log"][:] = 4.0
    w["l0.mix.conv"] *= np.array([4.0, 2.0, 1.0, 0.5])
    toks = tokens(200, cfg["vocab"], 64)
    m = load(tmp_path, cfg, w, dtype, 200)
    want = P.logits(toks, cfg, w)
    for sizes in ([200], [2], [3, 1, 2, 5, 128, 1]):
        assert error(feed(m, toks, sizes), want) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_recurrent_state_far_outweighs_the_input(tmp_path, dtype):
    """Step sizes and decays that spread over orders of magnitude between the heads of one layer."""
    cfg = config([mamba2(heads=6, groups=2, state=40, norm_groups=6)])
    w = P.random_weights(cfg, 65)
    w["l0.mix.A_log"][:] = [-8.0, -4.0, -2.0, 0.0, 2.0, 3.0]
    w["l0.mix.dt_bias"][:] = [3.0, -4.0, 1.0, -6.0, 0.0, 2.0]
    toks = tokens(300, cfg["vocab"], 66)
    m = load(tmp_path, cfg, w, dtype, 300)
    want = P.logits(toks, cfg, w)
    for sizes in ([300], [64, 65, 1], [280, 1]):
        got = feed(m, toks, sizes)
        assert error(got, want, 0.95) < TOL[dtype]
        assert error(got, want) < 3 * TOL[dtype]
    m.close()


def test_greedy_generation(tmp_path):
    """generate_greedy (chained on the device), forward_greedy and the command line give the plain implementation's tokens."""
    cfg = mixed()
    w = P.random_weights(cfg, 81)
    prompt = tokens(30, cfg["vocab"], 82)
    want = P.greedy(prompt, 24, cfg, w)
    m = load(tmp_path, cfg, w, "float32", 128)
    first = int(np.argmax(m.forward_prefill(prompt, 0)))
    rest, _ = m.generate_greedy(first, 30, 23)
    assert [first] + [int(t) for t in rest] == want
    assert m.seq_len == 53
    after = m.forward(want[-1], 53)
    m.truncate_kv(0)
    tok = int(np.argmax(m.forward_prefill(prompt, 0)))
    got = [tok]
    for i in range(23):
        tok = m.forward_greedy(tok, 30 + i)
        got.append(tok)
    assert got == want
    np.testing.assert_array_equal(m.forward(tok, 53), after)
    m.close()
    r = subprocess.run([sys.executable, "-m", "cera_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--tokens", ",".join(map(str, prompt)),
                        "--n", "24"], capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()] == want


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(tmp_path, dtype):
    """400 chained steps; then the whole sequence as one prompt gives the same logits."""
    cfg = mixed()
    w = P.random_weights(cfg, 91)
    m = load(tmp_path, cfg, w, dtype, 512)
    toks = tokens(20, cfg["vocab"], 92)
    toks.append(int(np.argmax(m.forward_prefill(toks, 0))))
    out, _ = m.generate_greedy(toks[-1], 20, 400)
    toks += [int(t) for t in out]
    want = P.logits(toks, cfg, w)
    assert error(m.forward(toks[420], 420)[None], want[-1:]) < TOL[dtype]
    assert error(feed(m, toks, [421]), want) < TOL[dtype]
    m.close()


def test_errors_leave_the_model_usable(tmp_path):
    cfg = mixed()
    w = P.random_weights(cfg, 95)
    m = load(tmp_path, cfg, w, "float32", 32)
    from cera_b200 import CeraCudaError
    toks = tokens(20, cfg["vocab"], 96)
    with pytest.raises(CeraCudaError):
        m.forward(cfg["vocab"], 0)
    with pytest.raises(CeraCudaError):
        m.forward_prefill(toks * 2, 0)
    m.forward_prefill(toks, 0, want_logits=False)
    with pytest.raises(CeraCudaError):
        m.truncate_kv(5)  # a recurrent state cannot go back
    assert m.seq_len == 20
    assert error(m.forward(3, 20)[None], P.logits(toks + [3], cfg, w)[-1:]) < TOL["float32"]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_only_model_can_be_truncated(tmp_path, dtype):
    cfg = config([attention(mlp=unit())], loop={"start": 0, "stop": 1, "times": 2})
    w = P.random_weights(cfg, 97)
    m = load(tmp_path, cfg, w, dtype, 64)
    toks = tokens(40, cfg["vocab"], 98)
    m.forward_prefill(toks, 0, want_logits=False)
    m.truncate_kv(25)
    other = toks[:25] + tokens(5, cfg["vocab"], 99)
    got = m.forward_prefill_logits_at(other[25:], 25, [0, 4])
    assert error(got, P.logits(other, cfg, w)[[25, 29]]) < TOL[dtype]
    m.close()


def test_missing_and_misshapen_tensors_are_refused(tmp_path):
    cfg = mixed()
    w = P.random_weights(cfg, 99)
    need_gpu()
    from cera_b200 import CeraCudaError, load_model
    from cera_b200.safetensors import SafetensorsError
    bad = {k: v for k, v in w.items() if k != "l1.mix.lam"}
    P.save(tmp_path, cfg, bad)
    with pytest.raises(SafetensorsError, match="l1.mix.lam"):
        load_model(tmp_path, dtype="float32", max_seq_len=16)
    for name, shape in (("l0.mix.in", (5, 72)), ("l2.mix.k", (80, 71)), ("l1.mix.ra", (3, 30, 29)), ("l0.mix.conv", (4, 3)), ("final.norm", (71,))):
        P.save(tmp_path, cfg, {**w, name: np.zeros(shape)})
        with pytest.raises(CeraCudaError):
            load_model(tmp_path, dtype="float32", max_seq_len=16)


def test_layer_description_options(tmp_path):
    """Attention without biases, norm and soft cap, plain norms, an output matrix of its own: the mechanisms' parameters."""
    need_gpu()
    from cera_b200 import Role, piditar
    from cera_b200.layered import LayeredModel
    from cera_b200.types import BF16
    cfg = config([attention(mlp=unit())], scale=1.0)
    c = cfg["layers"][0]["mixer"]
    w = P.random_weights(cfg, 111)
    head = P.from_bf16(P.to_bf16(np.random.default_rng(112).standard_normal((101, 72)) / 8)).astype(np.float64)
    kw, layers = piditar.describe(cfg)
    kw.update(norm_offset=0.0, tied_output=0, embedding_scale=0.0)
    layers[0].attn_bias = layers[0].qk_norm = 0
    layers[0].softcap = 0.0
    toks = tokens(60, 101, 113)

    def plain(x, g):
        return P.rms_norm(x, g, 1e-5)
    x = w["embed"][toks]
    h = plain(x, w["l0.norm1"])
    q, k, v = (h @ w[f"l0.mix.{n}"].T for n in "qkv")
    turn = lambda a, n: np.stack([P.rotate_front(a[t].reshape(n, -1), t, c["rot"]["dims"], c["rot"]["base"]) for t in range(60)])  # noqa: E731
    q, k, v = turn(q, 6), turn(k, 2), v.reshape(60, 2, -1)
    out = np.zeros((60, 6, 24))
    for t in range(60):
        for i in range(6):
            e = np.exp(k[:t + 1, i // 3] @ q[t, i] * c["scale"])
            out[t, i] = e / e.sum() @ v[:t + 1, i // 3]
    x = x + out.reshape(60, -1) @ w["l0.mix.o"].T
    x = x + P.gated_ff(plain(x, w["l0.norm2"]), {n: w[f"l0.mlp.{n}"] for n in ("gate", "up", "down")})
    want = plain(x, w["final.norm"]) @ head.T
    for dtype in DTYPES:
        m = LayeredModel(layers, dtype=dtype, max_seq_len=60, **kw)
        for name, role, layer, _ in piditar.tensor_roles(layers) + [("head", Role.OUTPUT, 0, None)]:
            if name.endswith(".b"):
                continue
            t = head if name == "head" else w[name]
            rows, cols = t.shape if t.ndim == 2 else (1, t.size)
            m.add_tensor(role, layer, BF16, rows, cols, P.to_bf16(t).reshape(-1))
        m.finalize()
        for sizes in ([60], [20, 1]):
            assert error(feed(m, toks, sizes), want) < TOL[dtype]
        m.close()


def test_no_bounded_wait_ran_out():
    need_gpu()
    from cera_b200 import _lib
    assert _lib.kernel_status() == 0
