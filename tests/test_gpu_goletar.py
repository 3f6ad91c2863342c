"""Goletar on the GPU against the plain float64 implementation: mechanisms alone, cuts of a prompt, decoding, state reuse,
keys far away and at tile edges, greedy generation through the public entry points."""
import copy
import subprocess
import sys

import numpy as np
import pytest

import goletar_ref as G
from goletar_util import TOL, aim, attention, config, error, mingru, moe, tokens
from gpu_util import need_gpu

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]

MECHANISMS = {
    "attention": [attention()],
    "attention_one_head": [attention(heads=1, dim=16, rot_dim=2, vdim=16, kv_rank=64, base=50.0)],
    "attention_many_heads": [attention(heads=21, dim=40, rot_dim=24, vdim=72, kv_rank=200)],
    "attention_wide": [attention(heads=10, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=0.07)],
    "attention_wide_values": [attention(heads=2, dim=100, rot_dim=66, vdim=250, kv_rank=320, scale=0.07)],
    "attention_beyond_tiles": [attention(heads=2, dim=300, rot_dim=64, vdim=300, kv_rank=640, scale=0.05)],
    "mingru": [mingru()],
    "mingru_wide": [mingru(width=650)],
    "experts_all": [mingru(width=8, mlp=moe(experts=3, top=3, ff=24))],
    "experts_one": [mingru(width=8, mlp=moe(experts=1, top=1, ff=130, limit=0.5))],
    "experts_many": [mingru(width=8, mlp=moe(experts=40, top=6, ff=72, limit=4.0))],
}
MIXED = [mingru(mlp=moe()), attention(mlp=moe(experts=9, top=3, ff=56)), attention(heads=5, vdim=24, base=20.0), mingru(width=33, mlp=moe(top=1))]
# the same with every expert in use: no routing decision that 16-bit rounding could turn over
MIXED_ALL = [mingru(mlp=moe(experts=2, top=2)), attention(mlp=moe(experts=3, top=3, ff=56)), attention(heads=5, vdim=24, base=20.0),
             mingru(width=33, mlp=moe(experts=1, top=1))]


def mixed(dtype):
    return config(MIXED if dtype == "float32" else MIXED_ALL)


def load(tmp_path, cfg, w, dtype, max_seq_len):
    need_gpu()
    from cera_b200 import load_model
    tmp_path.mkdir(exist_ok=True)
    G.save(tmp_path, cfg, w)
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
    cfg = config(MECHANISMS[name], width=72 if "wide" not in name else 136)
    w = G.random_weights(cfg, 11)
    toks = tokens(150, cfg["vocab"], 12)
    want = G.logits(toks, cfg, w)
    m = load(tmp_path, cfg, w, dtype, 160)
    most = 0.8 if dtype == "bfloat16" and name == "experts_many" else 1.0
    for sizes in ([150], [40, 1], [1]):
        assert error(feed(m, toks, sizes), want, most) < TOL[dtype], sizes
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[2], [3, 2, 15, 16, 17, 1, 64, 63, 2], [100, 2, 7], [129, 128, 1, 1]])
def test_portions_of_a_prompt(tmp_path, dtype, sizes):
    cfg = mixed(dtype)
    w = G.random_weights(cfg, 21)
    toks = tokens(330, cfg["vocab"], 22)
    m = load(tmp_path, cfg, w, dtype, 330)
    assert error(feed(m, toks, sizes), G.logits(toks, cfg, w)) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("width,vocab,eps", [(64, 40, 1e-6), (65, 1000, 1e-3), (250, 77, 1e-2)])
def test_other_sizes(tmp_path, width, vocab, eps):
    cfg = config([mingru(width=width + 1, mlp=moe(ff=65, experts=2, top=2)), attention(heads=4, dim=8, rot_dim=6, vdim=9, kv_rank=70)], width=width, vocab=vocab, eps=eps,
                 buckets=1 + vocab // 2, mul_prev=2_000_000_011, mul_cur=4_000_000_007)
    w = G.random_weights(cfg, 23)
    w["l0.norm1"], w["l1.norm1b"] = np.float64(-0.5), np.float64(2.0)
    toks = tokens(90, vocab, 24)
    want = G.logits(toks, cfg, w)
    for dtype in DTYPES:
        m = load(tmp_path / dtype, cfg, w, dtype, 90)
        assert error(feed(m, toks, [60, 5, 1]), want) < TOL[dtype]
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sequence_does_not_see_the_one_before(tmp_path, dtype):
    cfg = mixed(dtype)
    w = G.random_weights(cfg, 31)
    m = load(tmp_path, cfg, w, dtype, 256)
    for n, seed in ((256, 1), (3, 2), (1, 3), (100, 4), (17, 5), (256, 6)):
        toks = tokens(n, cfg["vocab"], seed)
        assert error(feed(m, toks, [max(n - 4, 1), 1]), G.logits(toks, cfg, w)) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_snapshots_interleave_sequences(tmp_path, dtype):
    cfg = mixed(dtype)
    w = G.random_weights(cfg, 32)
    m = load(tmp_path, cfg, w, dtype, 96)
    seqs = [tokens(n, cfg["vocab"], 40 + n) for n in (70, 33, 96)]
    want = [G.logits(t, cfg, w) for t in seqs]
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
    cfg = config([attention(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, base=10000.0)], vocab=101)
    q_tok, k_tok = 7, 9
    w = aim(cfg, G.random_weights(cfg, 41), 0, q_tok, k_tok, 14.0)
    m = load(tmp_path, cfg, w, dtype, 340)
    base = [t if t not in (q_tok, k_tok) else 11 for t in tokens(330, 101, 42)]
    for edge in EDGES:
        toks = list(base)
        toks[edge] = k_tok
        asks = [p for p in (edge + 1, edge + 2, edge + 63, edge + 64, edge + 65, 200, 329) if edge < p < 330]
        for p in asks:
            toks[p] = q_tok
        want = G.logits(toks, cfg, w)
        lost = list(toks)
        lost[edge] = 11
        wrong = G.logits(lost, cfg, w)
        rows = np.array(asks)
        assert min(error(wrong[[r]], want[[r]]) for r in rows) > 5 * TOL[dtype], "the planted mistake must show"
        for sizes in ([330], [edge + 1, 64, 2, 1], [max(edge, 1), 1]):
            assert error(feed(m, toks, sizes)[rows], want[rows]) < TOL[dtype], (edge, sizes)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_across_prompt_chunks(tmp_path, dtype):
    """A prompt longer than one internal chunk (2048 tokens): a key at its start, at the chunk's edge, and queries beyond."""
    cfg = config([attention(heads=2, dim=32, rot_dim=16, vdim=16, kv_rank=64, base=10000.0), mingru(width=40)], vocab=101)
    q_tok, k_tok = 7, 9
    w = aim(cfg, G.random_weights(cfg, 43), 0, q_tok, k_tok, 14.0)
    base = [t if t not in (q_tok, k_tok) else 11 for t in tokens(2200, 101, 44)]
    m = load(tmp_path, cfg, w, dtype, 2200)
    for edge in (0, 2047, 2048):
        toks = list(base)
        toks[edge] = k_tok
        asks = [2049, 2111, 2112, 2199]
        for p in asks:
            toks[p] = q_tok
        want = G.logits(toks, cfg, w)[asks]
        m.truncate_kv(0)
        assert error(m.forward_prefill_logits_at(toks, 0, asks), want) < TOL[dtype]
        m.truncate_kv(0)
        m.forward_prefill(toks[:2198], 0, want_logits=False)
        m.forward(toks[2198], 2198)
        assert error(m.forward(toks[2199], 2199)[None], want[-1:]) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_weighs_in(tmp_path, dtype):
    """Heavy, absent-like and very heavy sinks, from the first token on."""
    cfg = config([attention(heads=3)])
    w = G.random_weights(cfg, 51)
    toks = tokens(70, cfg["vocab"], 52)
    for k, sink in enumerate(([4.0, -30.0, 0.5], [9.0, 3.0, -1.0], [60.0, -60.0, 2.0])):
        w["l0.mix.sink"] = np.array(sink)
        want = G.logits(toks, cfg, w)
        m = load(tmp_path / str(k), cfg, w, dtype, 70)
        assert error(feed(m, toks, [70]), want) < TOL[dtype]
        assert error(feed(m, toks, [1]), want) < TOL[dtype]
        m.close()
    w["l0.mix.sink"] = np.array([-60.0] * 3)
    assert error(G.logits(toks, cfg, w), want) > 5 * TOL[dtype]


def test_state_survives_a_long_memory(tmp_path):
    """minGRU with nearly closed gates: what the first tokens wrote is still there hundreds of tokens later."""
    cfg = config([mingru(width=96)])
    w = G.random_weights(cfg, 61)
    w["l0.mix.z.b"][:] = -7.0
    toks = tokens(600, cfg["vocab"], 62)
    want = G.logits(toks, cfg, w)
    other = [t + 1 if i < 40 and t < 100 else t for i, t in enumerate(toks)]
    assert error(G.logits(other, cfg, w)[-1:], want[-1:]) > 5e-3
    m = load(tmp_path, cfg, w, "float32", 600)
    for sizes in ([600], [500, 1], [31, 33, 2]):
        assert error(feed(m, toks, sizes), want) < 1e-4
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_uneven_experts(tmp_path, dtype):
    """Every token of a long portion goes to the same few experts; others get none or a handful."""
    cfg = config([mingru(width=40, mlp=moe(experts=12, top=2, ff=48))])
    w = G.random_weights(cfg, 71)
    toks = [5] * 300 + tokens(8, cfg["vocab"], 72) + [5] * 100
    m = load(tmp_path, cfg, w, dtype, 408)
    assert error(feed(m, toks, [408]), G.logits(toks, cfg, w)) < TOL[dtype]
    m.close()


def test_clamps_bite(tmp_path):
    cfg = config([mingru(width=40, mlp=moe(experts=4, top=2, ff=48, limit=0.2))])
    w = G.random_weights(cfg, 73)
    toks = tokens(40, cfg["vocab"], 74)
    loose = copy.deepcopy(cfg)
    loose["layers"][0]["mlp"]["expert"]["limit"] = 50.0
    want = G.logits(toks, cfg, w)
    assert error(G.logits(toks, loose, w), want) > 0.1
    m = load(tmp_path, cfg, w, "float32", 40)
    assert error(feed(m, toks, [30, 1]), want) < TOL["float32"]
    m.close()


def test_greedy_generation(tmp_path):
    """generate_greedy (chained on the device), forward_greedy and the command line give the plain implementation's tokens."""
    cfg = config(MIXED)
    w = G.random_weights(cfg, 81)
    w["head"] *= 4.0
    prompt = tokens(30, cfg["vocab"], 82)
    want = G.greedy(prompt, 24, cfg, w)
    m = load(tmp_path, cfg, w, "float32", 128)
    first = int(np.argmax(m.forward_prefill(prompt, 0)))
    rest, _ = m.generate_greedy(first, 30, 23)
    assert [first] + [int(t) for t in rest] == want
    assert m.seq_len == 53
    # the state a chained run leaves (the previous token included) is the one single steps leave
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
    cfg = mixed(dtype)
    w = G.random_weights(cfg, 91)
    m = load(tmp_path, cfg, w, dtype, 512)
    toks = tokens(20, cfg["vocab"], 92)
    toks.append(int(np.argmax(m.forward_prefill(toks, 0))))
    out, _ = m.generate_greedy(toks[-1], 20, 400)
    toks += [int(t) for t in out]
    want = G.logits(toks, cfg, w)
    assert error(m.forward(toks[420], 420)[None], want[-1:]) < TOL[dtype]
    assert error(feed(m, toks, [421]), want) < TOL[dtype]
    m.close()


def test_errors_leave_the_model_usable(tmp_path):
    cfg = config(MIXED)
    w = G.random_weights(cfg, 95)
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
    with pytest.raises(CeraCudaError):
        m.shift_kv(0, 1)
    assert m.seq_len == 20
    assert error(m.forward(3, 20)[None], G.logits(toks + [3], cfg, w)[-1:]) < TOL["float32"]
    m.close()


def test_attention_only_model_can_be_truncated(tmp_path):
    cfg = config([attention(mlp=moe())])
    w = G.random_weights(cfg, 97)
    m = load(tmp_path, cfg, w, "float32", 64)
    toks = tokens(40, cfg["vocab"], 98)
    m.forward_prefill(toks, 0, want_logits=False)
    m.truncate_kv(25)
    got = m.forward_prefill_logits_at(toks[25:30], 25, [0, 4])
    assert error(got, G.logits(toks[:30], cfg, w)[[25, 29]]) < TOL["float32"]
    m.close()


def test_missing_tensor_is_named(tmp_path):
    cfg = config(MIXED)
    w = G.random_weights(cfg, 99)
    del w["l1.mix.sink"]
    need_gpu()
    from cera_b200 import load_model
    from cera_b200.safetensors import SafetensorsError
    G.save(tmp_path, cfg, w)
    with pytest.raises(SafetensorsError, match="l1.mix.sink"):
        load_model(tmp_path, dtype="float32", max_seq_len=16)


def test_no_bounded_wait_ran_out():
    need_gpu()
    from cera_b200 import _lib
    assert _lib.kernel_status() == 0


def moe_by_rule(h, w, c, softmax, renorm, weight_input):
    """The plain routed feed-forward under the other rules a layer description can name."""
    z = h @ w["router"].T
    s = np.exp(z - z.max(-1, keepdims=True)) if softmax else G.sigmoid(z)
    if softmax:
        s /= s.sum(-1, keepdims=True)
    out = np.zeros_like(h)
    for t in range(len(h)):
        ids = np.argsort(-s[t], kind="stable")[:c["router"]["top"]]
        wt = s[t][ids] / (s[t][ids].sum() if renorm else 1.0)
        for e, x in zip(ids, wt):
            m = (w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], c["expert"]["limit"])
            out[t] += G.clamped_glu(x * h[t], *m) if weight_input else x * G.clamped_glu(h[t], *m)
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rule", [(1, 0, 1), (0, 1, 0), (1, 1, 0)])
def test_other_rules_of_a_layer_description(monkeypatch, dtype, rule):
    """Softmax scores, renormalised weights, weights on the output, per-channel norms: the mechanisms' parameters, not this design's."""
    need_gpu()
    from cera_b200 import goletar
    from cera_b200.layered import LayeredModel
    from cera_b200.types import BF16
    softmax, renorm, weight_input = rule
    cfg = config([attention(mlp=moe(experts=3, top=3)), mingru(mlp=moe(experts=4, top=4, ff=72))])
    w = G.random_weights(cfg, 111)
    rng = np.random.default_rng(112)
    for name in ("l0.norm1", "l0.norm1b", "l1.norm2", "l1.norm2b", "final.norm"):
        w[name] = G.from_bf16(G.to_bf16(1.0 + 0.3 * rng.standard_normal(72))).astype(np.float64)
    kw, layers = goletar.describe(cfg)
    for d in layers:
        d.router_softmax, d.router_renorm, d.weight_input = softmax, renorm, weight_input
    m = LayeredModel(layers, dtype=dtype, max_seq_len=120, **kw)
    for name, role, layer, expert in goletar.tensor_roles(layers):
        v = w[name]
        rows, cols = v.shape if v.ndim == 2 else (1, v.size)
        m.add_tensor(role, layer, BF16, rows, cols, G.to_bf16(v).reshape(-1), expert=expert)
    m.finalize()
    monkeypatch.setattr(G, "moe", lambda h, ww, c: moe_by_rule(h, ww, c, *rule))
    toks = tokens(110, cfg["vocab"], 113)
    want = G.logits(toks, cfg, w)
    for sizes in ([110], [50, 1]):
        assert error(feed(m, toks, sizes), want) < TOL[dtype], sizes
    m.close()
