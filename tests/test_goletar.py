"""Goletar without a GPU: the configuration and tensor names, the safetensors reader, the registry, and the plain
implementation's own consistency."""
import json
import struct

import numpy as np
import pytest

import goletar_ref as G
from goletar_util import attention, config, mingru, moe, tokens
from cera_b200 import goletar, registry, trace
from cera_b200.layered import Ff, Mixer
from cera_b200.safetensors import SafetensorsError, SafetensorsFile
from cera_b200.types import BF16


def small():
    return config([attention(mlp=moe()), mingru(), mingru(width=36, mlp=moe(experts=3, top=1, limit=0.75))])


def test_describe_reads_every_size_from_the_config():
    kw, layers = goletar.describe(small())
    assert kw == dict(hidden_size=72, vocab_size=101, norm_eps=1e-5, bigram_buckets=53, bigram_mul_prev=31, bigram_mul_cur=17)
    a, b, c = layers
    assert (a.mixer, a.n_heads, a.head_dim, a.rot_dim, a.value_dim, a.kv_rank) == (Mixer.LATENT_ATTENTION, 3, 24, 8, 40, 48)
    assert (a.rope_base, round(a.attn_scale, 6)) == (1000.0, 0.2)
    assert (a.ff, a.ff_width, a.n_experts, a.n_used, a.act_limit) == (Ff.MOE, 40, 5, 2, 1.5)
    assert round(a.act_alpha, 6) == 1.702 and a.act_shift == 1.0 and (a.router_softmax, a.router_renorm, a.weight_input) == (0, 0, 1)
    assert (b.mixer, b.recurrent_width, b.ff) == (Mixer.MINGRU, 100, Ff.NONE)
    assert (c.recurrent_width, c.n_experts, c.n_used, c.act_limit) == (36, 3, 1, 0.75)


def test_tensor_names_are_those_of_the_design():
    cfg = small()
    _, layers = goletar.describe(cfg)
    assert sorted(n for n, *_ in goletar.tensor_roles(layers)) == sorted(G.tensor_shapes(cfg))


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="conv"), lambda c: c["layers"][0]["mlp"].update(kind="dense"),
                                    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4)])
def test_describe_refuses_what_it_does_not_know(change):
    cfg = small()
    change(cfg)
    with pytest.raises(ValueError):
        goletar.describe(cfg)


def test_safetensors_round_trip(tmp_path):
    cfg = small()
    w = G.random_weights(cfg, 3)
    G.save(tmp_path, cfg, w)
    with SafetensorsFile(tmp_path / "model.safetensors") as f:
        for name, v in w.items():
            rows, cols, kind, data = f.get(name)
            assert kind == BF16 and rows * cols == v.size
            np.testing.assert_array_equal(G.from_bf16(data.view(np.uint16)).reshape(v.shape), v)
        assert not f.has("nothing")
        with pytest.raises(SafetensorsError):
            f.get("nothing")
        del data


def test_safetensors_refuses_bad_offsets(tmp_path):
    head = json.dumps({"a": {"dtype": "F32", "shape": [4], "data_offsets": [0, 16]}}).encode()
    p = tmp_path / "x.safetensors"
    p.write_bytes(struct.pack("<Q", len(head)) + head + b"\0" * 8)
    with pytest.raises(SafetensorsError):
        SafetensorsFile(p)


def test_registry_refuses_an_unknown_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nobody"}))
    with pytest.raises(ValueError, match="Nobody"):
        registry.load_model(tmp_path)


class FakeModel:
    """Counts what a trace asks of a model."""

    class cfg:
        vocab_size = 7

    def __init__(self):
        self.seq_len, self.log = 0, []

    def truncate_kv(self, n):
        self.seq_len = n

    def forward_prefill_logits_at(self, toks, start, want):
        assert start == self.seq_len
        self.seq_len += len(toks)
        self.log.append((list(toks), start, list(want)))
        return np.full((len(want), 7), start, dtype=np.float32)


def test_trace_runner_keeps_one_sequence():
    m = FakeModel()
    r = trace.TraceRunner(m)
    assert r.step([{"id": "a", "tokens": [1, 2, 3], "want": [0, 2]}]).shape == (2, 7)
    assert r.step([{"id": "a", "tokens": [4], "want": []}]).shape == (0, 7)
    with pytest.raises(RuntimeError):
        r.step([{"id": "b", "tokens": [4], "want": []}])
    r.end(["a"])
    assert m.seq_len == 0
    r.step([{"id": "b", "tokens": [5], "want": [0]}])
    assert m.log[-1] == ([5], 0, [0])


# ---- the plain implementation ---------------------------------------------------------------------------------------

def test_rotation_keeps_relative_positions():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal(8), rng.standard_normal(8)
    a = G.rotate(q, 9, 100.0) @ G.rotate(k, 4, 100.0)
    assert a == pytest.approx(G.rotate(q, 105, 100.0) @ G.rotate(k, 100, 100.0))
    np.testing.assert_array_equal(G.rotate(q, 0, 100.0), q)


def test_sink_takes_weight_and_counts_once():
    p = G.sink_softmax(np.array([0.0, 0.0]), 0.0)
    np.testing.assert_allclose(p, [1 / 3, 1 / 3])
    np.testing.assert_allclose(G.sink_softmax(np.array([1000.0]), -5.0), [1.0])


def test_mingru_state_carries_over_a_cut():
    cfg = config([mingru()])
    w = {k[7:]: v for k, v in G.random_weights(cfg, 1).items() if k.startswith("l0.mix.")}
    h = np.random.default_rng(2).standard_normal((9, 72))
    whole, s = G.mingru(h, w)
    a, s1 = G.mingru(h[:4], w)
    b, s2 = G.mingru(h[4:], w, s1)
    np.testing.assert_allclose(np.concatenate([a, b]), whole)
    np.testing.assert_allclose(s2, s)


def test_expert_weight_scales_the_input():
    rng = np.random.default_rng(3)
    gate, up, down, h = rng.standard_normal((6, 4)), rng.standard_normal((6, 4)), rng.standard_normal((4, 6)), rng.standard_normal(4)
    a = G.clamped_glu(0.5 * h, gate, up, down, 2.0)
    b = 0.5 * G.clamped_glu(h, gate, up, down, 2.0)
    assert np.abs(a - b).max() > 1e-3


def test_causality_and_first_token():
    cfg = small()
    w = G.random_weights(cfg, 4)
    t = tokens(12, 101, 5)
    np.testing.assert_allclose(G.logits(t[:7], cfg, w), G.logits(t, cfg, w)[:7], atol=1e-10)
    x = G.embed(t, w["embed"], w["bigram"], 53, 31, 17)
    np.testing.assert_array_equal(x[0], w["embed"][t[0]] + w["bigram"][53])
    np.testing.assert_array_equal(x[1], w["embed"][t[1]] + w["bigram"][(t[0] * 31 + t[1] * 17) % 53])
