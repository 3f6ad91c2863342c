"""Piditar without a GPU: the configuration and tensor names, the loader's view of stacked tensors, and the plain
implementation's own consistency."""
import math

import numpy as np
import pytest

import piditar_ref as P
from piditar_util import aim, attention, config, error, mamba2, rglru, tokens, unit
from cera_b200 import piditar, registry
from cera_b200.layered import Ff, Mixer
from cera_b200.safetensors import SafetensorsFile


def small(**kw):
    return config([attention(mlp=unit()), rglru(), mamba2(mlp=unit(ff=33))], **kw)


def test_describe_reads_every_size_from_the_config():
    kw, (a, b, c) = piditar.describe(small(loop={"start": 1, "stop": 3, "times": 4}))
    assert kw == dict(hidden_size=72, vocab_size=101, norm_eps=1e-5, embedding_scale=1.5, norm_offset=1.0, tied_output=1, no_post_norms=1,
                      loop_start=1, loop_stop=3, loop_times=4)
    assert (a.mixer, a.n_heads, a.n_kv_heads, a.head_dim, a.value_dim, a.rot_dim) == (Mixer.ATTENTION, 6, 2, 40, 24, 16)
    assert (a.rope_base, round(a.attn_scale, 6), a.softcap, a.qk_norm, a.attn_bias) == (1000.0, 0.2, 6.0, 1, 1)
    assert (a.ff, a.ff_width, a.act_limit, a.act_alpha, a.act_shift) == (Ff.GATED, 56, math.inf, 1.0, 0.0)
    assert (b.mixer, b.recurrent_width, b.n_blocks, b.conv_taps, b.decay, b.ff) == (Mixer.RGLRU, 90, 3, 3, 8.0, Ff.NONE)
    assert (c.mixer, c.n_heads, c.value_dim, c.state_size, c.n_groups, c.n_norm_groups, c.conv_taps) == (Mixer.SSM, 4, 24, 20, 2, 1, 4)
    assert c.ff_width == 33


def test_a_config_without_a_loop_runs_every_layer_once():
    cfg = small()
    del cfg["loop"]
    assert piditar.describe(cfg)[0]["loop_times"] == 1
    assert P.passes(cfg) == [(0, False), (1, False), (2, False)]


def test_passes_of_a_loop():
    assert P.passes(small(loop={"start": 1, "stop": 2, "times": 3})) == [(0, False), (1, False), (1, True), (1, True), (2, False)]
    assert P.passes(small(loop={"start": 0, "stop": 3, "times": 2})) == [(i, again) for again in (False, True) for i, again in
                                                                         ((0, again), (1, False), (2, False))]


def test_tensor_names_are_those_of_the_design():
    cfg = small()
    _, layers = piditar.describe(cfg)
    assert sorted(n for n, *_ in piditar.tensor_roles(layers)) == sorted(P.tensor_shapes(cfg))


@pytest.mark.parametrize("change", [lambda c: c["layers"][0].update(type="conv"), lambda c: c["layers"][0]["mlp"].update(kind="moe")])
def test_describe_refuses_what_it_does_not_know(change):
    cfg = small()
    change(cfg)
    with pytest.raises(ValueError):
        piditar.describe(cfg)


def test_registry_knows_the_design():
    assert "Piditar" in registry.FOLDER_ARCHITECTURES


def test_stacked_tensors_come_as_one_tall_matrix(tmp_path):
    cfg = small()
    w = P.random_weights(cfg, 3)
    P.save(tmp_path, cfg, w)
    with SafetensorsFile(tmp_path / "model.safetensors") as f:
        rows, cols, _, data = f.get("l1.mix.ra")
        assert (rows, cols) == (90, 30)
        np.testing.assert_array_equal(P.from_bf16(data.view(np.uint16)).reshape(3, 30, 30), w["l1.mix.ra"])
        assert f.get("l1.mix.ra.b")[:2] == (3, 30) and f.get("l2.mix.D")[:2] == (1, 4)
        del data


# ---- the plain implementation ---------------------------------------------------------------------------------------

def test_rotation_turns_the_front_only_and_keeps_relative_positions():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal(10), rng.standard_normal(10)
    a = P.rotate_front(q, 9, 6, 100.0) @ P.rotate_front(k, 4, 6, 100.0)
    assert a == pytest.approx(P.rotate_front(q, 105, 6, 100.0) @ P.rotate_front(k, 100, 6, 100.0))
    np.testing.assert_array_equal(P.rotate_front(q, 7, 6, 100.0)[6:], q[6:])


def test_convolution_meets_the_current_position_with_its_last_tap():
    x = np.arange(1.0, 6.0)[:, None]
    np.testing.assert_allclose(P.causal_conv(x, np.array([[0.0, 0.0, 1.0]]), np.zeros(1)), x)
    np.testing.assert_allclose(P.causal_conv(x, np.array([[1.0, 0.0, 0.0]]), np.zeros(1))[:, 0], [0, 0, 1, 2, 3])
    np.testing.assert_allclose(P.causal_conv(x, np.array([[10.0, 100.0]]), np.ones(1))[:, 0], [101, 211, 321, 431, 541])


def test_recurrences_carry_over_a_cut():
    """With one tap nothing but the state crosses a cut."""
    rng = np.random.default_rng(2)
    h = rng.standard_normal((9, 72))
    cfg = config([rglru(conv=1), mamba2(conv=1)])
    w = P.random_weights(cfg, 1)
    lru = {k[7:]: v for k, v in w.items() if k.startswith("l0.mix.")}
    ssm = {k[7:]: v for k, v in w.items() if k.startswith("l1.mix.")}
    for run in (lambda x, s=None: P.rglru(x, lru, cfg["layers"][0]["mixer"], s), lambda x, s=None: P.mamba2(x, ssm, cfg["layers"][1]["mixer"], 1e-5, s)):
        whole, s = run(h)
        a, s1 = run(h[:4])
        b, s2 = run(h[4:], s1)
        np.testing.assert_allclose(np.concatenate([a, b]), whole)
        np.testing.assert_allclose(s2, s)


def test_state_space_form_equals_its_unrolled_sum():
    """y_t = sum over j <= t of (C_t . B_j) exp(sum of log decays after j) dt_j x_j + D x_t, one head alone."""
    cfg = config([mamba2(heads=1, groups=1, vdim=3, state=5, conv=1)])
    m = cfg["layers"][0]["mixer"]
    w = {k[7:]: v for k, v in P.random_weights(cfg, 4).items() if k.startswith("l0.mix.")}
    w["o"] = np.eye(3)
    h = np.random.default_rng(5).standard_normal((6, 72))
    p = h @ w["in"].T
    z, xbc, dt = p[:, :3], P.silu(p[:, 3:16] * w["conv"][:, 0] + w["conv.b"]), P.softplus(p[:, 16] + w["dt_bias"])
    x, b, c = xbc[:, :3], xbc[:, 3:8], xbc[:, 8:]
    la = -np.exp(w["A_log"]) * dt
    y = np.stack([sum((c[t] @ b[j]) * np.exp(la[j + 1:t + 1].sum()) * dt[j] * x[j] for j in range(t + 1)) + w["D"] * x[t] for t in range(6)])
    np.testing.assert_allclose(P.mamba2(h, w, m, 1e-5)[0], P.rms_norm(y * P.silu(z), w["norm"], 1e-5))


def test_causality():
    cfg = small(loop={"start": 0, "stop": 2, "times": 2})
    w = P.random_weights(cfg, 4)
    t = tokens(12, 101, 5)
    np.testing.assert_allclose(P.logits(t[:7], cfg, w), P.logits(t, cfg, w)[:7], atol=1e-10)


def test_every_pass_and_branch_shows_in_the_logits():
    cfg = small(loop={"start": 0, "stop": 2, "times": 2})
    w = P.random_weights(cfg, 6)
    t = tokens(40, 101, 7)
    want = P.logits(t, cfg, w)

    def differs(**kw):
        other = {**cfg, **kw}
        return error(P.logits(t, other, w), want, 0.5) > 0.05
    assert differs(loop={"start": 0, "stop": 2, "times": 1}) and differs(loop={"start": 1, "stop": 2, "times": 2}) and differs(embedding={"scale": 0.7})
    for name in w:  # every tensor
        v = dict(w)
        v[name] = w[name] + 0.5 * np.abs(w[name]).max()
        assert error(P.logits(t, cfg, v), want) > 0.02, name


def test_aimed_key_stands_out():
    cfg = config([attention(scale=0.6, softcap=30.0)])
    w = aim(cfg, P.random_weights(cfg, 8), 7, 9)
    t = [x if x not in (7, 9) else 11 for x in tokens(60, 101, 9)]
    t[3], t[59] = 9, 7
    lost = list(t)
    lost[3] = 11
    assert error(P.logits(lost, cfg, w)[-1:], P.logits(t, cfg, w)[-1:]) > 0.1
