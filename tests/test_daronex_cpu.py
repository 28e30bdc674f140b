"""Host side of Daronex: configuration, the fused and padded matrices -- and the oracle checked against
other ways to compute the same thing."""
import json

import numpy as np
import pytest

import dar_cases as dc
from cpp_tensorlib_b200 import daronex, registry, stack
from oracle import daronex as orc


def test_registry_knows_it():
    assert registry.model_class(dict(architecture="Daronex")) is daronex.Daronex


def test_layer_spec_reads_every_constant():
    m, = daronex.layer_spec(dc.full(6, 24, 10, 40, 33, 52, 123.0, 0.3, 48, kv_from=4))["mixers"]
    assert (m.kind, m.heads, m.dim, m.vdim, m.q_rank, m.kv_rank, m.rot_dims, m.window, m.gate, m.kv_from) == \
        (stack.LATENT, 6, 24, 40, 33, 52, 10, 0, 0, 4)
    assert np.allclose([m.rot_base, m.scale, m.out_scale], [123.0, 0.3, 1.0])
    s = daronex.layer_spec(dc.win(9, 6, 24, 10, 40, 33, 52, 77.0, 0.2, 48))
    m, = s["mixers"]
    assert (m.window, m.gate, m.kv_from, s["ff"], s["act"]) == (9, 1, -1, 48, stack.SQUARED_RELU)
    assert np.allclose([m.rot_base, m.scale], [77.0, 0.2])
    s = daronex.layer_spec(dc.gla(6, 10, 14, 2.5, 0), 12)
    m, = s["mixers"]
    assert (m.kind, m.heads, m.dim, m.vdim, m.rank, s["ff"]) == (stack.GLA, 6, 10, 14, 12, 0) and np.isclose(m.tau, 2.5)
    with pytest.raises(ValueError):
        daronex.layer_spec(dict(type="other", mixer={}))
    with pytest.raises(ValueError):
        daronex.layer_spec(dict(dc.full(), mlp=dict(kind="other")))


def loaded(cfg, w, monkeypatch):
    got = {}
    z = daronex.Daronex.__new__(daronex.Daronex)
    z.config, z.f32 = cfg, True
    monkeypatch.setattr(z, "set_matrix", lambda l, n, a, mixer=0: got.__setitem__((l, n), np.array(z.weight(a))), raising=False)
    monkeypatch.setattr(z, "set_vector", lambda l, n, v, mixer=0: got.__setitem__((l, n), np.array(v)), raising=False)
    z.load(w)
    return got


def test_matrices_keep_every_row(monkeypatch):
    """Every part of the fused and padded matrices lies where the native side reads it."""
    cfg = dc.CONFIGS["odd"]
    w = dc.Weights(cfg, 1)
    got = loaded(cfg, w, monkeypatch)
    p8 = stack.pad8
    m, p = cfg["layers"][1]["mixer"], "l1.mix."        # the windowed kind: rotate-half rows become pairs
    H, D, R, E, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    order = [x for i in range(R // 2) for x in (i, i + R // 2)]
    at = 0
    dkv = w.f32(p + "dkv")
    for t in (w.f32(p + "dq"), dkv[:C], dkv[C:][order], w.f32(p + "g")):
        assert np.array_equal(got[1, "input"][at:at + len(t)], t)
        assert not got[1, "input"][at + len(t):at + p8(len(t))].any()
        at += p8(len(t))
    assert at == len(got[1, "input"])
    uq = w.f32(p + "uq").reshape(H, D + R, -1)
    q = got[1, "q_up"].reshape(H, p8(D) + p8(R), -1)
    assert np.array_equal(q[:, :D], uq[:, :D]) and np.array_equal(q[:, p8(D):p8(D) + R], uq[:, D:][:, order])
    assert not q[:, D:p8(D)].any() and not q[:, p8(D) + R:].any()
    k, v = got[1, "kv_up"][:H * p8(D)].reshape(H, p8(D), -1), got[1, "kv_up"][H * p8(D):].reshape(H, p8(E), -1)
    assert np.array_equal(k[:, :D].reshape(H * D, -1), w.f32(p + "uk")) and not k[:, D:].any()
    assert np.array_equal(v[:, :E].reshape(H * E, -1), w.f32(p + "uv")) and not v[:, E:].any()
    # a layer that reads another one's latent projects none; norms around zero; the decay's weights
    assert len(got[4, "input"]) == p8(cfg["layers"][4]["mixer"]["q_rank"]) and (4, "k_norm") not in got
    assert np.allclose(got[2, "norm1"], 1 + w.f32("l2.norm1")) and np.array_equal(got[2, "q_norm"], w.f32("l2.mix.dq.norm"))
    assert np.array_equal(got[0, "decay_up"], w.f32("l0.mix.a2").T)
    assert np.array_equal(got[0, "norm"].reshape(3, -1)[2], w.f32("l0.mix.norm"))
    assert np.array_equal(got[0, "head"], w.f32("head")) and np.array_equal(got[0, "gate_up"], w.f32("l0.mlp.up"))
    assert (1, "gate_up") not in got and (1, "norm2") not in got


def test_paired_rows_turn_one_rotation_into_the_other():
    rng = np.random.default_rng(0)
    x, pos = rng.standard_normal((9, 1, 10)), np.arange(9)
    pair = lambda a: stack.paired_rows(a.reshape(9, 10, 1)).reshape(9, 1, 10)
    assert np.allclose(pair(orc.rotate(x, pos, 50.0, True)), orc.rotate(pair(x), pos, 50.0, False))


# ---- the oracle against other ways ----------------------------------------------------------------
def test_oracle_window_rule():
    for i in range(30):
        for j in range(30):
            assert orc.sees(i, j, 5) == (j <= i and j >= i - 4) and orc.sees(i, j, None) == (j <= i)


def test_oracle_attention_is_masked_softmax():
    rng = np.random.default_rng(0)
    q, k, v = (rng.standard_normal((17, 3, n)) for n in (6, 6, 5))
    for window in (None, 5):
        mask = np.array([[orc.sees(i, j, window) for j in range(17)] for i in range(17)])
        got = orc.attend(q, k, v, 0.7, window)
        for h in range(3):
            s = np.where(mask, q[:, h] @ k[:, h].T * 0.7, -np.inf)
            p = np.exp(s - s.max(1, keepdims=True))
            assert np.allclose(got[:, h], p / p.sum(1, keepdims=True) @ v[:, h])


@pytest.mark.parametrize("half", [False, True])
def test_oracle_rotation_keeps_distance(half):
    x = np.random.default_rng(1).standard_normal((2, 1, 8))
    a = orc.rotate(x, np.array([3, 10]), 100.0, half)
    b = orc.rotate(x, np.array([53, 60]), 100.0, half)
    assert np.allclose(a[0, 0] @ a[1, 0], b[0, 0] @ b[1, 0])
    assert not np.allclose(a, orc.rotate(x, np.array([3, 10]), 100.0, not half))


def test_oracle_gated_linear_is_a_decayed_sum():
    rng = np.random.default_rng(2)
    q, k, v = (rng.standard_normal((9, 2, n)) for n in (5, 5, 3))
    al = rng.random((9, 2, 5))
    got = orc.gated_linear(q, k, v, al)
    for t in range(9):
        for h in range(2):
            y = sum((q[t, h] * k[s, h] * np.prod(al[s + 1:t + 1, h], axis=0)).sum() * v[s, h] for s in range(t + 1))
            assert np.allclose(got[t, h], y)


def test_oracle_decay():
    z = np.linspace(-30, 30, 25)
    assert np.allclose(orc.decay(z, 4.0), orc.sigmoid(z) ** 0.25, rtol=1e-12)


@pytest.mark.parametrize("change,place", [(+1, "outside"), (-1, "inside")])
def test_planted_keys_show_a_shifted_edge(change, place):
    """The planted queries see a window that is one token off."""
    cfg, cases = dc.planted_case()
    w = dc.Weights(cfg, 5, dc.plant(cfg)).f64()
    toks, at = cases[place]
    want = orc.forward(cfg, w, toks)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mixer"]["mask"]["size"] += change
    off = orc.forward(bad, w, toks)
    assert np.sqrt(np.mean((off - want) ** 2, axis=1))[at] > 0.2 * want.std()


@pytest.mark.parametrize("name", list(dc.CONFIGS))
def test_tensor_shapes_run_through_the_oracle(name):
    cfg = dc.CONFIGS[name]
    out = orc.forward(cfg, dc.Weights(cfg, 2).f64(), dc.tokens(cfg, 6))
    assert out.shape == (6, cfg["vocab"]) and np.isfinite(out).all()
