"""Host side of the layer-stack model: configuration, fused matrices, safetensors, registry, trace
replay -- and the oracle checked against other ways to compute the same thing."""
import json

import numpy as np
import pytest

import zav_cases as zc
from cpp_tensorlib_b200 import registry, stack, trace, zavilorn
from cpp_tensorlib_b200.safetensors import SafeTensors, bf16_to_f32, f32_to_bf16, save
from oracle import zavilorn as orc


def test_registry_chooses_by_config():
    assert registry.model_class(dict(architecture="Zavilorn")) is zavilorn.Zavilorn
    assert registry.architecture(dict(architectures=["Qwen2ForCausalLM"])) == "Qwen2ForCausalLM"
    with pytest.raises(ValueError):
        registry.architecture(dict(architecture="Other"))
    with pytest.raises(ValueError):
        registry.load_model("/nowhere", dtype="int8")


def test_safetensors_round_trip(tmp_path):
    rng = np.random.default_rng(0)
    a = dict(x=rng.standard_normal((3, 5)).astype(np.float32), y=np.arange(7, dtype=np.int32),
             z=f32_to_bf16(rng.standard_normal((2, 3, 4)).astype(np.float32)))
    save(tmp_path / "m.safetensors", a)
    t = SafeTensors(tmp_path / "m.safetensors")
    assert t.names() == list(a) and t.shape("z") == (2, 3, 4)
    for n in a:
        assert np.array_equal(t.raw(n), a[n])
    assert np.array_equal(t.f32("z"), bf16_to_f32(a["z"]))
    assert np.array_equal(f32_to_bf16(t.f32("z")), a["z"])


def test_layer_spec_reads_every_constant():
    e = zc.par((6, 3, 24, 40), (4, 2, 16, 32), window=9, keep=2, rot=10, base=123.0, scale=0.3, conv=5, ff=48, limit=1.25,
               scales=(0.5, 0.7))
    s = zavilorn.layer_spec(e)
    a, d = s["mixers"]
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first, a.rot_dims) == (1, 6, 3, 24, 40, 9, 2, 10)
    assert np.allclose([a.rot_base, a.scale, a.out_scale, d.out_scale, s["limit"]], [123.0, 0.3, 0.5, 0.7, 1.25])
    assert (d.kind, d.heads, d.kv_heads, d.dim, d.vdim, d.conv, s["ff"]) == (2, 4, 2, 16, 32, 5, 48)
    m, = zavilorn.layer_spec(zc.mam(6, 3, 10, 14, 2, 4))["mixers"]
    assert (m.kind, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, m.norm_groups) == (3, 6, 3, 10, 14, 2, 4)
    with pytest.raises(ValueError):
        zavilorn.layer_spec(dict(type="other", mixer={}))


def test_fused_matrices_keep_every_row(monkeypatch):
    """Every part of the fused input, output and gate|up matrices lies where the native side reads it."""
    cfg = zc.CONFIGS["odd"]
    got = {}
    z = zavilorn.Zavilorn.__new__(zavilorn.Zavilorn)
    z.config, z.f32 = cfg, True
    monkeypatch.setattr(z, "set_matrix", lambda l, n, a: got.__setitem__((l, n), z.weight(a)), raising=False)
    monkeypatch.setattr(z, "set_vector", lambda l, n, v, mixer=0: got.__setitem__((l, n, mixer), v), raising=False)
    w = zc.Weights(cfg, 1)
    z.load(w)
    at = 0
    for n in ("left.q", "left.k", "left.v", "left.g", "right.q", "right.k", "right.v", "right.g", "right.b", "right.a"):
        t = w.f32("l0.mix." + n)
        assert np.array_equal(got[0, "input"][at:at + len(t)], t)
        assert not got[0, "input"][at + len(t):at + stack.pad8(len(t))].any()
        at += stack.pad8(len(t))
    assert at == len(got[0, "input"])
    lo, ro = w.f32("l0.mix.left.o"), w.f32("l0.mix.right.o")
    assert np.array_equal(got[0, "output"][:, :lo.shape[1]], lo)
    k = stack.pad8(lo.shape[1])
    assert np.array_equal(got[0, "output"][:, k:k + ro.shape[1]], ro)
    assert np.array_equal(got[0, "gate_up"][0::2], w.f32("l0.mlp.gate"))
    assert np.array_equal(got[0, "gate_up"][1::2], w.f32("l0.mlp.up"))
    inner, h = 3 * 7, 3
    full = w.f32("l1.mix.in")
    z8, x8 = stack.pad8(inner), stack.pad8(inner + 20)
    assert np.array_equal(got[1, "input"][:inner], full[:inner])
    assert np.array_equal(got[1, "input"][z8:z8 + inner + 20], full[inner:2 * inner + 20])
    assert np.array_equal(got[1, "input"][z8 + x8:z8 + x8 + h], full[-h:])


class FakeModel:
    captured = True

    def __init__(self):
        self.log = []

    def set_pos(self, p):
        self.log.append(("pos", p))

    def extend(self, tokens, want):
        self.log.append((list(tokens), list(want)))
        return np.array([[t * 10 + w] for t, w in zip([tokens[i] for i in want], want)], np.float32).reshape(len(want), 1)


def test_trace_replay(tmp_path):
    m, out = FakeModel(), []
    lines = [json.dumps(s) for s in (
        dict(step=0, entries=[dict(id="a", tokens=[5, 6, 7], want=[2, 0])], end=[]),
        dict(step=1, entries=[dict(id="a", tokens=[8], want=[])], end=["a"]),
        dict(step=2, entries=[dict(id="b", tokens=[9], want=[0])], end=["b"]))]
    trace.replay(m, lines, str(tmp_path), out.append)
    assert out == ["done 0", "done 1", "done 2"]
    assert m.log == [("pos", 0), ([5, 6, 7], [0, 2]), ([8], []), ("pos", 0), ([9], [0])]
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [72.0, 50.0]
    assert not (tmp_path / "1.f32").exists()
    with pytest.raises(ValueError):
        trace.replay(m, [json.dumps(dict(step=0, entries=[dict(id="a", tokens=[1], want=[])], end=[])),
                         json.dumps(dict(step=1, entries=[dict(id="b", tokens=[1], want=[])], end=[]))],
                     str(tmp_path), out.append)


# ---- the oracle against other ways ------------------------------------------------------------
def test_oracle_window_rule():
    for i in range(30):
        for j in range(30):
            assert orc.sees(i, j, 5, 2) == (j <= i and (j >= i - 4 or j in (0, 1)))


def test_oracle_attention_is_masked_softmax():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((17, 4, 6)), rng.standard_normal((17, 2, 6)), rng.standard_normal((17, 2, 5))
    got = orc.window_attention(q, k, v, 0.7, 5, 2)
    mask = np.array([[orc.sees(i, j, 5, 2) for j in range(17)] for i in range(17)])
    for h in range(4):
        s = np.where(mask, q[:, h] @ k[:, h // 2].T * 0.7, -np.inf)
        p = np.exp(s - s.max(1, keepdims=True))
        assert np.allclose(got[:, h], p / p.sum(1, keepdims=True) @ v[:, h // 2])


def test_oracle_rotation_keeps_distance():
    x = np.random.default_rng(1).standard_normal((2, 1, 8))
    a = orc.rotate(x, np.array([3, 10]), 6, 100.0)
    b = orc.rotate(x, np.array([53, 60]), 6, 100.0)
    assert np.allclose(a[0, 0] @ a[1, 0], b[0, 0] @ b[1, 0])
    assert np.array_equal(a[..., 6:], x[..., 6:]) and not np.allclose(a[..., :6], x[..., :6])


def test_oracle_ssd_is_a_decayed_sum():
    rng = np.random.default_rng(2)
    x, B, C = rng.standard_normal((9, 4, 3)), rng.standard_normal((9, 2, 5)), rng.standard_normal((9, 2, 5))
    dt, A, D = rng.random((9, 4)), rng.random(4), rng.standard_normal(4)
    got = orc.ssd(x, B, C, dt, A, D)
    for t in range(9):
        for h in range(4):
            y = D[h] * x[t, h] + sum(np.exp(-A[h] * dt[s + 1:t + 1, h].sum()) * dt[s, h] * (C[t, h // 2] @ B[s, h // 2]) * x[s, h]
                                     for s in range(t + 1))
            assert np.allclose(got[t, h], y)


def test_oracle_delta_rule_overwrites():
    """With beta 1 and no decay a unit key reads back exactly the value written last under it."""
    k = np.zeros((3, 1, 4))
    k[0, 0, 0] = k[1, 0, 1] = k[2, 0, 0] = 1
    v = np.random.default_rng(3).standard_normal((3, 1, 2))
    o = orc.delta_rule(k, k, v, np.ones((3, 1)), np.ones((3, 1)))
    assert np.allclose(o, v)
    o = orc.delta_rule(k[[0, 1, 0]], k, v * np.array([1, 1, 0])[:, None, None], np.array([[1.], [1.], [0.]]), np.full((3, 1), 0.5))
    assert np.allclose(o[2, 0], 0.25 * v[0, 0])


def planted_case():
    """A configuration and sequences (tokens, place of the query) with one asked-for key each: name -> ..."""
    cfg = zc.config([zc.par(window=20, keep=3, rot=8, scales=(4.0, 1.0)), zc.mam()])
    pairs = dict(first_in=(2, 40), first_out=(3, 40), inside=(50, 69), outside=(71, 91), near=(100, 103))
    return cfg, {k: (zc.planted_tokens(cfg, 130, [p]), p[1]) for k, p in pairs.items()}


@pytest.mark.parametrize("mask_edit,place", [
    (dict(size=+1), "outside"), (dict(size=-1), "inside"), (dict(keep_first=+1), "first_out"), (dict(keep_first=-1), "first_in")])
def test_planted_keys_show_a_shifted_edge(mask_edit, place):
    """The planted queries see a window or a kept run that is one token off."""
    cfg, cases = planted_case()
    w = zc.Weights(cfg, 5, zc.plant(cfg)).f64()
    toks, at = cases[place]
    want = orc.forward(cfg, w, toks)
    bad = json.loads(json.dumps(cfg))
    for k, d in mask_edit.items():
        bad["layers"][0]["mixer"]["left"]["mask"][k] += d
    off = orc.forward(bad, w, toks)
    rms = np.sqrt(np.mean((off - want) ** 2, axis=1)) / want.std()
    assert rms[at] > 0.2


@pytest.mark.parametrize("name", list(zc.CONFIGS))
def test_tensor_shapes_run_through_the_oracle(name):
    cfg = zc.CONFIGS[name]
    out = orc.forward(cfg, zc.Weights(cfg, 2).f64(), zc.tokens(cfg, 6))
    assert out.shape == (6, cfg["vocab"]) and np.isfinite(out).all()
