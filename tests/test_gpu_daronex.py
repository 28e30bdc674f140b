"""Daronex on the GPU against the plain oracle: each mechanism alone (also in layers of another design),
whole models, prompts against decoding, portions, reused rows and states, window edges, generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import dar_cases as dc
from oracle import daronex as orc
from oracle import zavilorn as zorc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = dict(float32=1e-4, bfloat16=0.035)
DTYPES = list(TOL)


def make(cfg, w, dtype, max_ctx=400):
    from cpp_tensorlib_b200.daronex import Daronex
    return Daronex.from_folder(cfg, w, dtype, max_ctx)


def weights(cfg, seed, edit=None):
    def both(w):
        dc.same_sign(cfg)(w)
        if edit:
            edit(w)
    return dc.Weights(cfg, seed, both)


def err(got, want):
    """Root mean square over the vocabulary of each row's difference, over the spread of the logits."""
    d = got - want
    return np.sqrt(np.mean((d - d.mean(-1, keepdims=True)) ** 2, axis=-1)) / want.std()


def ok(e, dtype):
    """f32: every position.  bf16: a position where two keys nearly tie, or a head's result nearly cancels
    before its norm, may be off by several times the usual rounding, so a few are allowed; the bulk of the
    positions has to lie far below the limit."""
    if dtype == "float32":
        return e.max() < TOL[dtype]
    return (e > TOL[dtype]).sum() <= max(1, 0.02 * len(e)) and e.max() < 0.25 and np.median(e) < 0.015


def run(m, toks, cuts):
    """Logits of every token, the sequence cut into portions of the given sizes, the rest one by one."""
    m.set_pos(0)
    out, at = [], 0
    for n in cuts:
        n = min(n, len(toks) - at)
        if n <= 0:
            break
        out.append(m.extend(toks[at:at + n], range(n)))
        at += n
    while at < len(toks):
        out.append(m.extend(toks[at:at + 1], [0]))
        at += 1
    return np.concatenate(out)


def close(m):
    st = (__import__("ctypes").c_int * 2)()
    from cpp_tensorlib_b200 import lib
    assert lib().tlb_device_status(st, 0) == 0
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(dc.CONFIGS))
def test_whole_prompt_and_decoding(name, dtype):
    cfg = dc.CONFIGS[name]
    w = weights(cfg, 11)
    toks = dc.tokens(cfg, 203, 1)
    want = orc.forward(cfg, w.f64(), toks)
    m = make(cfg, w, dtype)
    assert ok(err(run(m, toks, [len(toks)]), want), dtype)
    assert ok(err(run(m, toks, [150]), want), dtype)      # a prompt, then token by token
    m.capture()
    assert ok(err(run(m, toks, []), want), dtype)         # every token decoded, through the graph
    close(m)


# ---- one mechanism at a time, in layers with the norm in front ------------------------------------------
def pre_norm_stack(dtype, layers, W, width, vocab, eps, logit_scale=1.0):
    from cpp_tensorlib_b200 import stack
    m = stack.LayerStack(width, vocab, eps, 1.0, layers, dtype, 128, logit_scale=logit_scale)
    m.set_matrix(0, "embed", W["embed"])
    m.set_vector(0, "final", np.ones(width))
    m.set_vector(0, "norm1", 1 + W["l0.norm1"])
    return m


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["full", "window", "gla", "feed_forward", "norm_behind"])
def test_each_mechanism_alone(kind, dtype):
    """full, window, gla, feed_forward: one of them in a pre-norm layer with a gain; the output head is the
    embedding.  norm_behind: a sublayer whose output is normed, nothing else of the design."""
    from cpp_tensorlib_b200 import daronex, stack
    E, V, eps, gain = 64, 80, 1e-5, 3.0
    entry = dict(full=dc.full(6, 40, 24, 24, 32, 48), window=dc.win(11, 6, 40, 24, 24, 32, 48),
                 gla=dc.gla(6, 24, 20, 3.0), feed_forward=dc.full(2, 16, 8, 16, 16, 16, ff=72),
                 norm_behind=dc.gla(2, 16, 16, ff=0))[kind]
    cfg = dc.config([entry], width=E, vocab=V, eps=eps, logit_scale=0.7)
    w = weights(cfg, 21)
    W = w.f64()
    toks = dc.tokens(cfg, 77, 3)
    if kind == "norm_behind":
        x = W["embed"][toks]
        y = orc.gla_mixer(x, W, "l0.mix.", entry["mixer"], eps)
        want = orc.rms_norm(x + orc.rms_norm(y, 1 + W["l0.norm1"], eps), 1 + W["final.norm"], eps) @ W["head"].T * 0.7
        m = make(cfg, w, dtype, 128)
        for cuts in ([77], [30], [3, 40]):
            assert ok(err(run(m, toks, cuts), want), dtype)
        close(m)
        return
    spec = daronex.layer_spec(entry, 6)
    spec["mixers"][0].out_scale = 0.0 if kind == "feed_forward" else gain
    if kind != "feed_forward":
        spec["ff"] = 0
    m = pre_norm_stack(dtype, [spec], {n: w.f32(n) for n in w.names()}, E, V, eps, 0.5)
    d = daronex.Daronex.__new__(daronex.Daronex)      # the loader of one mixer, on this stack
    d.__dict__.update(m.__dict__)
    x = W["embed"][toks]
    h = orc.rms_norm(x, 1 + W["l0.norm1"], eps)
    mix = entry["mixer"]
    if kind == "gla":
        d._load_gla(0, "l0.mix.", mix, w)
        x = x + gain * orc.gla_mixer(h, W, "l0.mix.", mix, eps)
    else:
        d._load_latent(0, "l0.mix.", mix, w, kind == "window")
        if kind != "feed_forward":
            lat = orc.latent_of(h, W, "l0.mix.", mix, eps, kind == "window")
            x = x + gain * orc.latent_attention(h, W, "l0.mix.", mix, eps, kind == "window", mix.get("mask", {}).get("size"), lat)
    if kind == "feed_forward":
        m.set_vector(0, "norm2", 1 + w.f32("l0.norm2"))
        m.set_matrix(0, "gate_up", w.raw("l0.mlp.up"))
        m.set_matrix(0, "down", w.raw("l0.mlp.down"))
        h2 = orc.rms_norm(x, 1 + W["l0.norm2"], eps)
        x = x + orc.squared_relu_ff(h2, W["l0.mlp.up"], W["l0.mlp.down"])
    want = orc.rms_norm(x, np.ones(E), eps) @ W["embed"].T * 0.5
    for cuts in ([77], [30], [3, 40]):
        assert ok(err(run(m, toks, cuts), want), dtype)
    d.h = None
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixers_of_both_designs_in_one_layer(dtype):
    """A pre-norm layer with a windowed attention beside a gated linear one, and one with a latent
    attention beside a delta rule: every mixer serves any layer of the stack."""
    import zav_cases as zc
    from cpp_tensorlib_b200 import daronex, stack, zavilorn
    E, V, eps = 64, 80, 1e-5
    par = zc.par((6, 2, 16, 24), (4, 2, 24, 16), window=11, keep=2, rot=8, conv=3, ff=0)
    zcfg = zc.config([par, par], width=E, vocab=V, emb=1.0, eps=eps)
    dcfg = dc.config([dc.gla(3, 24, 20, 3.0, 0), dc.full(5, 16, 8, 24, 24, 40, ff=0)], width=E, vocab=V, eps=eps)
    zw, dw = zc.Weights(zcfg, 31), weights(dcfg, 32)
    Z, D = zw.f64(), dw.f64()
    za, zd = zavilorn.layer_spec(par)["mixers"]
    g, = daronex.layer_spec(dcfg["layers"][0], 6)["mixers"]
    f, = daronex.layer_spec(dcfg["layers"][1])["mixers"]
    for c, s in ((za, 0.8), (zd, 1.1), (g, 0.7), (f, 1.3)):
        c.out_scale = s
    m = stack.LayerStack(E, V, eps, 1.0, [dict(mixers=[za, g]), dict(mixers=[zd, f])], dtype, 128)
    m.set_matrix(0, "embed", zw.raw("embed"))
    m.set_vector(0, "final", np.ones(E))
    for i in (0, 1):
        m.set_vector(i, "norm1", zw.f32(f"l{i}.norm1"))
    l, p = "l0.mix.left.", "l0.mix."
    m.set_input(0, [zw.raw(l + n) for n in "qkvg"] + [dw.raw(p + n) for n in ("q", "k", "v", "g", "a1")])
    m.set_output(0, [zw.raw(l + "o"), dw.raw(p + "o")])
    m.set_vector(0, "q_norm", zw.f32(l + "q.norm"), 0)
    m.set_vector(0, "k_norm", zw.f32(l + "k.norm"), 0)
    m.set_vector(0, "norm", np.tile(dw.f32(p + "norm"), 3), 1)
    m.set_vector(0, "decay_up", dw.f32(p + "a2").T, 1)
    m.set_vector(0, "decay_bias", dw.f32(p + "a2.b"), 1)
    r, p = "l1.mix.right.", "l1.mix."
    dkv, C = dw.raw(p + "dkv"), 40
    m.set_input(1, [zw.raw(r + n) for n in "qkvgba"] + [dw.raw(p + "dq"), dkv[:C], dkv[C:]])
    m.set_output(1, [zw.raw(r + "o"), dw.raw(p + "o")])
    m.set_vector(1, "conv", np.concatenate([stack.pad_rows(zw.f32(r + n + ".conv")) for n in "qkv"]), 0)
    for n in ("norm", "dt_bias", "A_log"):
        m.set_vector(1, n, zw.f32(r + n), 0)
    m.set_vector(1, "q_norm", dw.f32(p + "dq.norm"), 1)
    m.set_vector(1, "k_norm", dw.f32(p + "dkv.norm"), 1)
    m.set_latent(1, 5, dw.raw(p + "uq"), dw.raw(p + "uk"), dw.raw(p + "uv"), 8, mixer=1)
    toks = dc.tokens(dcfg, 90, 4)
    x = Z["embed"][toks]
    h = orc.rms_norm(x, Z["l0.norm1"], eps)
    x = x + 0.8 * zorc.attention_mixer(h, Z, l, par["mixer"]["left"], eps) + \
        0.7 * orc.gla_mixer(h, D, "l0.mix.", dcfg["layers"][0]["mixer"], eps)
    h = orc.rms_norm(x, Z["l1.norm1"], eps)
    c = dcfg["layers"][1]["mixer"]
    x = x + 1.1 * zorc.delta_mixer(h, Z, r, par["mixer"]["right"], eps) + \
        1.3 * orc.latent_attention(h, D, "l1.mix.", c, eps, False, None, orc.latent_of(h, D, "l1.mix.", c, eps, False))
    want = orc.rms_norm(x, np.ones(E), eps) @ Z["embed"].T
    for cuts in ([90], [50], [2, 3, 40]):
        assert ok(err(run(m, toks, cuts), want), dtype)
    close(m)


# ---- how a sequence is cut, and what ran before ------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["base", "real"])
def test_portions_of_any_size(name, dtype):
    cfg = dc.CONFIGS[name]
    w = weights(cfg, 31)
    toks = dc.tokens(cfg, 240, 5)
    m = make(cfg, w, dtype)
    want = orc.forward(cfg, w.f64(), toks)
    for cuts in ([240], [2] * 120, [3, 2, 5, 7, 2, 2, 64, 65, 63, 2], [1, 2, 1, 100, 1, 2, 33, 31], [128, 64, 48], [17] * 14,
                 [15] * 16, [239]):
        assert ok(err(run(m, toks, cuts), want), dtype), cuts
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
def test_small_passes_wrap_the_kept_rows(dtype, monkeypatch):
    """Passes of 16 rows and rings far shorter than the sequence: rows are used many times, also by a layer
    that reads another one's with a wider window."""
    monkeypatch.setenv("TLB_PREFILL_CHUNK", "16")
    cfg = dc.config([dc.win(21), dc.gla(), dc.win(5, 4, 64, 16, 32, 24, 40), dc.win(34, kv_from=0, heads=3), dc.win(8, kv_from=0)])
    w = weights(cfg, 41)
    toks = dc.tokens(cfg, 330, 6)
    want = orc.forward(cfg, w.f64(), toks)
    m = make(cfg, w, dtype)
    big = make(cfg, w, dtype, 4000)
    assert m.state_bytes() == big.state_bytes()           # a window's state does not grow with the context
    big.close()
    for cuts in ([330], [100, 1, 1, 40], [], [7] * 47):
        assert ok(err(run(m, toks, cuts), want), dtype), cuts
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_one_after_the_other(dtype):
    """What a sequence leaves behind does not reach the next one, whatever their lengths."""
    cfg = dc.CONFIGS["base"]
    w = weights(cfg, 51)
    m = make(cfg, w, dtype, 300)
    m.capture()
    for seed, n, cuts in ((1, 260, [260]), (2, 1, []), (3, 2, [2]), (4, 3, []), (5, 90, [2, 3, 4]), (1, 260, [100]), (6, 37, [36])):
        toks = dc.tokens(cfg, n, seed)
        assert ok(err(run(m, toks, cuts), orc.forward(cfg, w.f64(), toks)), dtype), (seed, n)
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[130], [], [40, 2, 29, 21, 2], [69], [91, 30]])
def test_window_edges(dtype, cuts):
    """One key that stands out, just inside and just outside the window."""
    cfg, cases = dc.planted_case()
    w = weights(cfg, 5, dc.plant(cfg))
    m = make(cfg, w, dtype)
    for name, (toks, at) in cases.items():
        e = err(run(m, toks, cuts), orc.forward(cfg, w.f64(), toks))
        assert ok(e, dtype) and e[at] < TOL[dtype], name
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,dims", [(150, (8, 128, 64, 128, 64, 256)), (64, (4, 32, 32, 64, 32, 64)),
                                         (65, (17, 64, 32, 96, 48, 136)), (127, (2, 24, 16, 40, 24, 512))])
def test_window_edges_of_the_tiled_widths(dtype, window, dims):
    """The same at the widths and tile borders of the prompt and decode kernels: planted keys on both sides
    of the window's edge and at the borders of 64."""
    cfg = dc.config([dc.win(window, *dims), dc.gla()], width=96)
    w = weights(cfg, 6, dc.plant(cfg))
    m = make(cfg, w, dtype, 460)
    m.capture()
    for pairs in ([(64, 64 + window - 1)], [(70, 70 + window), (300, 303)], [(63, 64), (260, 260 + window - 1)], [(127, 127 + window)],
                  [(0, window - 1), (128, 128 + window)], [(0, window)]):
        toks = dc.planted_tokens(cfg, 450, pairs, 3)
        want = orc.forward(cfg, w.f64(), toks)
        for cuts in ([450], [64, 64, 130, 100], [199, 2, 2]):
            e = err(run(m, toks, cuts), want)
            assert ok(e, dtype) and max(e[i] for _, i in pairs) < TOL[dtype], (pairs, cuts)
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_and_a_shared_latent(dtype):
    """A key that stands out far back, the first token's among them, in an attention over everything and in
    a layer that reads its latent."""
    cfg = dc.config([dc.full(), dc.gla(ff=0), dc.full(heads=2, kv_from=0)])

    def edit(w):
        dc.plant(cfg)(w)
        p = "l2.mix."         # the reader asks through the same entry of the latent
        w[p + "uk"][::16] = 0
        w[p + "uk"][::16, 0] = 2.0
    w = weights(cfg, 7, edit)
    m = make(cfg, w, dtype, 720)
    m.capture()
    for pairs in ([(0, 690)], [(64, 650)], [(63, 660)], [(5, 300), (301, 699)]):
        toks = dc.planted_tokens(cfg, 700, pairs, 4)
        want = orc.forward(cfg, w.f64(), toks)
        moved = list(toks)
        moved[pairs[0][0]] = 9
        assert err(orc.forward(cfg, w.f64(), moved), want)[pairs[0][1]] > 0.2
        for cuts in ([700], [640], [256, 256, 100]):
            e = err(run(m, toks, cuts), want)
            assert ok(e, dtype) and max(e[i] for _, i in pairs) < TOL[dtype], (pairs, cuts)
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_remembers_far_tokens(dtype):
    """Slow decays: the recurrent state carries tokens over hundreds of steps, in prompts and decoding."""
    cfg = dc.config([dc.gla(4, 32, 32, 16.0), dc.win(2, 2), dc.gla(2, 64, 24, 16.0)])

    def slow(w):
        for n in w:
            if n.endswith("a2.b"):
                w[n] = w[n] * 0.3 + 4.0
    w = weights(cfg, 61, slow)
    toks = dc.tokens(cfg, 700, 7)
    want = orc.forward(cfg, w.f64(), toks)
    changed = [t if i else (t + 1) % cfg["vocab"] for i, t in enumerate(toks)]
    assert err(orc.forward(cfg, w.f64(), changed)[600:], want[600:]).min() > 5 * TOL["float32"]
    m = make(cfg, w, dtype, 710)
    m.capture()
    for cuts in ([700], [650], [10]):
        assert ok(err(run(m, toks, cuts), want), dtype)
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dims", [(3, 48, 40), (2, 128, 64), (1, 136, 24)])
def test_decays_of_every_strength(dtype, dims):
    """Channels that forget within a token beside ones that hardly decay, in one head: inside a chunk the
    running sums reach thousands, far outside an exponential's range."""
    cfg = dc.config([dc.gla(*dims, 0.5), dc.gla(*dims, 16.0)])

    def edit(w):
        rng = np.random.default_rng(1)
        for i in (0, 1):
            b = w[f"l{i}.mix.a2.b"]
            b[:] = rng.choice([-30.0, -6.0, 0.0, 6.0, 14.0], b.shape)
    w = weights(cfg, 71, edit)
    toks = dc.tokens(cfg, 300, 8)
    want = orc.forward(cfg, w.f64(), toks)
    m = make(cfg, w, dtype)
    assert ok(err(run(m, toks, [300]), want), dtype)
    assert ok(err(run(m, toks, [131, 2, 100]), want), dtype)
    close(m)


# ---- entry points ---------------------------------------------------------------------------------
def folder(tmp_path, cfg, w):
    from cpp_tensorlib_b200.safetensors import save
    save(tmp_path / "model.safetensors", {n: w.raw(n) for n in w.names()})
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    return str(tmp_path)


def greedy(cfg, w, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(np.argmax(orc.forward(cfg, w, t)[-1])))
    return t[len(prompt):]


@pytest.mark.parametrize("prompt_len", [1, 2, 45])
def test_greedy_generation(tmp_path, prompt_len):
    from cpp_tensorlib_b200.registry import load_model
    cfg = dc.CONFIGS["base"]
    w = weights(cfg, 81)
    m = load_model(folder(tmp_path, cfg, w), "float32", 128)
    prompt = dc.tokens(cfg, prompt_len, 9)
    want = greedy(cfg, w.f64(), prompt, 30)
    assert m.generate(prompt, 30) == want
    assert m.generate(prompt, 30) == want        # a second sequence on the same state
    if prompt_len > 1:                           # device-resident feedback from the prompt pass
        m.set_pos(0)
        m.prefill(prompt)
        m.run(29)
        assert m.last_token() == want[-1]
    close(m)


def test_command_line_and_trace(tmp_path):
    cfg = dc.CONFIGS["odd"]
    w = weights(cfg, 91)
    d = folder(tmp_path, cfg, w)
    prompt = dc.tokens(cfg, 24, 10)
    r = subprocess.run([sys.executable, "-m", "cpp_tensorlib_b200", "generate", "--model", d, "--dtype", "float32", "--tokens",
                        ",".join(map(str, prompt)), "-n", "8"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.strip().split(",")] == greedy(cfg, w.f64(), prompt, 8)
    want = orc.forward(cfg, w.f64(), prompt)
    steps = [dict(step=0, entries=[dict(id="q", tokens=prompt[:17], want=[6, 1])], end=[]),
             dict(step=1, entries=[dict(id="q", tokens=prompt[17:18], want=[0])], end=[]),
             dict(step=2, entries=[dict(id="q", tokens=prompt[18:], want=[])], end=["q"]),
             dict(step=3, entries=[dict(id="r", tokens=prompt[:1], want=[0])], end=["r"])]
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "24"], input="\n".join(map(json.dumps, steps)) + "\n", cwd=ROOT, capture_output=True,
                           text=True, timeout=300)
        assert r.returncode == 0, r.stderr
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        for n, rows in ((0, [6, 1]), (1, [17]), (3, [0])):
            got = np.fromfile(out / f"{n}.f32", "<f4").reshape(len(rows), -1)
            assert err(got, want[rows]).max() < 3 * TOL[dtype]
        assert not (out / "2.f32").exists()


def test_refusals():
    from cpp_tensorlib_b200 import TlbError
    cfg = dc.CONFIGS["base"]
    m = make(cfg, weights(cfg, 1), "bfloat16", 32)
    m.extend(dc.tokens(cfg, 20), [])
    with pytest.raises(TlbError):
        m.set_pos(7)
    with pytest.raises(TlbError):
        m.extend(dc.tokens(cfg, 13), [])   # 33 tokens
    m.extend(dc.tokens(cfg, 12), [])
    with pytest.raises(TlbError):
        m.step(1)
    close(m)
    for bad in (dc.config([dc.full(kv_from=0)]), dc.config([dc.full(), dc.full(kv_rank=40, kv_from=0)]),
                dc.config([dc.gla(), dc.full(kv_from=0)]), dc.config([dc.full(), dc.full(kv_from=0), dc.full(kv_from=1)]),
                dc.config([dc.full(kv_rank=9000)])):
        with pytest.raises(TlbError):
            make(bad, weights(bad, 1), "bfloat16", 32)
