"""The layer-stack model on the GPU against the plain oracle: each mechanism alone, whole models,
prompts against decoding, portions, reused state, window edges, generation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import zav_cases as zc
from oracle import zavilorn as orc
from test_zavilorn_cpu import planted_case

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = dict(float32=2e-4, bfloat16=0.035)
DTYPES = list(TOL)


def make(cfg, w, dtype, max_ctx=400):
    from cpp_tensorlib_b200.zavilorn import Zavilorn
    m = Zavilorn(cfg, dtype, max_ctx)
    m.load(w)
    return m


def err(got, want):
    """Root mean square over the vocabulary of each row's difference, over the spread of the logits."""
    d = got - want
    return np.sqrt(np.mean((d - d.mean(-1, keepdims=True)) ** 2, axis=-1)) / want.std()


def ok(e, dtype):
    """f32: every position.  bf16: a position where two keys nearly tie, or a head's result nearly
    cancels before its norm, may be off by several times the usual rounding, so a few are allowed;
    the bulk of the positions has to lie far below the limit."""
    if dtype == "float32":
        return e.max() < TOL[dtype]
    return (e > TOL[dtype]).sum() <= max(1, 0.02 * len(e)) and e.max() < 0.25 and np.median(e) < 0.012


def run(m, toks, cuts):
    """Logits of every token, the sequence cut into portions of the given sizes."""
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
@pytest.mark.parametrize("name", list(zc.CONFIGS))
def test_whole_prompt_and_decoding(name, dtype):
    cfg = zc.CONFIGS[name]
    w = zc.Weights(cfg, 11)
    toks = zc.tokens(cfg, 203, 1)
    want = orc.forward(cfg, w.f64(), toks)
    m = make(cfg, w, dtype)
    whole = run(m, toks, [len(toks)])
    assert ok(err(whole, want), dtype)
    tail = run(m, toks, [150])                 # a prompt, then token by token
    assert ok(err(tail, want), dtype)
    m.capture()
    single = run(m, toks, [])                  # every token decoded, through the graph
    assert ok(err(single, want), dtype)
    close(m)


# ---- one mechanism at a time --------------------------------------------------------------------
def head_logits(x, embed, eps):
    return orc.rms_norm(x, np.ones(x.shape[1]), eps) @ embed.T


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "delta", "ssd", "feed_forward"])
def test_each_mechanism_alone(kind, dtype):
    from cpp_tensorlib_b200 import stack
    E, V, eps = 64, 80, 1e-5
    par = zc.par((6, 2, 40, 24), (6, 3, 24, 40), window=11, keep=2, rot=16, conv=3, scales=(1.0, 1.0))
    mam = zc.mam(6, 2, 24, 20, 3, 3)
    cfg = zc.config([mam if kind == "ssd" else par], width=E, vocab=V, emb=1.0, eps=eps)
    w = zc.Weights(cfg, 21)
    W = w.f64()
    W["final.norm"][:] = 1.0
    toks = zc.tokens(cfg, 77, 3)
    x = W["embed"][toks]
    h = orc.rms_norm(x, W["l0.norm1"], eps)
    l, r = par["mixer"]["left"], par["mixer"]["right"]
    gain = 3.0
    if kind == "attention":
        mixers = [stack.mixer_cfg(stack.ATTN, 6, 2, 40, 24, gain, window=11, keep_first=2, rot_dims=16, rot_base=l["rot"]["base"], scale=l["scale"])]
        x = x + gain * orc.attention_mixer(h, W, "l0.mix.left.", l, eps)
    elif kind == "delta":
        mixers = [stack.mixer_cfg(stack.DELTA, 6, 3, 24, 40, gain, conv=3)]
        x = x + gain * orc.delta_mixer(h, W, "l0.mix.right.", r, eps)
    elif kind == "ssd":
        mixers = [stack.mixer_cfg(stack.SSD, 6, 2, 24, 20, gain, conv=3, norm_groups=3)]
        x = x + gain * orc.mamba2_mixer(h, W, "l0.mix.", mam["mixer"], eps)
    else:   # behind an attention whose result is scaled away
        mixers = [stack.mixer_cfg(stack.ATTN, 6, 2, 40, 24, 0.0, window=11, keep_first=2, rot_dims=16, rot_base=10.0, scale=1.0)]
        mlp = par["mlp"]
        h2 = orc.rms_norm(x, W["l0.norm2"], eps)
        x = x + orc.clipped_glu(h2 @ W["l0.mlp.gate"].T, h2 @ W["l0.mlp.up"].T, mlp["limit"]) @ W["l0.mlp.down"].T
    ff = kind == "feed_forward"
    m = stack.LayerStack(E, V, eps, 1.0, [dict(mixers=mixers, ff=par["mlp"]["ff"] if ff else 0, limit=par["mlp"]["limit"])],
                         dtype, 128)
    m.set_matrix(0, "embed", w.raw("embed"))
    m.set_vector(0, "final", np.ones(E))
    m.set_vector(0, "norm1", w.f32("l0.norm1"))
    p = "l0.mix." if kind == "ssd" else ("l0.mix.right." if kind == "delta" else "l0.mix.left.")
    pad = stack.pad_rows
    if kind in ("attention", "feed_forward"):
        m.set_input(0, [w.raw(p + n) for n in "qkvg"])
        m.set_vector(0, "q_norm", w.f32(p + "q.norm"))
        m.set_vector(0, "k_norm", w.f32(p + "k.norm"))
    elif kind == "delta":
        m.set_input(0, [w.raw(p + n) for n in "qkvgba"])
        m.set_vector(0, "conv", np.concatenate([pad(w.f32(p + n + ".conv")) for n in "qkv"]))
    else:
        t, inner = w.raw(p + "in"), 120
        m.set_input(0, [t[:inner], t[inner:-6], t[-6:]])
        m.set_vector(0, "conv", pad(w.f32(p + "conv")))
        m.set_vector(0, "conv_bias", pad(w.f32(p + "conv.b")))
        m.set_vector(0, "skip", w.f32(p + "D"))
    if kind in ("delta", "ssd"):
        for n, k in (("norm", "norm"), ("dt_bias", "dt_bias"), ("A_log", "A_log")):
            m.set_vector(0, n, w.f32(p + k))
    m.set_output(0, [w.raw(p + "o")])
    if ff:
        m.set_vector(0, "norm2", w.f32("l0.norm2"))
        m.set_gate_up(0, w.raw("l0.mlp.gate"), w.raw("l0.mlp.up"))
        m.set_matrix(0, "down", w.raw("l0.mlp.down"))
    want = head_logits(x, W["embed"], eps)
    assert ok(err(run(m, toks, [77]), want), dtype)
    assert ok(err(run(m, toks, [30]), want), dtype)
    close(m)


# ---- how a sequence is cut, and what ran before ----------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["base", "real"])
def test_portions_of_any_size(name, dtype):
    cfg = zc.CONFIGS[name]
    w = zc.Weights(cfg, 31)
    toks = zc.tokens(cfg, 240, 5)
    m = make(cfg, w, dtype)
    whole = run(m, toks, [len(toks)])
    want = orc.forward(cfg, w.f64(), toks)
    assert ok(err(whole, want), dtype)
    for cuts in ([2] * 120, [3, 2, 5, 7, 2, 2, 64, 65, 63, 2], [1, 2, 1, 100, 1, 2, 33, 31], [128, 64, 48], [17] * 14, [239]):
        assert ok(err(run(m, toks, cuts), want), dtype), cuts
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
def test_small_passes_wrap_the_ring(dtype, monkeypatch):
    """Passes of 16 rows and a cache ring far shorter than the sequence: slots are used many times."""
    monkeypatch.setenv("TLB_PREFILL_CHUNK", "16")
    cfg = zc.config([zc.par(window=21, keep=3), zc.mam(), zc.par((4, 1, 64, 32), window=5, keep=0, rot=16)])
    w = zc.Weights(cfg, 41)
    toks = zc.tokens(cfg, 330, 6)
    want = orc.forward(cfg, w.f64(), toks)
    m = make(cfg, w, dtype)
    assert m.state_bytes() < make(cfg, w, dtype, 4000).state_bytes() * 2
    for cuts in ([330], [100, 1, 1, 40], [], [7] * 47):
        assert ok(err(run(m, toks, cuts), want), dtype), cuts
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sequences_one_after_the_other(dtype):
    """What a sequence leaves behind does not reach the next one, whatever their lengths."""
    cfg = zc.CONFIGS["base"]
    w = zc.Weights(cfg, 51)
    m = make(cfg, w, dtype, 300)
    m.capture()
    for seed, n, cuts in ((1, 260, [260]), (2, 1, []), (3, 2, [2]), (4, 3, []), (5, 90, [2, 3, 4]), (1, 260, [100]), (6, 37, [36])):
        toks = zc.tokens(cfg, n, seed)
        assert ok(err(run(m, toks, cuts), orc.forward(cfg, w.f64(), toks)), dtype), (seed, n)
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[130], [], [40, 2, 29, 21, 2], [69], [91, 30]])
def test_window_edges_and_kept_tokens(dtype, cuts):
    """One key that stands out, just inside and just outside the window and the kept run."""
    cfg, cases = planted_case()
    w = zc.Weights(cfg, 5, zc.plant(cfg))
    m = make(cfg, w, dtype)
    for name, (toks, at) in cases.items():
        e = err(run(m, toks, cuts), orc.forward(cfg, w.f64(), toks))
        assert ok(e, dtype) and e[at] < TOL[dtype], name
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,dims", [(150, (8, 2, 128, 128)), (64, (4, 4, 64, 64)), (65, (6, 1, 96, 96)), (127, (2, 2, 80, 48))])
def test_window_edges_of_the_tiled_widths(dtype, window, dims):
    """The same at the widths and tile borders of the prompt kernels: planted keys on both sides of the
    window's edge, of the kept run's, and at the borders of 64."""
    keep = 5
    cfg = zc.config([zc.par(dims, window=window, keep=keep, rot=32, scales=(4.0, 1.0))], width=96)
    w = zc.Weights(cfg, 6, zc.plant(cfg))
    m = make(cfg, w, dtype, 460)
    for pairs in ([(keep - 1, 200)], [(keep, 201)], [(0, 300)], [(64, 64 + window - 1)], [(70, 70 + window), (300, 303)],
                  [(63, 64), (260, 260 + window - 1)], [(127, 127 + window)]):
        toks = zc.planted_tokens(cfg, 450, pairs, 3)
        want = orc.forward(cfg, w.f64(), toks)
        for cuts in ([450], [64, 64, 130, 100], [199, 2, 2]):
            e = err(run(m, toks, cuts), want)
            assert ok(e, dtype) and max(e[i] for _, i in pairs) < TOL[dtype], (pairs, cuts)
    close(m)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_remembers_far_tokens(dtype):
    """Slow decays: the recurrent state carries tokens over hundreds of steps, in prompts and decoding."""
    cfg = zc.config([zc.mam(4, 2, 32, 32), zc.par((2, 1, 16, 16), (4, 4, 32, 32), window=2, keep=0)], width=64)

    def slow(w):
        for n in w:
            if n.endswith("A_log"):
                w[n] = w[n] * 0.2 - 4.0
            if n.endswith("mix.D"):
                w[n] *= 0.1
    w = zc.Weights(cfg, 61, slow)
    toks = zc.tokens(cfg, 700, 7)
    want = orc.forward(cfg, w.f64(), toks)
    changed = [t if i else (t + 1) % cfg["vocab"] for i, t in enumerate(toks)]
    assert err(orc.forward(cfg, w.f64(), changed)[600:], want[600:]).min() > 5 * TOL["float32"]
    m = make(cfg, w, dtype, 710)
    m.capture()
    for cuts in ([700], [650], [10]):
        assert ok(err(run(m, toks, cuts), want), dtype)
    close(m)


def test_strong_decay_and_large_steps():
    """Decays that forget within a token, and ones near one, in the same model."""
    cfg = zc.config([zc.mam(4, 2, 64, 64), zc.par(right=(4, 2, 64, 64))], width=64)

    def edit(w):
        w["l0.mix.A_log"][:] = [3.0, -6.0, 1.0, 5.0]
        w["l0.mix.dt_bias"][:] = [3.0, 2.0, -6.0, 4.0]
        w["l1.mix.right.A_log"][:] = [4.0, -7.0, 0.0, 2.0]
        w["l1.mix.right.dt_bias"][:] = [4.0, 0.0, -5.0, 6.0]
    w = zc.Weights(cfg, 71, edit)
    toks = zc.tokens(cfg, 300, 8)
    want = orc.forward(cfg, w.f64(), toks)
    for dtype in DTYPES:
        m = make(cfg, w, dtype)
        assert ok(err(run(m, toks, [300]), want), dtype)
        assert ok(err(run(m, toks, [131, 2, 100]), want), dtype)
        close(m)


# ---- entry points ------------------------------------------------------------------------------
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
    cfg = zc.CONFIGS["base"]
    w = zc.Weights(cfg, 81)
    m = load_model(folder(tmp_path, cfg, w), "float32", 128)
    prompt = zc.tokens(cfg, prompt_len, 9)
    want = greedy(cfg, w.f64(), prompt, 30)
    assert m.generate(prompt, 30) == want
    assert m.generate(prompt, 30) == want        # a second sequence on the same state
    # device-resident feedback from the prompt pass
    if prompt_len > 1:
        m.set_pos(0)
        m.prefill(prompt)
        m.run(29)
        assert m.last_token() == want[-1]
    close(m)


def test_command_line_and_trace(tmp_path):
    cfg = zc.CONFIGS["odd"]
    w = zc.Weights(cfg, 91)
    d = folder(tmp_path, cfg, w)
    prompt = zc.tokens(cfg, 12, 10)
    r = subprocess.run([sys.executable, "-m", "cpp_tensorlib_b200", "generate", "--model", d, "--dtype", "float32", "--tokens",
                        ",".join(map(str, prompt)), "-n", "8"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.strip().split(",")] == greedy(cfg, w.f64(), prompt, 8)
    out = tmp_path / "out"
    out.mkdir()
    steps = [dict(step=0, entries=[dict(id="q", tokens=prompt[:7], want=[6, 1])], end=[]),
             dict(step=1, entries=[dict(id="q", tokens=prompt[7:8], want=[0])], end=[]),
             dict(step=2, entries=[dict(id="q", tokens=prompt[8:], want=[])], end=["q"]),
             dict(step=3, entries=[dict(id="r", tokens=prompt[:1], want=[0])], end=["r"])]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "16"], input="\n".join(map(json.dumps, steps)) + "\n", cwd=ROOT, capture_output=True,
                       text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    want = orc.forward(cfg, w.f64(), prompt)
    for n, rows in ((0, [6, 1]), (1, [7]), (3, [0])):
        got = np.fromfile(out / f"{n}.f32", "<f4").reshape(len(rows), -1)
        assert err(got, want[rows]).max() < TOL["float32"]
    assert not (out / "2.f32").exists()


def test_refusals():
    from cpp_tensorlib_b200 import TlbError
    cfg = zc.CONFIGS["base"]
    m = make(cfg, zc.Weights(cfg, 1), "bfloat16", 32)
    m.extend(zc.tokens(cfg, 20), [])
    with pytest.raises(TlbError):
        m.set_pos(7)                       # a recurrent state cannot be moved back
    m.set_pos(20)
    with pytest.raises(TlbError):
        m.extend(zc.tokens(cfg, 13), [])   # 33 tokens
    with pytest.raises(TlbError):
        m.step(cfg["vocab"])
    m.extend(zc.tokens(cfg, 12), [])
    with pytest.raises(TlbError):
        m.step(1)
    close(m)


def test_qwen2_folder_through_the_registry(tmp_path):
    """The int4 decoder from a checkpoint folder generates what it generates from loaded arrays."""
    import cases
    import torch
    from cpp_tensorlib_b200.decoder import Q4Decoder
    from cpp_tensorlib_b200.registry import load_model
    from cpp_tensorlib_b200.safetensors import save
    c = cases.TINY64
    wts = cases.decoder_weights(c, 5)
    HD, nq, nk = c["hd"], c["n_q"], c["n_kv"]
    t = {"model.embed_tokens.weight": wts["embed"], "model.norm.weight": wts["onorm"], "lm_head.weight": wts["lm_head"].T}
    for l, L in enumerate(wts["layers"]):
        p = f"model.layers.{l}."
        q = L["wqkv"].T
        t.update({p + "self_attn.q_proj.weight": q[:nq * HD], p + "self_attn.k_proj.weight": q[nq * HD:(nq + nk) * HD],
                  p + "self_attn.v_proj.weight": q[(nq + nk) * HD:], p + "self_attn.o_proj.weight": L["wo"].T,
                  p + "mlp.gate_proj.weight": L["wgu"].T[:c["ff"]], p + "mlp.up_proj.weight": L["wgu"].T[c["ff"]:],
                  p + "mlp.down_proj.weight": L["wd"].T, p + "input_layernorm.weight": L["an"],
                  p + "post_attention_layernorm.weight": L["fn"], p + "self_attn.q_proj.bias": L["bq"],
                  p + "self_attn.k_proj.bias": L["bk"], p + "self_attn.v_proj.bias": L["bv"]})
    save(tmp_path / "model.safetensors", {k: np.ascontiguousarray(v, dtype=np.float32) for k, v in t.items()})
    if nq * HD != c["hidden"]:
        pytest.skip("this configuration's heads do not make up its width")
    (tmp_path / "config.json").write_text(json.dumps(dict(
        architectures=["Qwen2ForCausalLM"], hidden_size=c["hidden"], num_hidden_layers=c["layers"], num_attention_heads=nq,
        num_key_value_heads=nk, intermediate_size=c["ff"], vocab_size=c["vocab"], rms_norm_eps=c["eps"], rope_theta=c["rope_base"])))
    a = load_model(str(tmp_path), "float32", 64)
    b = Q4Decoder(c, 64)
    b.load(wts)
    prompt = [3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5, 8]
    assert a.generate(prompt, 12) == b.generate(prompt, 12)
    a.set_pos(0)
    lg = a.extend(prompt, [4, 11])
    b.set_pos(0)
    b.prefill(prompt)
    assert np.array_equal(lg[1], b.host_logits())
    torch.cuda.synchronize()
    a.close()
    b.close()
