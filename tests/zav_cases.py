"""Small Zavilorn configurations and weights for the tests, and the oracle's view of them."""
import numpy as np

from cpp_tensorlib_b200.safetensors import bf16_to_f32, f32_to_bf16
from cpp_tensorlib_b200.zavilorn import tensor_shapes


def par(left=(4, 2, 16, 16), right=(4, 2, 16, 16), window=20, keep=3, rot=8, base=1000.0, scale=None, conv=4, ff=40,
        limit=2.0, scales=(0.8, 1.1)):
    h, g, d, e = left
    rh, rg, rd, re = right
    return dict(type="parallel", mlp=dict(kind="dense", ff=ff, limit=limit) if ff else None, mixer=dict(
        left=dict(heads=h, kv_heads=g, dim=d, vdim=e, mask=dict(size=window, keep_first=keep),
                  rot=dict(base=base, dims=rot), scale=scale or d ** -0.5),
        right=dict(heads=rh, kv_heads=rg, dim=rd, vdim=re, conv=conv), left_scale=scales[0], right_scale=scales[1]))


def mam(heads=4, groups=2, state=16, vdim=16, conv=4, norm_groups=2, ff=0, limit=3.0):
    return dict(type="mamba2", mlp=dict(kind="dense", ff=ff, limit=limit) if ff else None,
                mixer=dict(heads=heads, groups=groups, state=state, vdim=vdim, conv=conv, norm_groups=norm_groups))


def config(layers, width=64, vocab=96, emb=4.0, eps=1e-5):
    return dict(architecture="Zavilorn", vocab=vocab, width=width, embedding=dict(scale=emb), norm=dict(eps=eps),
                layers=layers)


CONFIGS = dict(
    base=config([par(), mam(), mam(ff=24), par(ff=0)]),
    # nothing a multiple of anything, one head, one tap, no kept tokens, every dimension rotated
    odd=config([par((3, 3, 22, 10), (6, 3, 20, 13), window=7, keep=0, rot=22, conv=1, ff=37),
                mam(3, 1, 10, 7, 2, 3, ff=11), mam(5, 5, 9, 6, 1, 1)], width=52, vocab=71, emb=1.0),
    # many query heads on one key head, values wider than keys, a window longer than the sequences
    wide=config([mam(6, 3, 40, 24, 3, 4), par((20, 1, 24, 40), (8, 1, 48, 80), window=4000, keep=1, rot=12, conv=5, ff=56)],
                width=72, vocab=128, emb=2.5),
    # the widths the tiled kernels are made for
    real=config([par((8, 2, 128, 128), (4, 2, 128, 128), window=150, keep=5, rot=64, conv=4, ff=192),
                 mam(6, 2, 128, 64, 4, 2), mam(4, 2, 64, 128, 4, 1), par((4, 4, 64, 64), (4, 4, 64, 64), window=64, keep=64, rot=32)],
                width=128, vocab=160, emb=3.0),
    narrow=config([par((2, 1, 96, 96), (2, 2, 32, 48), window=33, keep=2, rot=96, conv=2, ff=64), mam(2, 1, 48, 32, 3, 2)],
                  width=96, vocab=64),
)


class Weights:
    """Random bf16-exact weights; `edit` may change the f32 dict before it is rounded."""

    def __init__(self, cfg, seed, edit=None, slow=True):
        rng = np.random.default_rng(seed)
        self.w = {}
        for n, s in tensor_shapes(cfg).items():
            a = rng.standard_normal(s).astype(np.float32)
            if n.endswith(("norm", "norm1", "norm2")):
                a = 1.0 + 0.3 * a
            elif n.endswith("A_log"):
                a = 0.5 * a - (1.0 if slow else 0.0)
            elif n.endswith("dt_bias"):
                a = a - (2.5 if slow else 0.0)
            elif n.endswith("conv"):
                a = a * s[1] ** -0.5
            elif n.endswith("conv.b"):
                a = 0.2 * a
            elif n == "embed":
                a = a / cfg["embedding"]["scale"]
            elif len(s) == 2:
                a = a * s[1] ** -0.5
            self.w[n] = a
        if edit:
            edit(self.w)
        self.w = {n: bf16_to_f32(f32_to_bf16(a)) for n, a in self.w.items()}

    def f32(self, n):
        return self.w[n]

    def raw(self, n):
        return f32_to_bf16(self.w[n])

    def __contains__(self, n):
        return n in self.w

    def names(self):
        return list(self.w)

    def f64(self):
        return {n: a.astype(np.float64) for n, a in self.w.items()}


def tokens(cfg, n, seed=0):
    return [int(t) for t in np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n)]


# ---- a key that stands out: token A asks for token B through a channel of its own --------------
A_TOK, B_TOK = 1, 2


def plant(cfg, layer=0, strength=60.0):
    """Edit of Weights: in every attention head of `layer`, a query of token A scores far higher on a key
    of token B than on anything else, in a dimension that is not rotated."""
    left = cfg["layers"][layer]["mixer"]["left"]
    d0 = left["rot"]["dims"]
    assert d0 < left["dim"]
    p = f"l{layer}.mix.left."

    def edit(w):
        w["embed"][:, :2] = 0
        w["embed"][A_TOK, 0] = w["embed"][B_TOK, 1] = 6.0 / cfg["embedding"]["scale"]
        w[f"l{layer}.norm1"][:2] = 1.0
        for name, ch, heads in (("q", 0, left["heads"]), ("k", 1, left["kv_heads"])):
            for h in range(heads):
                w[p + name][h * left["dim"] + d0] = 0
                w[p + name][h * left["dim"] + d0, ch] = strength ** 0.5
                w[p + name + ".norm"][h * left["dim"] + d0] = 2.0
    return edit


def planted_tokens(cfg, n, pairs, seed=0):
    """Random tokens without A and B, then B at j and A at i for each (j, i)."""
    t = [x if x > 2 else x + 3 for x in tokens(cfg, n, seed)]
    for j, i in pairs:
        t[j], t[i] = B_TOK, A_TOK
    return t
