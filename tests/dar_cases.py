"""Small Daronex configurations and weights for the tests, and the oracle's view of them."""
import numpy as np

from cpp_tensorlib_b200.daronex import tensor_shapes
from cpp_tensorlib_b200.safetensors import bf16_to_f32, f32_to_bf16
from zav_cases import tokens  # noqa: F401


def _latent(heads, dim, rot, vdim, q_rank, kv_rank, base, scale):
    return dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, rot=dict(base=base, dims=rot),
                scale=scale or (dim + rot) ** -0.5)


def _mlp(ff):
    return dict(kind="dense", ff=ff) if ff else None


def full(heads=4, dim=16, rot=8, vdim=16, q_rank=24, kv_rank=32, base=1000.0, scale=None, ff=40, kv_from=None):
    m = _latent(heads, dim, rot, vdim, q_rank, kv_rank, base, scale)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mlp=_mlp(ff), mixer=m)


def win(size=20, heads=4, dim=16, rot=8, vdim=16, q_rank=24, kv_rank=32, base=3000.0, scale=None, ff=40, kv_from=None):
    e = full(heads, dim, rot, vdim, q_rank, kv_rank, base, scale, ff, kv_from)
    e["mixer"]["mask"] = dict(size=size)
    return dict(e, type="latent_attention_2")


def gla(heads=4, dim=16, vdim=24, tau=8.0, ff=40):
    return dict(type="gla", mlp=_mlp(ff), mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=tau))


def config(layers, width=64, vocab=96, eps=1e-5, logit_scale=1.5):
    return dict(architecture="Daronex", vocab=vocab, width=width, norm=dict(eps=eps), logit_scale=logit_scale, layers=layers)


CONFIGS = dict(
    base=config([full(), gla(), win(), full(kv_from=0, heads=2, vdim=24), gla(ff=0), win(ff=0, heads=8)]),
    # nothing a multiple of anything, one head, decays of every strength
    odd=config([gla(3, 9, 7, 1.0, 37), win(7, 3, 11, 6, 13, 21, 19, ff=0), full(1, 5, 2, 3, 7, 10, ff=11), gla(1, 21, 13, 3.0, 0),
                full(5, 10, 2, 6, 9, 10, kv_from=2)], width=45, vocab=71, logit_scale=0.3),
    # more heads than a tile of 16, a latent and heads that the prompt tiles do not take, a state too wide for chunks
    wide=config([full(20, 144, 56, 24, 40, 200, ff=56), gla(2, 264, 40, 16.0), win(4000, 17, 24, 8, 136, 33, 136),
                 full(18, 8, 56, 16, 40, 200, kv_from=0)], width=72, vocab=128),
    # the widths the tiled kernels are made for
    real=config([win(150, 8, 128, 64, 128, 96, 512, ff=192), gla(2, 128, 128, 16.0), full(4, 64, 32, 64, 64, 256, ff=128),
                 gla(3, 64, 192, 8.0), full(2, 96, 32, 96, 72, 256, kv_from=2), gla(1, 200, 72, 4.0)], width=128, vocab=160),
    # a latent wider than the tensor-pipe decoding takes, more than one pass of its columns
    deep=config([full(5, 16, 8, 24, 40, 1064), gla(3, 20, 28), full(2, 192, 8, 8, 16, 1064, kv_from=0)], vocab=88),
    narrow=config([gla(2, 48, 32, 5.0, 64), full(2, 8, 56, 32, 16, 64), win(33, 6, 40, 8, 48, 24, 120)], width=96, vocab=64),
)


class Weights:
    """Random bf16-exact weights; `edit` may change the f32 dict before it is rounded."""

    def __init__(self, cfg, seed, edit=None, rank=6):
        rng = np.random.default_rng(seed)
        self.w = {}
        for n, s in tensor_shapes(cfg, rank).items():
            a = rng.standard_normal(s).astype(np.float32)
            if n.endswith(("norm1", "norm2")) or n == "final.norm":
                a = 0.3 * a
            elif n.endswith("norm"):
                a = 1.0 + 0.3 * a
            elif n.endswith("a2.b"):
                a = 2.0 + 1.5 * a
            elif n == "head":
                a = a * s[1] ** -0.5
            elif len(s) == 2 and n != "embed":
                a = a * s[1] ** -0.5
            self.w[n] = a
        if edit:
            edit(self.w)
        self.w = {n: bf16_to_f32(f32_to_bf16(a)) for n, a in self.w.items()}

    def f32(self, n):
        return self.w[n]

    def raw(self, n):
        return f32_to_bf16(self.w[n])

    def shape(self, n):
        return self.w[n].shape

    def names(self):
        return list(self.w)

    def f64(self):
        return {n: a.astype(np.float64) for n, a in self.w.items()}


def same_sign(cfg):
    """Edit of Weights: queries of the gated linear layers lean on their keys, so that the product of a token's
    own query and key does not come out of a cancellation (which the norm behind it would blow up)."""
    def edit(w):
        for i, L in enumerate(cfg["layers"]):
            if L["type"] == "gla":
                p = f"l{i}.mix."
                w[p + "q"] = 0.6 * w[p + "q"] + 0.8 * w[p + "k"]
    return edit


# ---- a key that stands out: token A asks for token B through channels of its own -----------------
A_TOK, B_TOK = 1, 2


def plant(cfg, layer=0, score=25.0):
    """Edit of Weights: in every head of the first layer, a latent attention, the query of token A scores
    about `score` on the key of token B, and that channel is zero for every other pair of tokens."""
    m = cfg["layers"][layer]["mixer"]
    p, D, R = f"l{layer}.mix.", m["dim"], m["rot_dim"]
    assert layer == 0

    def edit(w):
        w["embed"][:, :2] = 0
        w["embed"][A_TOK, 0] = w["embed"][B_TOK, 1] = 8.0
        for lat, ch in (("dq", 0), ("dkv", 1)):
            w[p + lat][0] = 0
            w[p + lat][0, ch] = 1.0
            w[p + lat + ".norm"][0] = 1.0
        # the channel of a latent whose other entries are near one in size: about 8 over the root mean square
        big = [8.0 / np.sqrt((64.0 + n - 1) / n) for n in (m["q_rank"], m["kv_rank"])]
        for h in range(m["heads"]):
            for name, row in (("uq", h * (D + R)), ("uk", h * D)):
                w[p + name][row] = 0
                w[p + name][row, 0] = np.sqrt(score / m["scale"] / (big[0] * big[1]))
    return edit


def planted_tokens(cfg, n, pairs, seed=0):
    """Random tokens without A and B, then B at j and A at i for each (j, i)."""
    t = [x if x > 2 else x + 3 for x in tokens(cfg, n, seed)]
    for j, i in pairs:
        t[j], t[i] = B_TOK, A_TOK
    return t


def planted_case():
    """A configuration and sequences (tokens, place of the query) with one asked-for key each: name -> ..."""
    cfg = config([win(20), gla()])
    pairs = dict(inside=(50, 69), outside=(71, 91), near=(100, 103))
    return cfg, {k: (planted_tokens(cfg, 130, [p]), p[1]) for k, p in pairs.items()}
