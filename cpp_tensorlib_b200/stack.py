"""Host side of the layer-stack decoder (``tlb_stack_*`` in include/tlb200.h): layer descriptions,
and the fused, padded matrices the native side reads.

A model describes each layer as a list of mixers (dicts with the fields of ``tlb_mixer_cfg``) and an
optional feed-forward, and hands the parts of every fused matrix over by name of the part; this
module knows the order and the padding.
"""
import ctypes as C

import numpy as np

from ._lib import check, lib
from .safetensors import bf16_to_f32, f32_to_bf16
from .sequence import Sequence

ATTN, DELTA, SSD, LATENT, GLA = 1, 2, 3, 4, 5
CLIPPED_GLU, SQUARED_RELU = 0, 1
MATRIX = dict(input=0, output=1, gate_up=2, down=3, embed=4, head=5, q_up=16, kv_up=24)
VECTOR = dict(norm1=0, norm2=1, final=2, q_norm=10, k_norm=11, norm=12, conv=13, conv_bias=14, dt_bias=15, A_log=16,
              skip=17, decay_up=18, decay_bias=19)


class MixerCfg(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("kind", "heads", "kv_heads", "dim", "vdim", "window", "keep_first",
                                         "rot_dims", "conv", "norm_groups", "q_rank", "kv_rank", "gate", "kv_from",
                                         "rank")] + \
               [(n, C.c_float) for n in ("rot_base", "scale", "out_scale", "tau")]


class LayerCfg(C.Structure):
    _fields_ = [("n_mixers", C.c_int32), ("ff", C.c_int32), ("act", C.c_int32), ("limit", C.c_float), ("mixer", MixerCfg * 2)]


class StackCfg(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("width", "vocab", "n_layers", "max_ctx", "f32", "post_norm")] + \
               [(n, C.c_float) for n in ("eps", "embed_scale", "logit_scale")]


def pad8(n):
    return (n + 7) // 8 * 8


def pad_rows(a, n=None):
    """`a` with zero rows behind it, up to a multiple of 8."""
    n = pad8(a.shape[0]) if n is None else n
    return a if a.shape[0] == n else np.concatenate([a, np.zeros((n - a.shape[0],) + a.shape[1:], a.dtype)])


def pad_cols(a):
    return np.ascontiguousarray(pad_rows(np.ascontiguousarray(a.T)).T)


def head_rows(a, heads, width=None):
    """Rows laid out head by head, each head padded with zero rows to `width` (default: a multiple of 8)."""
    h = np.ascontiguousarray(a).reshape(heads, -1, a.shape[-1])
    out = np.zeros((heads, pad8(h.shape[1]) if width is None else width, a.shape[-1]), a.dtype)
    out[:, :h.shape[1]] = h
    return out


def paired_rows(a):
    """Rows of the rotate-half layout (i pairs with i + n/2) in the order that puts a pair side by side; the
    last two axes are rows and columns."""
    n = a.shape[-2] // 2
    return np.stack([a[..., :n, :], a[..., n:, :]], axis=-2).reshape(a.shape)


def mixer_cfg(kind, heads, kv_heads, dim, vdim, out_scale=1.0, **more):
    return MixerCfg(kind=kind, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, out_scale=out_scale, **more)


class LayerStack(Sequence):
    """layers: list of dicts ``mixers`` (list of MixerCfg), ``ff``, ``act`` and ``limit``.  post_norm: the
    norms of a layer are behind its sublayers instead of in front of them."""

    def __init__(self, width, vocab, eps, embed_scale, layers, dtype, max_ctx, post_norm=False, logit_scale=1.0):
        super().__init__(vocab, max_ctx)
        self.f32 = dtype == "float32"
        cfg = StackCfg(width, vocab, len(layers), max_ctx, int(self.f32), int(post_norm), eps, embed_scale, logit_scale)
        arr = (LayerCfg * len(layers))()
        for a, L in zip(arr, layers):
            a.n_mixers, a.ff, a.limit = len(L["mixers"]), L.get("ff", 0), L.get("limit", 0.0)
            a.act = L.get("act", CLIPPED_GLU)
            for i, m in enumerate(L["mixers"]):
                a.mixer[i] = m
        check(lib().tlb_stack_create(C.byref(cfg), arr, C.byref(self.h)))

    def weight(self, a):
        """A matrix (f32, or raw bf16 as uint16) in the model's own type."""
        if self.f32:
            return bf16_to_f32(a) if a.dtype == np.uint16 else np.asarray(a, np.float32)
        return np.asarray(a) if a.dtype == np.uint16 else f32_to_bf16(a)

    def set_matrix(self, layer, name, a, mixer=0):
        a = np.ascontiguousarray(self.weight(a))
        check(lib().tlb_stack_set_matrix(self.h, layer, MATRIX[name] + mixer, a.ctypes.data, a.shape[0], a.shape[1]))

    def set_vector(self, layer, name, v, mixer=0):
        v = np.ascontiguousarray(v, np.float32).reshape(-1)
        check(lib().tlb_stack_set_vector(self.h, layer, mixer, VECTOR[name], v.ctypes.data, v.size))

    def set_input(self, layer, parts):
        """Input projections of all mixers of a layer, in the order of the projected row."""
        self.set_matrix(layer, "input", np.concatenate([pad_rows(self.weight(p)) for p in parts]))

    def set_output(self, layer, parts):
        self.set_matrix(layer, "output", np.concatenate([pad_cols(self.weight(p)) for p in parts], axis=1))

    def set_gate_up(self, layer, gate, up):
        a = np.stack([self.weight(gate), self.weight(up)], axis=1)
        self.set_matrix(layer, "gate_up", a.reshape(-1, a.shape[-1]))

    def set_latent(self, layer, heads, q_up, k_up, v_up, rot_dims, half=False, mixer=0):
        """The products behind the latents: queries [heads * (dim + rot_dims), q_rank], keys [heads * dim,
        kv_rank], values [heads * vdim, kv_rank].  half: rotated rows come in the rotate-half layout (the
        latent's own rotated rows, in the input projection, are the caller's to pair)."""
        q, k, v = (self.weight(a) for a in (q_up, k_up, v_up))
        q = q.reshape(heads, -1, q.shape[-1])
        dim = q.shape[1] - rot_dims
        rot = paired_rows(q[:, dim:]) if half else q[:, dim:]
        parts = [head_rows(p, heads) for p in (q[:, :dim].reshape(heads * dim, -1), rot.reshape(heads * rot_dims, -1)) if p.size]
        self.set_matrix(layer, "q_up", np.concatenate(parts, axis=1).reshape(-1, q.shape[-1]), mixer)
        self.set_matrix(layer, "kv_up", np.concatenate([head_rows(p, heads).reshape(-1, p.shape[-1]) for p in (k, v)]), mixer)

    def state_bytes(self):
        return int(lib().tlb_stack_state_bytes(self.h))
