"""Zavilorn: a decoder-only stack of 'parallel' layers (sliding-window attention beside a gated delta
rule) and 'mamba2' layers, each with an optional clipped gated feed-forward, tied embeddings.

This module reads config.json and names the tensors; the layers themselves are the layer stack's
mixers.  Every size and constant comes from the configuration.
"""
import numpy as np

from .safetensors import bf16_to_f32, f32_to_bf16
from .stack import ATTN, DELTA, SSD, LayerStack, mixer_cfg, pad_rows


def layer_spec(entry):
    """One entry of config 'layers' as the layer stack's description."""
    m = entry["mixer"]
    if entry["type"] == "parallel":
        a, d = m["left"], m["right"]
        mixers = [
            mixer_cfg(ATTN, a["heads"], a["kv_heads"], a["dim"], a["vdim"], m["left_scale"], window=a["mask"]["size"],
                      keep_first=a["mask"]["keep_first"], rot_dims=a["rot"]["dims"], rot_base=a["rot"]["base"],
                      scale=a["scale"]),
            mixer_cfg(DELTA, d["heads"], d["kv_heads"], d["dim"], d["vdim"], m["right_scale"], conv=d["conv"]),
        ]
    elif entry["type"] == "mamba2":
        mixers = [mixer_cfg(SSD, m["heads"], m["groups"], m["state"], m["vdim"], conv=m["conv"],
                            norm_groups=m["norm_groups"])]
    else:
        raise ValueError(f"unknown layer type {entry['type']!r}")
    spec = dict(mixers=mixers, ff=0)
    mlp = entry.get("mlp")
    if mlp:
        if mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
        spec.update(ff=mlp["ff"], limit=mlp["limit"])
    return spec


class Zavilorn(LayerStack):
    def __init__(self, config, dtype="bfloat16", max_ctx=4096):
        self.config = config
        super().__init__(config["width"], config["vocab"], config["norm"]["eps"], config["embedding"]["scale"],
                         [layer_spec(e) for e in config["layers"]], dtype, max_ctx)

    @classmethod
    def from_folder(cls, config, tensors, dtype, max_ctx):
        d = cls(config, dtype, max_ctx)
        d.load(tensors)
        return d

    def load(self, t):
        """t: a SafeTensors, or anything with its raw() and f32()."""
        self.set_matrix(0, "embed", t.raw("embed"))
        self.set_vector(0, "final", t.f32("final.norm"))
        for i, entry in enumerate(self.config["layers"]):
            p, m = f"l{i}.", entry["mixer"]
            self.set_vector(i, "norm1", t.f32(p + "norm1"))
            if entry["type"] == "parallel":
                self._load_parallel(i, p + "mix.", t)
            else:
                self._load_mamba2(i, p + "mix.", m, t)
            if entry.get("mlp"):
                self.set_vector(i, "norm2", t.f32(p + "norm2"))
                self.set_gate_up(i, t.raw(p + "mlp.gate"), t.raw(p + "mlp.up"))
                self.set_matrix(i, "down", t.raw(p + "mlp.down"))

    def _load_parallel(self, i, p, t):
        l, r = p + "left.", p + "right."
        self.set_input(i, [t.raw(l + n) for n in ("q", "k", "v", "g")] +
                       [t.raw(r + n) for n in ("q", "k", "v", "g", "b", "a")])
        self.set_output(i, [t.raw(l + "o"), t.raw(r + "o")])
        self.set_vector(i, "q_norm", t.f32(l + "q.norm"), 0)
        self.set_vector(i, "k_norm", t.f32(l + "k.norm"), 0)
        self.set_vector(i, "conv", np.concatenate([pad_rows(t.f32(r + n + ".conv")) for n in "qkv"]), 1)
        self.set_vector(i, "norm", t.f32(r + "norm"), 1)
        self.set_vector(i, "dt_bias", t.f32(r + "dt_bias"), 1)
        self.set_vector(i, "A_log", t.f32(r + "A_log"), 1)

    def _load_mamba2(self, i, p, m, t):
        inner = m["heads"] * m["vdim"]
        xbc = inner + 2 * m["groups"] * m["state"]
        w = t.raw(p + "in")
        self.set_input(i, [w[:inner], w[inner:inner + xbc], w[inner + xbc:]])
        self.set_output(i, [t.raw(p + "o")])
        self.set_vector(i, "conv", pad_rows(t.f32(p + "conv")))
        self.set_vector(i, "conv_bias", pad_rows(t.f32(p + "conv.b")))
        for name, key in (("dt_bias", "dt_bias"), ("A_log", "A_log"), ("skip", "D"), ("norm", "norm")):
            self.set_vector(i, name, t.f32(p + key))


def tensor_shapes(config):
    """name -> shape of every tensor of a model with this configuration."""
    w, out = config["width"], {"embed": (config["vocab"], config["width"]), "final.norm": (config["width"],)}
    for i, entry in enumerate(config["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        out[p + "norm1"] = (w,)
        if entry["type"] == "parallel":
            a, d, l, r = m["left"], m["right"], p + "mix.left.", p + "mix.right."
            q, k = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            v, o = a["kv_heads"] * a["vdim"], a["heads"] * a["vdim"]
            out.update({l + "q": (q, w), l + "k": (k, w), l + "v": (v, w), l + "g": (o, w), l + "o": (w, o),
                        l + "q.norm": (q,), l + "k.norm": (k,)})
            q, o, h = d["kv_heads"] * d["dim"], d["heads"] * d["vdim"], d["heads"]
            for n, rows in (("q", q), ("k", q), ("v", o)):
                out.update({r + n: (rows, w), r + n + ".conv": (rows, d["conv"])})
            out.update({r + "b": (h, w), r + "a": (h, w), r + "A_log": (h,), r + "dt_bias": (h,),
                        r + "norm": (d["vdim"],), r + "g": (o, w), r + "o": (w, o)})
        else:
            h, inner = m["heads"], m["heads"] * m["vdim"]
            c = inner + 2 * m["groups"] * m["state"]
            p2 = p + "mix."
            out.update({p2 + "in": (inner + c + h, w), p2 + "conv": (c, m["conv"]), p2 + "conv.b": (c,),
                        p2 + "dt_bias": (h,), p2 + "A_log": (h,), p2 + "D": (h,), p2 + "norm": (inner,),
                        p2 + "o": (w, inner)})
        if entry.get("mlp"):
            f = entry["mlp"]["ff"]
            out.update({p + "norm2": (w,), p + "mlp.gate": (f, w), p + "mlp.up": (f, w), p + "mlp.down": (w, f)})
    return out


class RandomTensors:
    """Random weights of a configuration, slices of one pool of normal numbers (raw() and f32() of a
    SafeTensors).  Matrices have standard deviation 1 / sqrt(columns), norms are near one, decay rates
    and step biases lie where the recurrences remember tens to hundreds of tokens."""

    def __init__(self, config, seed=0, pool=1 << 24, shapes=None):
        self.shapes = shapes or tensor_shapes(config)
        self.rng = np.random.default_rng(seed)
        self.pool = self.rng.standard_normal(pool, dtype=np.float32)

    def __contains__(self, name):
        return name in self.shapes

    def names(self):
        return list(self.shapes)

    def f32(self, name):
        shape = self.shapes[name]
        n = int(np.prod(shape))
        at = int(self.rng.integers(len(self.pool)))
        a = np.resize(np.roll(self.pool, -at) if n > len(self.pool) - at else self.pool[at:at + n], shape)
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            a = 1.0 + 0.1 * a
        elif name.endswith("A_log"):
            a = 0.3 * a
        elif name.endswith("dt_bias"):
            a = -3.0 + 0.5 * a
        elif len(shape) == 2 and name != "embed":
            a = a / np.float32(np.sqrt(shape[1]))
        return bf16_to_f32(f32_to_bf16(a)).reshape(shape)

    def raw(self, name):
        return f32_to_bf16(self.f32(name))
