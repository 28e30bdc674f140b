"""Zavilorn: a decoder-only stack of 'parallel' layers (sliding-window attention beside a gated delta
rule) and 'mamba2' layers, each with an optional clipped gated feed-forward, tied embeddings.

This module reads config.json and names the tensors; the layers themselves are the layer stack's
mixers.  Every size and constant comes from the configuration.
"""
import numpy as np

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
