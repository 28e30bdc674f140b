"""Daronex: a decoder-only stack of latent attentions (whole context, some of them on the latent of an
earlier layer; or a sliding window with an output gate) and gated linear attentions, norms behind the
sublayers, feed-forwards with a squared relu, an output head of its own.

This module reads config.json and names the tensors; the layers themselves are the layer stack's
mixers.  Every size and constant comes from the configuration or from a tensor's shape.
"""
import numpy as np

from .stack import GLA, LATENT, SQUARED_RELU, LayerStack, mixer_cfg, paired_rows
from .zavilorn import RandomTensors as _RandomTensors

FULL, WINDOW = "latent_attention", "latent_attention_2"


def layer_spec(entry, decay_rank=0):
    """One entry of config 'layers' as the layer stack's description; decay_rank: columns of a gla layer's
    second decay projection."""
    m, kind = entry["mixer"], entry["type"]
    if kind in (FULL, WINDOW):
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError("the rotated part of a latent attention is rotated as a whole")
        src = m.get("kv_from")
        mixer = mixer_cfg(LATENT, m["heads"], m["heads"], m["dim"], m["vdim"], q_rank=m["q_rank"], kv_rank=m["kv_rank"],
                          rot_dims=m["rot_dim"], rot_base=m["rot"]["base"], scale=m["scale"],
                          window=m["mask"]["size"] if kind == WINDOW else 0, gate=int(kind == WINDOW),
                          kv_from=-1 if src is None else src)
    elif kind == "gla":
        mixer = mixer_cfg(GLA, m["heads"], m["heads"], m["dim"], m["vdim"], tau=m["tau"], rank=decay_rank)
    else:
        raise ValueError(f"unknown layer type {kind!r}")
    spec = dict(mixers=[mixer], ff=0)
    mlp = entry.get("mlp")
    if mlp:
        if mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
        spec.update(ff=mlp["ff"], act=SQUARED_RELU)
    return spec


class Daronex(LayerStack):
    def __init__(self, config, decay_ranks, dtype="bfloat16", max_ctx=4096):
        """decay_ranks: layer -> width between a gla layer's two decay projections (only the weights say)."""
        self.config = config
        super().__init__(config["width"], config["vocab"], config["norm"]["eps"], 1.0,
                         [layer_spec(e, decay_ranks.get(i, 0)) for i, e in enumerate(config["layers"])], dtype, max_ctx,
                         post_norm=True, logit_scale=config["logit_scale"])

    @classmethod
    def from_folder(cls, config, tensors, dtype, max_ctx):
        ranks = {i: tensors.shape(f"l{i}.mix.a1")[0] for i, e in enumerate(config["layers"]) if e["type"] == "gla"}
        d = cls(config, ranks, dtype, max_ctx)
        d.load(tensors)
        return d

    def load(self, t):
        """t: a SafeTensors, or anything with its raw() and f32()."""
        self.set_matrix(0, "embed", t.raw("embed"))
        self.set_matrix(0, "head", t.raw("head"))
        self.set_vector(0, "final", 1.0 + t.f32("final.norm"))      # these norms are stored around zero
        for i, entry in enumerate(self.config["layers"]):
            p, m = f"l{i}.", entry["mixer"]
            self.set_vector(i, "norm1", 1.0 + t.f32(p + "norm1"))
            if entry["type"] == "gla":
                self._load_gla(i, p + "mix.", m, t)
            else:
                self._load_latent(i, p + "mix.", m, t, entry["type"] == WINDOW)
            if entry.get("mlp"):
                self.set_vector(i, "norm2", 1.0 + t.f32(p + "norm2"))
                self.set_matrix(i, "gate_up", t.raw(p + "mlp.up"))
                self.set_matrix(i, "down", t.raw(p + "mlp.down"))

    def _load_latent(self, i, p, m, t, window):
        """The rotate-half layout of the windowed kind becomes adjacent pairs here, in the queries' rows and
        in the shared key part's, so that one rotation serves both kinds."""
        parts = [t.raw(p + "dq")]
        if m.get("kv_from") is None:
            w, C = t.raw(p + "dkv"), m["kv_rank"]
            parts += [w[:C], paired_rows(w[C:]) if window else w[C:]]
            self.set_vector(i, "k_norm", t.f32(p + "dkv.norm"))
        if window:
            parts.append(t.raw(p + "g"))
        self.set_input(i, parts)
        self.set_output(i, [t.raw(p + "o")])
        self.set_vector(i, "q_norm", t.f32(p + "dq.norm"))
        self.set_latent(i, m["heads"], t.raw(p + "uq"), t.raw(p + "uk"), t.raw(p + "uv"), m["rot_dim"], half=window)

    def _load_gla(self, i, p, m, t):
        self.set_input(i, [t.raw(p + n) for n in ("q", "k", "v", "g", "a1")])
        self.set_output(i, [t.raw(p + "o")])
        self.set_vector(i, "norm", np.tile(t.f32(p + "norm"), m["heads"]))
        self.set_vector(i, "decay_up", t.f32(p + "a2").T)
        self.set_vector(i, "decay_bias", t.f32(p + "a2.b"))


def tensor_shapes(config, decay_rank=16):
    """name -> shape of every tensor of a model with this configuration."""
    w, v = config["width"], config["vocab"]
    out = {"embed": (v, w), "head": (v, w), "final.norm": (w,)}
    for i, entry in enumerate(config["layers"]):
        p, m = f"l{i}.mix.", entry["mixer"]
        o = m["heads"] * m["vdim"]
        out.update({f"l{i}.norm1": (w,), p + "o": (w, o)})
        if entry["type"] == "gla":
            q = m["heads"] * m["dim"]
            out.update({p + "q": (q, w), p + "k": (q, w), p + "v": (o, w), p + "g": (o, w), p + "norm": (m["vdim"],),
                        p + "a1": (decay_rank, w), p + "a2": (q, decay_rank), p + "a2.b": (q,)})
        else:
            C, R = m["kv_rank"], m["rot_dim"]
            out.update({p + "dq": (m["q_rank"], w), p + "dq.norm": (m["q_rank"],),
                        p + "uq": (m["heads"] * (m["dim"] + R), m["q_rank"]), p + "uk": (m["heads"] * m["dim"], C),
                        p + "uv": (o, C)})
            if m.get("kv_from") is None:
                out.update({p + "dkv": (C + R, w), p + "dkv.norm": (C,)})
            if entry["type"] == WINDOW:
                out[p + "g"] = (o, w)
        if entry.get("mlp"):
            f = entry["mlp"]["ff"]
            out.update({f"l{i}.norm2": (w,), f"l{i}.mlp.up": (f, w), f"l{i}.mlp.down": (w, f)})
    return out


class RandomTensors(_RandomTensors):
    """Random weights of a configuration (see zavilorn.RandomTensors).  Norms stored around zero lie there;
    decay biases lie where the recurrence remembers tens to hundreds of tokens."""

    def __init__(self, config, seed=0, decay_rank=16):
        super().__init__(config, seed, shapes=tensor_shapes(config, decay_rank))

    def f32(self, name):
        if name.endswith(("norm1", "norm2")) or name == "final.norm":
            return super().f32(name) - 1.0
        a = super().f32(name)
        return a + 3.0 if name.endswith("a2.b") else a

    def shape(self, name):
        return self.shapes[name]
