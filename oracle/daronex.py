"""Plain, slow restatement of the Daronex decoder in numpy (TEST INFRASTRUCTURE ONLY).

One function per mechanism, keys and values of every head written out, the recurrence token by token,
every size and constant an argument.  Nothing here is shared with the product path.  The working type is
the weights': float64 for a reference, float32 to see what rounding alone does.
"""
import numpy as np


def sigmoid(z):
    with np.errstate(over="ignore"):
        return 1.0 / (1.0 + np.exp(-z))


def rms_norm(x, w, eps):
    """The last axis over its root mean square, times w."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps)) * w


def rotate(x, pos, base, half):
    """x [T, heads, R], all of it rotated.  Pairs (2i, 2i + 1), or with `half` (i, i + R / 2)."""
    R = x.shape[-1]
    n = R // 2
    a = pos[:, None].astype(np.float64) * float(base) ** (-2.0 * np.arange(n) / R)
    c, s = (f(a)[:, None].astype(x.dtype) for f in (np.cos, np.sin))
    first, second = (slice(0, n), slice(n, R)) if half else (slice(0, R, 2), slice(1, R, 2))
    out = np.empty_like(x)
    out[..., first] = x[..., first] * c - x[..., second] * s
    out[..., second] = x[..., second] * c + x[..., first] * s
    return out


def sees(i, j, window):
    """Whether position i sees j; window None: everything before it."""
    return j <= i and (window is None or i - j < window)


def attend(q, k, v, scale, window):
    """q, k [T, H, D], v [T, H, E] -> [T, H, E]; softmax over the visible keys."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    for i in range(T):
        lo = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            s = (k[lo:i + 1, h] @ q[i, h]) * q.dtype.type(scale)
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, h]
    return out


def latent_of(h, W, p, c, eps, half):
    """What a token leaves behind: the normed latent [T, kv_rank] and the rotated shared key part [T, rot_dim]."""
    t = h @ W[p + "dkv"].T
    C = c["kv_rank"]
    r = rotate(t[:, None, C:], np.arange(len(h)), c["rot"]["base"], half)[:, 0]
    return rms_norm(t[:, :C], W[p + "dkv.norm"], eps), r


def latent_attention(h, W, p, c, eps, half, window, kept):
    """kept: (latent, rotated key part) of this layer or of the one it shares with."""
    T, H, D, R, E = len(h), c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    lat, kr = kept
    q = (rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).reshape(T, H, D + R)
    q = np.concatenate([q[..., :D], rotate(q[..., D:], np.arange(T), c["rot"]["base"], half)], -1)
    k = np.concatenate([(lat @ W[p + "uk"].T).reshape(T, H, D), np.repeat(kr[:, None], H, 1)], -1)
    v = (lat @ W[p + "uv"].T).reshape(T, H, E)
    o = attend(q, k, v, c["scale"], window).reshape(T, H * E)
    if p + "g" in W:
        o = o * sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def decay(z, tau):
    """sigmoid(z) ** (1 / tau)"""
    return np.exp((np.minimum(z, 0) - np.log1p(np.exp(-np.abs(z)))) / z.dtype.type(tau))


def gated_linear(q, k, v, alpha):
    """q, k, alpha [T, H, D], v [T, H, E] -> [T, H, E]: a state of D x E per head, rows decaying by alpha."""
    T, H, D = k.shape
    S = np.zeros((H, D, v.shape[2]), v.dtype)
    out = np.zeros_like(v)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", S, q[t])
    return out


def gla_mixer(h, W, p, c, eps):
    T, H, D, E = len(h), c["heads"], c["dim"], c["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, D) * h.dtype.type(D ** -0.5)
    k = (h @ W[p + "k"].T).reshape(T, H, D)
    v = (h @ W[p + "v"].T).reshape(T, H, E)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    o = rms_norm(gated_linear(q, k, v, decay(z, c["tau"]).reshape(T, H, D)), W[p + "norm"], eps)
    g = h @ W[p + "g"].T
    return (o.reshape(T, H * E) * (g * sigmoid(g))) @ W[p + "o"].T


def squared_relu_ff(h, up, down):
    return np.maximum(h @ up.T, 0) ** 2 @ down.T


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; `layers_out` (a list) receives the residual per layer."""
    F, eps = W["embed"].dtype, cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p, c = "l%d." % i, L["mixer"]
        if L["type"] == "gla":
            y = gla_mixer(x, W, p + "mix.", c, eps)
        else:
            half = {"latent_attention": False, "latent_attention_2": True}[L["type"]]
            j = c.get("kv_from")
            if j is None:
                j = i
                kept[i] = latent_of(x, W, p + "mix.", c, eps, half)
            y = latent_attention(x, W, p + "mix.", c, eps, half, c["mask"]["size"] if half else None, kept[j])
        x = x + rms_norm(y, 1 + W[p + "norm1"], eps)
        if L.get("mlp"):
            y = squared_relu_ff(x, W[p + "mlp.up"], W[p + "mlp.down"])
            x = x + rms_norm(y, 1 + W[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, 1 + W["final.norm"], eps) @ W["head"].T * F.type(cfg["logit_scale"])
