"""Plain, slow restatement of the Zavilorn decoder in numpy (TEST INFRASTRUCTURE ONLY).

One function per mechanism, token by token where the mechanism is a recurrence, every size and
constant an argument.  Nothing here is shared with the product path.  `F` is the working type:
float64 for a reference, float32 to see what rounding alone does.
"""
import numpy as np


def sigmoid(z):
    with np.errstate(over="ignore"):
        return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0) + np.log1p(np.exp(-np.abs(z)))


def rms_norm(x, w, eps, parts=1):
    """Each of `parts` equal slices of the last axis divided by its own root mean square, times w."""
    s = x.reshape(x.shape[:-1] + (parts, x.shape[-1] // parts))
    s = s / np.sqrt(np.mean(s * s, axis=-1, keepdims=True) + s.dtype.type(eps))
    return s.reshape(x.shape) * w


def rotate(x, pos, dims, base):
    """Interleaved rotary: x [T, heads, D]; dimension 2i pairs with 2i+1, the first `dims` only."""
    F = x.dtype.type
    out = x.copy()
    i = np.arange(dims // 2)
    f = (float(base) ** (-2.0 * i / dims)).astype(x.dtype)
    a = pos.astype(x.dtype)[:, None] * f[None]
    c, s = np.cos(a)[:, None].astype(F), np.sin(a)[:, None].astype(F)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def sees(i, j, window, keep):
    """Whether the query at position i sees the key at position j."""
    return j <= i and (i - j < window or j < keep)


def window_attention(q, k, v, scale, window, keep):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]; softmax over the visible keys."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    pj = np.arange(T)
    for i in range(T):
        vis = np.nonzero((pj <= i) & ((i - pj < window) | (pj < keep)))[0]
        for h in range(H):
            g = h // (H // G)
            s = (k[vis, g] @ q[i, h]) * q.dtype.type(scale)
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[vis, g]
    return out


def causal_conv(x, w, b=None):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start; then silu."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x)
    for t in range(T):
        for a in range(taps):
            if t - (taps - 1 - a) >= 0:
                y[t] += w[:, a] * x[t - (taps - 1 - a)]
    return silu(y if b is None else y + b)


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + x.dtype.type(1e-6))


def delta_rule(q, k, v, beta, g):
    """Gated delta rule: q, k [T, G, D], v [T, H, E], beta, g [T, H] -> [T, H, E]."""
    T, H, E = v.shape
    G, D = k.shape[1:]
    S = np.zeros((H, D, E), v.dtype)
    out = np.zeros_like(v)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // (H // G)], q[t, h // (H // G)]
            S[h] *= g[t, h]
            u = beta[t, h] * (v[t, h] - S[h].T @ kk)
            S[h] += np.outer(kk, u)
            out[t, h] = S[h].T @ qq
    return out


def ssd(x, B, C, dt, A, D):
    """Mamba-2: x [T, H, E], B, C [T, G, N], dt [T, H], A [H] (positive rate), D [H] -> [T, H, E]."""
    T, H, E = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, E), x.dtype)
    out = np.zeros_like(x)
    for t in range(T):
        for h in range(H):
            bb, cc = B[t, h // (H // G)], C[t, h // (H // G)]
            S[h] = np.exp(-A[h] * dt[t, h]) * S[h] + dt[t, h] * np.outer(bb, x[t, h])
            out[t, h] = S[h].T @ cc + D[h] * x[t, h]
    return out


def clipped_glu(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(gate.dtype.type(1.702) * g) * (u + 1)


# ---- layers -------------------------------------------------------------------------------

def attention_mixer(h, W, p, c, eps, pos0=0):
    T = h.shape[0]
    H, G, D, E = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    pos = np.arange(pos0, pos0 + T)
    q = rms_norm(h @ W[p + "q"].T, W[p + "q.norm"], eps).reshape(T, H, D)
    k = rms_norm(h @ W[p + "k"].T, W[p + "k.norm"], eps).reshape(T, G, D)
    v = (h @ W[p + "v"].T).reshape(T, G, E)
    q, k = (rotate(a, pos, c["rot"]["dims"], c["rot"]["base"]) for a in (q, k))
    o = window_attention(q, k, v, c["scale"], c["mask"]["size"], c["mask"]["keep_first"])
    return (o.reshape(T, H * E) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def delta_mixer(h, W, p, c, eps):
    T = h.shape[0]
    H, G, D, E = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (causal_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q, k = unit(q.reshape(T, G, D)), unit(k.reshape(T, G, D))
    q = q * h.dtype.type(D ** -0.5)
    beta = sigmoid(h @ W[p + "b"].T)
    g = np.exp(-np.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    o = delta_rule(q, k, v.reshape(T, H, E), beta, g)
    o = rms_norm(o, W[p + "norm"], eps) * silu(h @ W[p + "g"].T).reshape(T, H, E)
    return o.reshape(T, H * E) @ W[p + "o"].T


def mamba2_mixer(h, W, p, c, eps):
    T = h.shape[0]
    H, E, N, G = c["heads"], c["vdim"], c["state"], c["groups"]
    inner = H * E
    zxbcdt = h @ W[p + "in"].T
    z, xbc, dt = np.split(zxbcdt, [inner, 2 * inner + 2 * G * N], axis=1)
    x, B, C = np.split(causal_conv(xbc, W[p + "conv"], W[p + "conv.b"]), [inner, inner + G * N], axis=1)
    dt = softplus(dt + W[p + "dt_bias"])
    y = ssd(x.reshape(T, H, E), B.reshape(T, G, N), C.reshape(T, G, N), dt, np.exp(W[p + "A_log"]), W[p + "D"])
    y = rms_norm(y.reshape(T, inner) * silu(z), W[p + "norm"], eps, c["norm_groups"])
    return y @ W[p + "o"].T


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; `layers_out` (a list) receives the residual per layer."""
    F = W["embed"].dtype
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * F.type(cfg["embedding"]["scale"])
    for i, L in enumerate(cfg["layers"]):
        p, c = "l%d." % i, L["mixer"]
        h = rms_norm(x, W[p + "norm1"], eps)
        if L["type"] == "parallel":
            x = x + (F.type(c["left_scale"]) * attention_mixer(h, W, p + "mix.left.", c["left"], eps) +
                     F.type(c["right_scale"]) * delta_mixer(h, W, p + "mix.right.", c["right"], eps))
        elif L["type"] == "mamba2":
            x = x + mamba2_mixer(h, W, p + "mix.", c, eps)
        else:
            raise KeyError(L["type"])
        m = L.get("mlp")
        if m:
            h = rms_norm(x, W[p + "norm2"], eps)
            x = x + clipped_glu(h @ W[p + "mlp.gate"].T, h @ W[p + "mlp.up"].T, F.type(m["limit"])) @ W[p + "mlp.down"].T
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["embed"].T
