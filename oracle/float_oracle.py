"""Plain, slow restatement of the floating-point decoder designs: numpy in float64, one function per
mechanism, one sequence at a time, no cache.  Test infrastructure; it shares no code with the product path.

`rnd` is applied to every activation that a reduced-precision run stores between its products (identity by default):
with a rounding function the result shows the error that rounding alone causes.

A sequence is an array of token ids; activations are [tokens, width].  `W` maps tensor names to arrays and
`cfg` is the parsed configuration.  Linear weights are [out, in].
"""
import numpy as np


def exact(x):
    return x


def rms_norm(x, w, eps):
    """y_n = x_n / sqrt(mean_m x_m^2 + eps) * w_n over the last dimension"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rotate_pairs(x, positions, base):
    """x [tokens, ..., R]: the pair (x_2i, x_2i+1) of the token at position p turns by p * base^(-2i / R)"""
    R = x.shape[-1]
    out = np.empty_like(x)
    for i in range(R // 2):
        a = positions * float(base) ** (-2.0 * i / R)
        a = a.reshape((-1,) + (1,) * (x.ndim - 2))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def window_mask(n, size):
    """[n, n] booleans: query i sees key j when 0 <= i - j < size"""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (i - j >= 0) & (i - j < size)


def softmax_rows(s, visible):
    s = np.where(visible, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_kv(h, W, p, mx, eps, rnd=exact):
    """the two cached parts of every token: the normed latent [T, C] and the rotated shared key part [T, R]"""
    y = h @ W[p + "dkv"].T
    C = mx["kv_rank"]
    c = rms_norm(y[:, :C], W[p + "dkv.norm"], eps)
    return rnd(c), rnd(rotate_pairs(y[:, C:], np.arange(len(h), dtype=np.float64), mx["rot"]["base"]))


def latent_queries(h, W, p, mx, eps, rnd=exact):
    """per head the unrotated [T, H, D] and the rotated [T, H, R] query"""
    H, D, R = mx["heads"], mx["dim"], mx["rot_dim"]
    cq = rnd(rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps))
    q = (cq @ W[p + "uq"].T).reshape(len(h), H, D + R)
    turned = rotate_pairs(q[:, :, D:], np.arange(len(h), dtype=np.float64), mx["rot"]["base"])
    return rnd(q[:, :, :D]), rnd(turned)


def latent_attention(h, c, kr, W, p, mx, eps, rnd=exact):
    """windowed softmax attention over per-head keys [W_uk c, k_rot] and values W_uv c, gated and projected"""
    T, H, D, V = len(h), mx["heads"], mx["dim"], mx["vdim"]
    qn, qr = latent_queries(h, W, p, mx, eps, rnd)
    kn = rnd(c @ W[p + "uk"].T).reshape(T, H, D)
    v = rnd(c @ W[p + "uv"].T).reshape(T, H, V)
    seen = window_mask(T, mx["mask"]["size"])
    o = np.empty((T, H, V))
    for j in range(H):
        s = (qn[:, j] @ kn[:, j].T + qr[:, j] @ kr.T) * mx["scale"]
        o[:, j] = rnd(rnd(softmax_rows(s, seen)) @ v[:, j])
    gate = sigmoid(h @ W[p + "g"].T)
    return rnd(o.reshape(T, H * V) * gate) @ W[p + "o"].T


def dense_ff(h, W, p, rnd=exact):
    return rnd(silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def forward(cfg, W, tokens, layers_out=None, rnd=exact):
    """logits [T, vocab] of every position of one sequence; layers_out receives x after each layer"""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)].astype(np.float64)
    held = {}
    for i, L in enumerate(cfg["layers"]):
        p, mx = "l%d." % i, L["mixer"]
        src = mx.get("kv_from")
        h = rnd(x)
        held[i] = latent_kv(h, W, p + "mix.", mx, eps, rnd) if src is None else held[src]
        y = latent_attention(h, held[i][0], held[i][1], W, p + "mix.", mx, eps, rnd)
        x = x + rms_norm(y, W[p + "norm1"], eps)
        if L.get("mlp") is not None:
            x = x + rms_norm(dense_ff(rnd(x), W, p + "mlp.", rnd), W[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rnd(rms_norm(x, W["final.norm"], eps)) @ W["embed"].T
