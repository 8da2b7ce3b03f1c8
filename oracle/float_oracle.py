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


# ---- windowed attention whose values are its unnormed keys ------------------------------------------------
def rotate_half(x, positions, dims, base):
    """x [tokens, ..., D]: of the first `dims` entries, (x_i, x_{i + dims/2}) of the token at position p turns by
    p * base^(-2i / dims); the rest stays"""
    out = x.copy()
    for i in range(dims // 2):
        a = (positions * float(base) ** (-2.0 * i / dims)).reshape((-1,) + (1,) * (x.ndim - 2))
        u, v = x[..., i], x[..., i + dims // 2]
        out[..., i] = u * np.cos(a) - v * np.sin(a)
        out[..., i + dims // 2] = v * np.cos(a) + u * np.sin(a)
    return out


def key_valued_attention(h, W, p, mx, eps, rnd=exact):
    """grouped heads; normed and rotated queries and keys, the projected keys themselves as values, output gate"""
    T, H, G, D = len(h), mx["heads"], mx["kv_heads"], mx["dim"]
    pos = np.arange(T, dtype=np.float64)
    q = rnd(h @ W[p + "q"].T + W[p + "q.b"]).reshape(T, H, D)
    v = rnd(h @ W[p + "k"].T + W[p + "k.b"]).reshape(T, G, D)
    turn = lambda x, w: rnd(rotate_half(rms_norm(x, W[p + w], eps), pos, mx["rot"]["dims"], mx["rot"]["base"]))
    q, k = turn(q, "q.norm"), turn(v, "k.norm")
    seen = window_mask(T, mx["mask"]["size"])
    o = np.empty((T, H, D))
    for j in range(H):
        g = j // (H // G)
        o[:, j] = rnd(softmax_rows(q[:, j] @ k[:, g].T * mx["scale"], seen)) @ v[:, g]
    return o.reshape(T, H * D) * sigmoid(rnd(h @ W[p + "g"].T))


# ---- recurrences --------------------------------------------------------------------------------------------
def decayed_sums(q, k, v, decay):
    """o_t = S_t^T q_t with S_t = decay_t S_{t-1} + k_t v_t^T for one head; q, k [T, N], v [T, P], decay [T]"""
    S, o = np.zeros((k.shape[1], v.shape[1])), np.empty_like(v)
    for t in range(len(q)):
        S = decay[t] * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o


def retention(h, W, p, mx, eps, rnd=exact):
    """linear attention with a fixed decay per head, every head's output at unit root mean square, silu gate"""
    T, H, D, V = len(h), mx["heads"], mx["dim"], mx["vdim"]
    pos = np.arange(T, dtype=np.float64)
    turn = lambda x: rnd(rotate_half(x.reshape(T, H, D), pos, mx["rot"]["dims"], mx["rot"]["base"]))
    q, k = turn(h @ W[p + "q"].T), turn(h @ W[p + "k"].T) * D ** -0.5
    v = rnd(h @ W[p + "v"].T).reshape(T, H, V)
    o = np.stack([decayed_sums(q[:, j], k[:, j], v[:, j], np.full(T, mx["decay"][j])) for j in range(H)], 1)
    o = rms_norm(rnd(o), 1.0, eps)
    return o.reshape(T, H * V) * silu(rnd(h @ W[p + "g"].T))


def parallel_mixer(h, W, p, mx, eps, rnd=exact):
    left = rnd(key_valued_attention(h, W, p + "left.", mx["left"], eps, rnd)) @ W[p + "left.o"].T
    right = rnd(retention(h, W, p + "right.", mx["right"], eps, rnd)) @ W[p + "right.o"].T
    return mx["left_scale"] * left + mx["right_scale"] * right


def short_conv(x, w, b):
    """causal convolution per channel, x [T, C], w [C, taps] whose last column weighs the current token"""
    taps = w.shape[1]
    out = np.tile(np.asarray(b, dtype=np.float64), (len(x), 1))
    for t in range(len(x)):
        for j in range(taps):
            if t - (taps - 1 - j) >= 0:
                out[t] += w[:, j] * x[t - (taps - 1 - j)]
    return out


def softplus(z):
    return np.logaddexp(0.0, z)


def gated_norm(o, z, w, groups, eps):
    """the gated row, each of its equal parts at unit root mean square, weighted"""
    y = (o * silu(z)).reshape(len(o), groups, -1)
    return rms_norm(y, 1.0, eps).reshape(o.shape) * w


def mamba2(h, W, p, mx, eps, rnd=exact):
    T, H, P, N, G = len(h), mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * P
    y = h @ W[p + "in"].T
    z, xbc, dt = rnd(y[:, :inner]), rnd(y[:, inner:2 * inner + 2 * G * N]), y[:, 2 * inner + 2 * G * N:]
    xbc = rnd(silu(short_conv(xbc, W[p + "conv"], W[p + "conv.b"])))
    x = xbc[:, :inner].reshape(T, H, P)
    B, C = xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + W[p + "dt_bias"])
    o = np.empty((T, H, P))
    for j in range(H):
        g = j // (H // G)
        decay = np.exp(-np.exp(W[p + "A_log"][j]) * dt[:, j])
        o[:, j] = decayed_sums(C[:, g], B[:, g] * dt[:, j:j + 1], x[:, j], decay) + W[p + "D"][j] * x[:, j]
    return rnd(gated_norm(rnd(o.reshape(T, inner)), z, W[p + "norm"], mx["norm_groups"], eps)) @ W[p + "o"].T


def dense_ff_biased(h, W, p, rnd=exact):
    gate, up = h @ W[p + "gate"].T + W[p + "gate.b"], h @ W[p + "up"].T + W[p + "up.b"]
    return rnd(silu(gate) * up) @ W[p + "down"].T + W[p + "down.b"]


RECURRENT_MIXERS = {"parallel": parallel_mixer, "mamba2": mamba2}


def forward_sandwich(cfg, W, tokens, layers_out=None, rnd=exact):
    """x <- x + N(f(N(x))) for every sublayer, norm weights stored around zero, scaled embedding, separate head"""
    eps = cfg["norm"]["eps"]
    N = lambda x, name: rms_norm(x, 1.0 + W[name], eps)
    x = W["embed"][np.asarray(tokens)].astype(np.float64) * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % i
        y = RECURRENT_MIXERS[L["type"]](rnd(N(x, p + "norm1")), W, p + "mix.", L["mixer"], eps, rnd)
        x = x + N(y, p + "norm1b")
        if L.get("mlp") is not None:
            x = x + N(dense_ff_biased(rnd(N(x, p + "norm2")), W, p + "mlp.", rnd), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x.copy())
    return rnd(N(x, "final.norm")) @ W["head"].T


def forward(cfg, W, tokens, layers_out=None, rnd=exact):
    """logits [T, vocab] of every position of one sequence; layers_out receives x after each layer"""
    if cfg["architecture"] == "Vifelix":
        return forward_sandwich(cfg, W, tokens, layers_out, rnd)
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
