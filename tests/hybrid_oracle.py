"""Plain, slow restatement of the hybrid (recurrent + latent attention) decoder in numpy.

One function per mechanism, whole sequences only, no cache, nothing shared with the library.  Weights are
a dict name -> float array with the checkpoint's tensor names; `cfg` is the parsed config.json.  Every
function works in the dtype it is given (float64 by default).
"""
import numpy as np


def rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm_zero_centred(x, w, eps):
    """RMS norm whose stored weight is the deviation from one"""
    return rms(x, eps) * (1 + w)


def sigmoid(z):
    return 0.5 * (1 + np.tanh(0.5 * z))


def softplus(z):
    return np.logaddexp(z, np.zeros_like(z))


def gelu_tanh(z):
    return 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))


def rotate_interleaved(x, pos, base, dims=None):
    """x [T, ..., d]: pairs (2i, 2i+1) of the first `dims` dimensions turned by pos * base^(-2i/dims)"""
    d = x.shape[-1] if dims is None else dims
    f = base ** (-np.arange(0, d, 2, dtype=np.float64) / d)
    a = np.asarray(pos, np.float64)[:, None] * f
    a = a.reshape(a.shape[:1] + (1,) * (x.ndim - 2) + a.shape[1:])
    c, s = np.cos(a).astype(x.dtype), np.sin(a).astype(x.dtype)
    y = x.copy()
    u, v = x[..., 0:d:2], x[..., 1:d:2]
    y[..., 0:d:2] = u * c - v * s
    y[..., 1:d:2] = v * c + u * s
    return y


def causal_conv(x, taps, bias):
    """per-channel convolution over time; taps[:, -1] weighs the newest input, inputs at negative times count as zero"""
    T, n = x.shape[0], taps.shape[1]
    xp = np.concatenate([np.zeros((n - 1, x.shape[1]), x.dtype), x])
    return sum(xp[k:k + T] * taps[:, k] for k in range(n)) + bias


def block_diagonal(u, w, b):
    """w [blocks, m, m], u [T, blocks*m]"""
    T = u.shape[0]
    return (np.einsum("bij,tbj->tbi", w, u.reshape(T, w.shape[0], -1)) + b).reshape(T, -1)


def linear_recurrence(r, i, u, lam):
    """gated diagonal recurrence with the state starting at zero; returns every state"""
    log_a = -8 * r * softplus(lam)
    a = np.exp(log_a)
    x = np.sqrt(-np.expm1(2 * log_a)) * i * u
    s, out = np.zeros_like(u[0]), np.empty_like(u)
    for t in range(len(u)):
        s = a[t] * s + x[t]
        out[t] = s
    return out


def rglru(h, w, p, m):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = sigmoid(block_diagonal(u, w[p + "ra"], w[p + "ra.b"]))
    i = sigmoid(block_diagonal(u, w[p + "ri"], w[p + "ri.b"]))
    return (linear_recurrence(r, i, u, w[p + "lam"]) * y) @ w[p + "o"].T


def window_attention(q, k, v, scale, window):
    """q, k [T, H, d], v [T, H, dv]; query i sees keys j with 0 <= i - j < window"""
    T = q.shape[0]
    s = np.einsum("ihd,jhd->hij", q, k) * scale
    dist = np.arange(T)[:, None] - np.arange(T)[None, :]
    s = np.where((dist >= 0) & (dist < window), s, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    return np.einsum("hij,jhd->ihd", e / e.sum(-1, keepdims=True), v)


def latent_attention(h, w, p, m, eps):
    T, H, dim, rd, vd, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos, base = np.arange(T), m["rot"]["base"]
    q = (h @ w[p + "q"].T).reshape(T, H, dim + rd)
    kv = h @ w[p + "dkv"].T
    c = rms(kv[:, :R], eps) * w[p + "dkv.norm"]
    kr = rotate_interleaved(kv[:, R:], pos, base)
    q = np.concatenate([q[..., :dim], rotate_interleaved(q[..., dim:], pos, base)], -1)
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, dim), np.repeat(kr[:, None], H, 1)], -1)
    v = (c @ w[p + "uv"].T).reshape(T, H, vd)
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"])
    o = o * sigmoid(h @ w[p + "g"].T)[..., None]
    return o.reshape(T, H * vd) @ w[p + "o"].T


def clamped_glu(h, w, p, limit):
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def layer_runs(cfg):
    """the layer index of every pass, in order"""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def layer(x, w, cfg, i):
    d, eps, p = cfg["layers"][i], cfg["norm"]["eps"], f"l{i}."
    h = norm_zero_centred(x, w[p + "norm1"], eps)
    y = rglru(h, w, p + "mix.", d["mixer"]) if d["type"] == "rglru" else latent_attention(h, w, p + "mix.", d["mixer"], eps)
    x = x + norm_zero_centred(y, w[p + "norm1b"], eps)
    if d["mlp"]:
        y = clamped_glu(norm_zero_centred(x, w[p + "norm2"], eps), w, p + "mlp.", d["mlp"]["limit"])
        x = x + norm_zero_centred(y, w[p + "norm2b"], eps)
    return x


def forward(cfg, w, tokens, dtype=np.float64):
    """-> logits [T, vocab], residual stream after every layer run [runs, T, width]"""
    w = {k: np.asarray(v, dtype) for k, v in w.items()}
    x = w["embed"][np.asarray(tokens)] * dtype(cfg["embedding"]["scale"])
    res = []
    for i in layer_runs(cfg):
        x = layer(x, w, cfg, i)
        res.append(x)
    return norm_zero_centred(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T, np.stack(res)
