"""Plain, slow restatement of the Lomodra decoder in numpy: three mixers (scalar-decay linear attention, chunked grouped-query
attention, gated delta rule), experts with a shared one, norms behind every sub-layer, per-layer token input.

One function per mechanism, whole sequences only, no cache, token loops where the mechanism is a recurrence; nothing is
shared with the library.  Weights are a dict name -> float array with the checkpoint's tensor names; `cfg` is the parsed
config.json.  Every function works in the dtype it is given (float64 by default).
"""
import numpy as np


def over_rms(x, eps):
    """every row divided by its root mean square"""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(z):
    return 0.5 * (1 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(z, np.zeros_like(z))


def gelu_tanh(z):
    return 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))


def split_heads(x, n):
    return x.reshape(x.shape[0], n, -1)


# ---- scalar-decay linear attention -----------------------------------------------------------------
def decayed_outer_products(q, k, v, decay):
    """q, k [T, H, d], v [T, H, e], decay [H]: o_t = S_t^T q_t of S_t = decay S_(t-1) + k_t v_t^T"""
    T, H, _ = q.shape
    s, o = np.zeros((H, q.shape[2], v.shape[2]), q.dtype), np.empty_like(v)
    for t in range(T):
        s = decay[:, None, None] * s + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hde,hd->he", s, q[t])
    return o


def lightning(h, w, p, m, eps):
    H = m["heads"]
    q, k, v = (split_heads(silu(h @ w[p + n].T), H) for n in ("q", "k", "v"))
    o = decayed_outer_products(q, k, v, np.asarray(m["decay"], h.dtype)).reshape(h.shape[0], -1)
    return (over_rms(o, eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- chunked attention ------------------------------------------------------------------------------
def chunked_attention(q, k, v, scale, chunk):
    """q [T, H, d], k [T, G, d], v [T, G, e]; query i sees the keys j <= i of its own chunk of positions"""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    pos = np.arange(T)
    seen = (pos[None, :] <= pos[:, None]) & (pos[None, :] // chunk == pos[:, None] // chunk)
    o = np.empty((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        s = np.where(seen, q[:, h] @ k[:, h // rep].T * scale, -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        o[:, h] = e / e.sum(-1, keepdims=True) @ v[:, h // rep]
    return o


def attention_keys(h, w, p, m, eps):
    """what a layer's cache holds: normed keys, values"""
    G = m["kv_heads"]
    return over_rms(split_heads(h @ w[p + "k"].T, G), eps) * w[p + "k.norm"], split_heads(h @ w[p + "v"].T, G)


def attention(h, w, p, m, eps, k, v):
    q = over_rms(split_heads(h @ w[p + "q"].T, m["heads"]), eps) * w[p + "q.norm"]
    o = chunked_attention(q, k, v, m["scale"], m["mask"]["size"])
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


# ---- gated delta rule -----------------------------------------------------------------------------------
def causal_conv(x, taps):
    """per-channel convolution over time; taps[:, -1] weighs the newest input, inputs at negative times count as zero"""
    T, n = x.shape[0], taps.shape[1]
    xp = np.concatenate([np.zeros((n - 1, x.shape[1]), x.dtype), x])
    return sum(xp[i:i + T] * taps[:, i] for i in range(n))


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def channel_decay(h, w, p, heads):
    """[T, heads, dim]: exp(-exp(A) softplus(a2 a1 h + dt))"""
    z = split_heads(h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "dt_bias"], heads)
    return np.exp(-np.exp(w[p + "A_log"])[:, None] * softplus(z))


def delta_rule(q, k, v, g, beta):
    """q, k, g [T, H, d], v [T, H, e], beta [T, H]: decay the rows, write what k does not recall of v, read with q"""
    T, H, d = k.shape
    s, o = np.zeros((H, d, v.shape[2]), q.dtype), np.empty_like(v)
    for t in range(T):
        s = g[t][:, :, None] * s
        u = beta[t][:, None] * (v[t] - np.einsum("hde,hd->he", s, k[t]))
        s = s + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hde,hd->he", s, q[t])
    return o


def channel_delta(h, w, p, m, eps):
    H, KV = m["heads"], m["kv_heads"]
    q, k, v = (split_heads(silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])), c) for n, c in (("q", KV), ("k", KV), ("v", H)))
    q, k = (np.repeat(unit(x), H // KV, axis=1) for x in (q, k))
    q = q * m["dim"] ** -0.5
    beta = sigmoid(h @ w[p + "b"].T)
    o = delta_rule(q, k, v, channel_decay(h, w, p, H), beta)
    gate = sigmoid(split_heads(h @ w[p + "g1"].T @ w[p + "g2"].T, H))
    return (over_rms(o, eps) * w[p + "norm"] * gate).reshape(h.shape[0], -1) @ w[p + "o"].T


# ---- feed-forward -----------------------------------------------------------------------------------------
def glu(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top):
    """[T, E] logits -> weights [T, E]: softmax over the `top` largest, zero elsewhere"""
    out = np.zeros_like(z)
    for t in range(len(z)):
        best = np.argsort(-z[t], kind="stable")[:top]
        e = np.exp(z[t, best] - z[t, best].max())
        out[t, best] = e / e.sum()
    return out


def experts(h, w, p, m):
    r = route(h @ w[p + "router"].T + w[p + "router.b"], m["router"]["top"])
    y = glu(h, w, p + "shared.") if m.get("shared") else np.zeros_like(h)
    for e in range(m["router"]["experts"]):
        t = r[:, e] > 0
        if t.any():
            y[t] += r[t, e][:, None] * glu(h[t], w, p + f"e{e}.")
    return y


# ---- the whole model -----------------------------------------------------------------------------------------
def token_input(x, w, i, tokens, dim, eps):
    p = f"l{i}.side."
    e = w["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return over_rms(y, eps) * w[p + "norm"]


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def forward(cfg, w, tokens, dtype=np.float64):
    """-> logits [T, vocab], residual stream after every layer [layers, T, width]"""
    w = {k: np.asarray(v, dtype) for k, v in w.items()}
    tokens, eps = np.asarray(tokens), cfg["norm"]["eps"]
    x, res, cache = w["embed"][tokens], [], {}
    for i, d in enumerate(cfg["layers"]):
        p, m = f"l{i}.", d["mixer"]
        if d["type"] == "lightning":
            y = lightning(x, w, p + "mix.", m, eps)
        elif d["type"] == "channel_delta":
            y = channel_delta(x, w, p + "mix.", m, eps)
        else:
            if m.get("kv_from") is None:
                cache[i] = attention_keys(x, w, p + "mix.", m, eps)
            y = attention(x, w, p + "mix.", m, eps, *cache[i if m.get("kv_from") is None else m["kv_from"]])
        x = x + over_rms(y, eps) * w[p + "norm1"]
        if d["mlp"]:
            x = x + over_rms(experts(x, w, p + "mlp.", d["mlp"]), eps) * w[p + "norm2"]
        if cfg.get("token_side"):
            x = x + token_input(x, w, i, tokens, cfg["token_side"]["dim"], eps)
        res.append(x)
    logits = over_rms(x, eps) * w["final.norm"] @ w["embed"].T
    if cfg.get("logit_softcap"):
        logits = soft_cap(logits, cfg["logit_softcap"])
    return logits, np.stack(res)
