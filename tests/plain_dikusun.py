"""A plain, slow Dikusun: every mechanism as one numpy function over a whole sequence, float64 throughout.

Nothing here is shared with the package: no cache, no state carried between calls, no kernels.  A sequence goes in
whole and every position's result comes out, so that the engine's cuttings (portions, decoding, batches) can be held
against it.  Weights are a dict of numpy arrays by tensor name; the configuration is the plain dict of config.json.

Notation: T tokens, E the model's width, H query heads, G key/value heads, D key width per head (and map), V value width.
"""
import numpy as np

F = np.float64


# ---- small functions --------------------------------------------------------------------------------------------------
def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, dtype=F)))


def silu(z):
    return z * sigmoid(z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -np.asarray(z, dtype=F))


def linear(h, w, name):
    """h W^T, plus the bias where the weights hold one."""
    y = h @ w[name].astype(F).T
    return y + w[name + ".b"].astype(F) if name + ".b" in w else y


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(np.square(x.astype(F)), axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight.astype(F)


def turn(x, positions, base, dims):
    """x [T, ..., n]: for i < dims / 2 the pair (i, i + dims / 2) of the last axis turned by position * base^(-2i / dims)."""
    half = dims // 2
    y = x.astype(F).copy()
    angle = np.outer(np.asarray(positions, dtype=F), F(base) ** (-2.0 * np.arange(half) / max(dims, 1)))
    angle = angle.reshape((len(positions),) + (1,) * (x.ndim - 2) + (half,))
    u, v = x[..., :half].astype(F), x[..., half:dims].astype(F)
    y[..., :half] = u * np.cos(angle) - v * np.sin(angle)
    y[..., half:dims] = v * np.cos(angle) + u * np.sin(angle)
    return y


# ---- mixers -----------------------------------------------------------------------------------------------------------
def softmax_attention(q, k, v, scale, window=None, softcap=None):
    """One head: q, k [T, D], v [T, V] -> [T, V]; position i sees j with 0 <= i - j < window (None: every j <= i)."""
    T = q.shape[0]
    out = np.zeros((T, v.shape[1]), dtype=F)
    for i in range(T):
        lo = 0 if window is None else max(0, i + 1 - window)
        s = (k[lo:i + 1] @ q[i]) * scale
        if softcap is not None:
            s = softcap * np.tanh(s / softcap)
        e = np.exp(s - s.max())
        out[i] = (e / e.sum()) @ v[lo:i + 1]
    return out


def latent_attention_mixer(h, w, pre, m, eps):
    """Queries through a normed latent of their own, keys and values through another; no positions."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(rms_norm(linear(h, w, pre + "dq"), w[pre + "dq.norm"], eps), w, pre + "uq").reshape(T, H, D)
    c = rms_norm(linear(h, w, pre + "dkv"), w[pre + "dkv.norm"], eps)
    k, v = linear(c, w, pre + "uk").reshape(T, H, D), linear(c, w, pre + "uv").reshape(T, H, V)
    o = np.concatenate([softmax_attention(q[:, i], k[:, i], v[:, i], m["scale"]) for i in range(H)], axis=1)
    return linear(o, w, pre + "o")


def difference_factor(w, pre, diff):
    """exp(lq1 . lk1) - exp(lq2 . lk2) + diff."""
    a, b, c, d = (w[pre + n].astype(F) for n in ("lq1", "lk1", "lq2", "lk2"))
    return np.exp(a @ b) - np.exp(c @ d) + diff


def differential_attention(q, k, v, scale, factor, diff, eps, window=None, softcap=None):
    """q [T, H, 2, D], k [T, G, 2, D], v [T, G, V] -> [T, H, V]: per head the two maps' attentions over the same values, the
    first minus `factor` times the second, over its root mean square, times 1 - diff."""
    T, H, G, V = q.shape[0], q.shape[1], k.shape[1], v.shape[2]
    out = np.zeros((T, H, V), dtype=F)
    for h in range(H):
        g = h // (H // G)
        a = [softmax_attention(q[:, h, n], k[:, g, n], v[:, g], scale, window, softcap) for n in (0, 1)]
        out[:, h] = unit_rms(a[0] - factor * a[1], eps) * (1.0 - diff)
    return out


def attention_mixer(h, w, pre, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(linear(h, w, pre + "q").reshape(T, H, 2, D), w[pre + "q.norm"], eps)
    k = rms_norm(linear(h, w, pre + "k").reshape(T, G, 2, D), w[pre + "k.norm"], eps)
    v = linear(h, w, pre + "v").reshape(T, G, V)
    if m.get("rot"):
        q, k = (turn(x, np.arange(T), m["rot"]["base"], m["rot"]["dims"]) for x in (q, k))
    o = differential_attention(q, k, v, m["scale"], difference_factor(w, pre, m["diff"]), m["diff"], eps,
                               (m.get("mask") or {}).get("size"), m.get("softcap"))
    o = o * sigmoid(linear(h, w, pre + "g"))[:, :, None]
    return linear(o.reshape(T, H * V), w, pre + "o")


def gated_recurrence(q, k, v, alpha):
    """Per head: S_t = diag(alpha_t) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t.  q, k, alpha [T, H, D]; v [T, H, V] -> [T, H, V]."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]), dtype=F)
    out = np.zeros(v.shape, dtype=F)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def gla_mixer(h, w, pre, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(h, w, pre + "q").reshape(T, H, D) / np.sqrt(F(D))
    k, v = linear(h, w, pre + "k").reshape(T, H, D), linear(h, w, pre + "v").reshape(T, H, V)
    alpha = np.exp(log_sigmoid(linear(linear(h, w, pre + "a1"), w, pre + "a2")) / m["tau"]).reshape(T, H, D)
    o = rms_norm(gated_recurrence(q, k, v, alpha), w[pre + "norm"], eps).reshape(T, H * V)
    return linear(o * silu(linear(h, w, pre + "g")), w, pre + "o")


MIXERS = {"latent_attention": latent_attention_mixer, "attention": attention_mixer, "gla": gla_mixer}


# ---- feed-forward -----------------------------------------------------------------------------------------------------
def clamped_unit(h, w, pre, limit):
    g = np.minimum(linear(h, w, pre + "gate"), limit)
    u = np.clip(linear(h, w, pre + "up"), -limit, limit)
    return linear(g * sigmoid(1.702 * g) * (u + 1.0), w, pre + "down")


# ---- the model --------------------------------------------------------------------------------------------------------
def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, w, tokens, streams=None):
    """Logits [T, vocab] of a whole sequence; `streams`, a list, receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)].astype(F) * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        x = x + rms_norm(MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + rms_norm(clamped_unit(x, w, p + "mlp.", layer["mlp"]["limit"]), w[p + "norm2"], eps)
        if streams is not None:
            streams.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].astype(F).T
