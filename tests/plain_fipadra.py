"""A plain, slow Fipadra: every mechanism as one numpy function over a whole sequence, float64 throughout.

Nothing here is shared with the package: no cache, no state carried between calls, no kernels.  A sequence goes in
whole and every position's result comes out, so that the engine's cuttings (portions, decoding, batches) can be held
against it.  Weights are a dict of numpy arrays by tensor name; the configuration is the plain dict of config.json.

Notation: T tokens, E the model's width, H value or query heads, D key width per head, V value width per head.
"""
import numpy as np

F = np.float64


# ---- small functions --------------------------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps), times w unless it is None."""
    x = x.astype(F)
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if w is None else y * w.astype(F)


def rotate(x, positions, base, dims, layout):
    """x [T, ..., n]: pair i of the first `dims` entries of the last axis turned by position * base^(-2i / dims); pairs are
    (i, i + dims / 2) in the layout "halves" and (2i, 2i + 1) in the layout "neighbours"."""
    y = x.astype(F).copy()
    n = dims // 2
    for i in range(n):
        a, b = (i, i + n) if layout == "halves" else (2 * i, 2 * i + 1)
        angle = np.asarray(positions, dtype=F) * F(base) ** (-2.0 * i / dims)
        angle = angle.reshape((-1,) + (1,) * (x.ndim - 2))
        c, s = np.cos(angle), np.sin(angle)
        u, v = x[..., a].astype(F), x[..., b].astype(F)
        y[..., a] = u * c - v * s
        y[..., b] = v * c + u * s
    return y


def causal_filter(u, taps_w):
    """y[t, c] = sum_j w[c, j] u[t - taps + 1 + j, c], u = 0 before the sequence.  u [T, channels]; w [channels, taps]."""
    T = u.shape[0]
    taps = taps_w.shape[1]
    y = np.zeros_like(u, dtype=F)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += u[:T - back].astype(F) * taps_w[:, j].astype(F)
    return y


# ---- mixers -----------------------------------------------------------------------------------------------------------
def retention(q, k, v, decay):
    """Per head: S_t = decay_h S_{t-1} + k_t v_t^T, o_t = S_t^T q_t.  q, k [T, H, D]; v [T, H, V]; decay [H] -> [T, H, V]."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]), dtype=F)
    out = np.zeros(v.shape, dtype=F)
    for t in range(T):
        S = np.asarray(decay, dtype=F)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def retention_mixer(h, w, pre, m, eps):
    """Rotated q and k (k over sqrt(D)), the decayed recurrence, each head over its root mean square, silu gate, output."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    q = (h @ w[pre + "q"].astype(F).T).reshape(T, H, D)
    k = (h @ w[pre + "k"].astype(F).T).reshape(T, H, D)
    v = (h @ w[pre + "v"].astype(F).T).reshape(T, H, V)
    rot = m.get("rot") or {"base": 1.0, "dims": 0}
    q = rotate(q, pos, rot["base"], rot["dims"], "halves")
    k = rotate(k, pos, rot["base"], rot["dims"], "halves") / np.sqrt(F(D))
    o = rms_norm(retention(q, k, v, m["decay"]), None, eps).reshape(T, H * V)
    return (o * silu(h @ w[pre + "g"].astype(F).T)) @ w[pre + "o"].astype(F).T


def delta_rule(q, k, v, beta, g):
    """Per head: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  q, k [T, H, D]; v [T, H, V]; beta, g [T, H]."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]), dtype=F)
    out = np.zeros(v.shape, dtype=F)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def delta_mixer(h, w, pre, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_filter(h @ w[pre + n].astype(F).T, w[pre + n + ".conv"])) for n in "qkv")
    q, k, v = q.reshape(T, G, D), k.reshape(T, G, D), v.reshape(T, H, V)
    q = q / np.sqrt((q * q).sum(axis=-1, keepdims=True) + 1e-6) / np.sqrt(F(D))
    k = k / np.sqrt((k * k).sum(axis=-1, keepdims=True) + 1e-6)
    q, k = np.repeat(q, H // G, axis=1), np.repeat(k, H // G, axis=1)
    beta = sigmoid(h @ w[pre + "b"].astype(F).T)
    step = softplus(h @ w[pre + "a"].astype(F).T + w[pre + "dt_bias"].astype(F))
    g = np.exp(-np.exp(w[pre + "A_log"].astype(F)) * step)
    o = rms_norm(delta_rule(q, k, v, beta, g), w[pre + "norm"], eps).reshape(T, H * V)
    return (o * silu(h @ w[pre + "g"].astype(F).T)) @ w[pre + "o"].astype(F).T


def windowed_attention(q, k, v, scale, window):
    """q, k [T, H, D], v [T, H, V] -> [T, H, V]; position i sees j with 0 <= i - j < window (None: every j <= i)."""
    T = q.shape[0]
    out = np.zeros(v.shape, dtype=F)
    for i in range(T):
        lo = 0 if window is None else max(0, i + 1 - window)
        s = np.einsum("hd,jhd->hj", q[i], k[lo:i + 1]) * scale
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[i] = np.einsum("hj,jhv->hv", e / e.sum(axis=1, keepdims=True), v[lo:i + 1])
    return out


def latent_attention_mixer(h, w, pre, m, eps):
    """Queries, keys and values through normed latents; one rotated key part for all heads; softmax under a window."""
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    rot = m.get("rot") or {"base": 1.0, "dims": 0}
    q = rms_norm(h @ w[pre + "dq"].astype(F).T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].astype(F).T
    q = q.reshape(T, H, D + R)
    both = h @ w[pre + "dkv"].astype(F).T
    c = rms_norm(both[:, :C], w[pre + "dkv.norm"], eps)
    k_rot = rotate(both[:, C:], pos, rot["base"], rot["dims"], "neighbours")
    q_rot = rotate(q[:, :, D:], pos, rot["base"], rot["dims"], "neighbours")
    k_plain = (c @ w[pre + "uk"].astype(F).T).reshape(T, H, D)
    v = (c @ w[pre + "uv"].astype(F).T).reshape(T, H, V)
    qq = np.concatenate([q[:, :, :D], q_rot], axis=2)
    kk = np.concatenate([k_plain, np.repeat(k_rot[:, None, :], H, axis=1)], axis=2)
    o = windowed_attention(qq, kk, v, m["scale"], (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * V) @ w[pre + "o"].astype(F).T


MIXERS = {"delta": delta_mixer, "latent_attention": latent_attention_mixer, "retention": retention_mixer}


# ---- feed-forward -----------------------------------------------------------------------------------------------------
def squared_relu_unit(h, up, down):
    return np.square(np.maximum(h @ up.astype(F).T, 0.0)) @ down.astype(F).T


def clamped_unit(h, gate, up, down, limit):
    g = np.minimum(h @ gate.astype(F).T, limit)
    u = np.clip(h @ up.astype(F).T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.astype(F).T


def choose(scores, choice_scores, top, group_count, group_keep, scale):
    """One row's experts and their weights.  The outputs form `group_count` equal groups of neighbours; only members of the
    `group_keep` groups with the largest best member can be chosen; of those the `top` largest choice scores; weights are
    the plain scores over their sum, times `scale`.  Equal scores: the lower index first.  Also returns how close the
    choice was (the gap to the first output or group left out, over the spread of the choice scores)."""
    n = len(scores)
    size = n // group_count
    best = choice_scores.reshape(group_count, size).max(axis=1)
    groups = np.argsort(-best, kind="stable")
    kept = sorted(groups[:group_keep])
    allowed = np.concatenate([np.arange(g * size, (g + 1) * size) for g in kept])
    order = allowed[np.argsort(-choice_scores[allowed], kind="stable")]
    chosen = order[:top]
    margin = np.inf
    if group_keep < group_count:
        margin = best[groups[group_keep - 1]] - best[groups[group_keep]]
    if top < len(order):
        margin = min(margin, choice_scores[order[top - 1]] - choice_scores[order[top]])
    p = scores[chosen] / (scores[chosen].sum() + 1e-20) * scale
    return chosen, p, margin / (choice_scores.std() + 1e-30)


def routed_experts(h, w, pre, mlp, margins=None):
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ w[pre + "router"].astype(F).T
    e = np.exp(z - z.max(axis=1, keepdims=True))
    s = e / e.sum(axis=1, keepdims=True)
    cs = s + w[pre + "correction"].astype(F)
    out = np.zeros_like(h)
    close = np.zeros(h.shape[0])
    for t in range(h.shape[0]):
        chosen, p, close[t] = choose(s[t], cs[t], r["top"], groups["count"], groups["keep"], r.get("scale", 1.0))
        for i, pi in zip(chosen, p):
            if i >= r["experts"]:                          # an identity expert: the input itself
                out[t] += pi * h[t]
            else:
                x = f"{pre}e{i}."
                out[t] += pi * clamped_unit(h[t:t + 1], w[x + "gate"], w[x + "up"], w[x + "down"], mlp["expert"]["limit"])[0]
    if margins is not None:
        margins.append(close)
    return out


def feed_forward(h, w, pre, mlp, margins=None):
    if mlp["kind"] == "dense":
        return squared_relu_unit(h, w[pre + "up"], w[pre + "down"])
    out = routed_experts(h, w, pre, mlp, margins)
    if mlp.get("shared") is not None:
        s = pre + "shared."
        out = out + clamped_unit(h, w[s + "gate"], w[s + "up"], w[s + "down"], mlp["shared"]["limit"]) * sigmoid(h @ w[s + "sg"].astype(F).T)
    return out


# ---- the model --------------------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, streams=None, margins=None):
    """Logits [T, vocab] of a whole sequence; `streams`, a list, receives the residual stream after every layer; `margins`,
    a list, one array [T] per routed feed-forward: how close each row's choice of experts was."""
    eps = cfg["norm"]["eps"]
    x = rms_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"], margins)
        x = x + y
        if streams is not None:
            streams.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].astype(F).T * cfg.get("logit_scale", 1.0)
