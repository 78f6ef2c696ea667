"""A plain, slow statement of the Papunex decoder in float64 numpy: one function per mechanism, whole sequences only, no cache, no
portions, no batches.  It shares no code with crabml_b200; the tests compare the framework with it.

Notation: x [T, D] is the residual stream of one sequence, positions 0 .. T-1; a matrix W is stored [out, in] and applied as x @ W.T.
`w` maps tensor names to float arrays, `conf` is the config.json dict as written (optional keys may be missing)."""
import numpy as np


def rms_norm(x, weight, eps):
    x = np.asarray(x, np.float64)
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


# ---- latent attention ----------------------------------------------------------------------------------------------------------------
def rotate_neighbours(v, base):
    """v [T, ..., n], row t at position t: coordinates 2i and 2i+1 turn together by t * base^(-2i / n)"""
    v = np.asarray(v, np.float64)
    T, n = v.shape[0], v.shape[-1]
    out = np.empty_like(v)
    for t in range(T):
        for i in range(n // 2):
            a = t * float(base) ** (-2.0 * i / n)
            p, q = v[t, ..., 2 * i], v[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = p * np.cos(a) - q * np.sin(a)
            out[t, ..., 2 * i + 1] = q * np.cos(a) + p * np.sin(a)
    return out


def latent_rows(h, w, p, m, eps):
    """what a cache holds of a layer: (the normed latents [T, rank], the rotated key part all heads share [T, rot_dim])"""
    rank = int(m["kv_rank"])
    a = h @ w[p + "dkv"].T
    return rms_norm(a[:, :rank], w[p + "dkv.norm"], eps), rotate_neighbours(a[:, rank:], m["rot"]["base"])


def softmax_with_sink(s, sink):
    """s: the scores of the visible keys; the denominator also holds exp(sink)"""
    mx = max(s.max(), sink)
    e = np.exp(s - mx)
    return e / (e.sum() + np.exp(sink - mx))


def latent_attention(h, latents, w, p, m):
    """latents: the (c, r) of the layer whose cache this layer reads (its own, or another's)"""
    c, r = latents
    T, H, dn, dr, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T).reshape(T, H, dn + dr)
    q_plain, q_rot = q[..., :dn], rotate_neighbours(q[..., dn:], m["rot"]["base"])
    k = (c @ w[p + "uk"].T).reshape(T, H, dn)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    out = np.zeros((T, H, dv))
    for i in range(T):
        for hh in range(H):
            s = (k[:i + 1, hh] @ q_plain[i, hh] + r[:i + 1] @ q_rot[i, hh]) * float(m["scale"])
            out[i, hh] = softmax_with_sink(s, float(w[p + "sink"][hh])) @ v[:i + 1, hh]
    gated = out.reshape(T, H * dv) * sigmoid(h @ w[p + "g"].T)
    return gated @ w[p + "o"].T


# ---- state space ---------------------------------------------------------------------------------------------------------------------
def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K]: the last tap multiplies the current row, rows before the start are zeros"""
    T, C = x.shape
    K = taps.shape[1]
    padded = np.concatenate([np.zeros((K - 1, C)), x])
    return np.stack([(padded[t:t + K] * taps.T).sum(0) for t in range(T)]) + bias


def state_space(x, B, Cm, dt, a_log, d_skip):
    """x [T, H, P], B, Cm [T, G, N], dt [T, H] (already positive); head h reads group h // (H / G).  -> [T, H, P]"""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, P))
    y = np.zeros((T, H, P))
    for t in range(T):
        for hh in range(H):
            g = hh // (H // G)
            S[hh] = np.exp(-np.exp(a_log[hh]) * dt[t, hh]) * S[hh] + dt[t, hh] * np.outer(B[t, g], x[t, hh])
            y[t, hh] = S[hh].T @ Cm[t, g] + d_skip[hh] * x[t, hh]
    return y


def gate_then_group_norm(y, z, weight, groups, eps):
    y = y * silu(z)
    parts = y.reshape(y.shape[0], groups, -1)
    parts = parts / np.sqrt((parts * parts).mean(-1, keepdims=True) + eps)
    return parts.reshape(y.shape) * weight


def mamba2(h, w, p, m, eps):
    T, H, P, N, G = h.shape[0], int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * P
    a = h @ w[p + "in"].T
    z, xbc, dt = a[:, :inner], a[:, inner:2 * inner + 2 * G * N], a[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, Cm = xbc[:, :inner].reshape(T, H, P), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    y = state_space(x, B, Cm, softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"]).reshape(T, inner)
    return gate_then_group_norm(y, z, w[p + "norm"], int(m["norm_groups"]), eps) @ w[p + "o"].T


# ---- feed-forwards -------------------------------------------------------------------------------------------------------------------
def squared_relu_ff(h, up, down):
    return relu_squared(h @ up.T) @ down.T


def route(h, router, top, scale):
    """-> (ids [T, top] by falling score, weights [T, top])"""
    z = h @ router.T
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    ids = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    chosen = np.take_along_axis(s, ids, -1)
    return ids, chosen / (chosen.sum(-1, keepdims=True) + 1e-20) * scale


def mixture(h, w, p, mlp):
    r = mlp["router"]
    ids, weights = route(h, w[p + "router"], int(r["top"]), float(r.get("scale", 1.0)))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t], weights[t]):
            out[t] += a * squared_relu_ff(h[t], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
    if mlp.get("shared"):
        out = out + squared_relu_ff(h, w[p + "shared.up"], w[p + "shared.down"]) * sigmoid(h @ w[p + "shared.sg"].T)
    return out


def feed_forward(h, w, p, mlp):
    if mlp["kind"] == "dense":
        return squared_relu_ff(h, w[p + "up"], w[p + "down"])
    return mixture(h, w, p, mlp)


# ---- the whole model -----------------------------------------------------------------------------------------------------------------
def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def forward(conf, weights, tokens, taps=None):
    """-> logits [T, vocab]; taps (a list): receives the residual stream after every layer"""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = float(conf["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)] * float(conf["embedding"]["scale"])
    latents = {}
    for i, L in enumerate(conf["layers"]):
        p, m = f"l{i}.", L["mixer"]
        if L["type"] == "latent_attention":
            j = m.get("kv_from")
            if j is None:
                latents[i] = latent_rows(x, w, p + "mix.", m, eps)
            y = latent_attention(x, latents[i if j is None else int(j)], w, p + "mix.", m)
        else:
            y = mamba2(x, w, p + "mix.", m, eps)
        x = x + rms_norm(y, w[p + "norm1"], eps)
        if L.get("mlp"):
            x = x + rms_norm(feed_forward(x, w, p + "mlp.", L["mlp"]), w[p + "norm2"], eps)
        if taps is not None:
            taps.append(x.copy())
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = float(conf.get("logit_softcap") or 0.0)
    return soft_cap(logits, cap) if cap > 0 else logits
