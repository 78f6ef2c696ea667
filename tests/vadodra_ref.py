"""A plain, slow statement of the Vadodra decoder in float64 numpy: one function per mechanism, whole sequences only, no cache, no
portions, no batches.  It shares no code with crabml_b200; the tests compare the framework with it.

Notation: x [T, D] is the residual stream of one sequence, row t at position t; a matrix W is kept [out, in] and used as x @ W.T.
`w` maps tensor names to float arrays, `conf` is the config.json dict as written."""
import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def layer_norm(x, weight, eps):
    x = np.asarray(x, np.float64)
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * weight


def rms_norm(x, weight, eps):
    x = np.asarray(x, np.float64)
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * weight


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


# ---- rotation ---------------------------------------------------------------------------------------------------------------------------
def frequency(i, rot):
    f = float(rot["base"]) ** (-2.0 * i / int(rot["dims"]))
    sc = rot.get("scaling")
    return f / float(sc["factor"]) if sc else f


def _turn(out, v, t, a, lo, hi):
    p, q = v[t, ..., lo], v[t, ..., hi]
    out[t, ..., lo] = p * np.cos(a) - q * np.sin(a)
    out[t, ..., hi] = q * np.cos(a) + p * np.sin(a)


def rotate_neighbours(v, rot):
    """v [T, ..., n]: of the first rot.dims coordinates, 2i and 2i + 1 turn together"""
    v = np.asarray(v, np.float64)
    out = v.copy()
    for t in range(v.shape[0]):
        for i in range(int(rot["dims"]) // 2):
            _turn(out, v, t, t * frequency(i, rot), 2 * i, 2 * i + 1)
    return out


def rotate_halves(v, rot):
    """v [T, ..., n]: of the first rot.dims coordinates, i and i + dims / 2 turn together"""
    v = np.asarray(v, np.float64)
    out = v.copy()
    half = int(rot["dims"]) // 2
    for t in range(v.shape[0]):
        for i in range(half):
            _turn(out, v, t, t * frequency(i, rot), i, i + half)
    return out


# ---- attention whose values are its raw keys ----------------------------------------------------------------------------------------------
def window_attention(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]"""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        lo = max(0, i - window + 1)
        for h in range(H):
            g = h // (H // G)
            out[i, h] = softmax(k[lo:i + 1, g] @ q[i, h] * scale) @ v[lo:i + 1, g]
    return out


def attention(h, w, p, m, eps):
    T, H, G, d = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = (h @ w[p + "q"].T).reshape(T, H, d)
    raw = (h @ w[p + "k"].T).reshape(T, G, d)
    q = rms_norm(q, w[p + "q.norm"], eps)
    k = rms_norm(raw, w[p + "k.norm"], eps)
    q, k = rotate_neighbours(q, m["rot"]), rotate_neighbours(k, m["rot"])
    return window_attention(q, k, raw, float(m["scale"]), int(m["mask"]["size"])).reshape(T, H * d) @ w[p + "o"].T


# ---- latent attention -------------------------------------------------------------------------------------------------------------------
def latent_rows(h, w, p, m, eps):
    """what a cache holds of a layer: (normed latents [T, rank], rotated key part of all heads [T, rot_dim])"""
    rank = int(m["kv_rank"])
    a = h @ w[p + "dkv"].T
    return rms_norm(a[:, :rank], w[p + "dkv.norm"], eps), rotate_halves(a[:, rank:], m["rot"])


def latent_attention(h, rows, w, p, m):
    """rows: the (c, r) of the layer whose cache this layer reads (its own, or another's)"""
    c, r = rows
    T, H, dn, dr, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T).reshape(T, H, dn + dr)
    q_plain, q_rot = q[..., :dn], rotate_halves(q[..., dn:], m["rot"])
    k = (c @ w[p + "uk"].T).reshape(T, H, dn)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    gate = sigmoid(h @ w[p + "g"].T)
    out = np.zeros((T, H, dv))
    for i in range(T):
        for hh in range(H):
            s = (k[:i + 1, hh] @ q_plain[i, hh] + r[:i + 1] @ q_rot[i, hh]) * float(m["scale"])
            out[i, hh] = gate[i, hh] * (softmax(s) @ v[:i + 1, hh])
    return out.reshape(T, H * dv) @ w[p + "o"].T


# ---- feed-forward -----------------------------------------------------------------------------------------------------------------------
def clamped_unit(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, w, p, mlp):
    return clamped_unit(h @ w[p + "gate"].T, h @ w[p + "up"].T, float(mlp["limit"])) @ w[p + "down"].T


# ---- the whole model --------------------------------------------------------------------------------------------------------------------
def forward(conf, weights, tokens, taps=None):
    """-> logits [T, vocab]; taps (a list): receives the residual stream after every layer"""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = float(conf["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)] * float(conf["embedding"]["scale"])
    caches = {}
    for i, L in enumerate(conf["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = layer_norm(x, w[p + "norm1"], eps)
        if L["type"] == "attention":
            y = attention(h, w, p + "mix.", m, eps)
        else:
            j = m.get("kv_from")
            if j is None:
                caches[i] = latent_rows(h, w, p + "mix.", m, eps)
            y = latent_attention(h, caches[i if j is None else int(j)], w, p + "mix.", m)
        if L.get("mlp"):
            y = y + feed_forward(h, w, p + "mlp.", L["mlp"])
        x = x + y
        if taps is not None:
            taps.append(x.copy())
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T
