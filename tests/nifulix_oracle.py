"""Plain float64 restatement of the Nifulix design, one function per mechanism, written for the tests only.  It shares no code
with the engine: numpy on the CPU, the retention token by token, attention over explicit lists of visible keys, latent keys
and values expanded per head.  Tensors come as a dict name -> array (names as in the model file).

Notation: W width, H heads, G key/value heads, d query/key size (latent: its unrotated part), dr rotated size, dv value size,
r latent size, w window length, n kept first positions.
"""
import numpy as np


def rms_unit(v, eps):
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    v = np.asarray(v, np.float64)
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


def rms_norm_around_one(v, w, eps):
    """The layer and final norm: the stored vector is the gain's distance from one."""
    return rms_unit(v, eps) * (1.0 + w)


def rms_norm_plain(v, w, eps):
    return rms_unit(v, eps) * w


def sigmoid(z):
    z = np.asarray(z, np.float64)
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return np.asarray(z, np.float64) * sigmoid(z)


def angles(p, dims, base):
    return [p * base ** (-2.0 * i / dims) for i in range(dims // 2)]


def rotate_halves(v, p, dims, base):
    """Coordinate i < dims/2 turns with coordinate i + dims/2; coordinates from dims on stay."""
    out = np.array(v, np.float64)
    for i, a in enumerate(angles(p, dims, base)):
        x, y = v[i], v[i + dims // 2]
        out[i], out[i + dims // 2] = x * np.cos(a) - y * np.sin(a), y * np.cos(a) + x * np.sin(a)
    return out


def rotate_neighbours(v, p, dims, base):
    """Coordinate 2i turns with coordinate 2i + 1; coordinates from dims on stay."""
    out = np.array(v, np.float64)
    for i, a in enumerate(angles(p, dims, base)):
        x, y = v[2 * i], v[2 * i + 1]
        out[2 * i], out[2 * i + 1] = x * np.cos(a) - y * np.sin(a), y * np.cos(a) + x * np.sin(a)
    return out


def in_window(i, j, window, keep=0):
    """Causal; with a window w > 0 only the keys less than w back and the first `keep` positions are seen."""
    return j <= i and (window <= 0 or i - j < window or j < keep)


def softmax(s):
    s = np.asarray(s, np.float64)
    e = np.exp(s - s.max())
    return e / e.sum()


def distance_slope(h, heads):
    return 2.0 ** (-8.0 * (h + 1) / heads)


def score(q, k, scale, cap, slope, dist):
    """Scaled product, squeezed by the cap, then lowered in proportion to the distance.  k: one key or a row per key."""
    s = k @ q * scale
    if cap:
        s = cap * np.tanh(s / cap)
    return s - slope * dist


def mixed_values(own, first, lam):
    return (1.0 - lam) * own + lam * first


def attention(mx, P, p, h, shared):
    """Grouped-query attention.  shared: dict that carries the first value-mixing layer's values through the forward pass."""
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    mask = mx.get("mask") or {}
    window, keep, cap = int(mask.get("size", 0)), int(mask.get("keep_first", 0)), float(mx.get("softcap") or 0.0)
    q = (h @ P[p + "q"].T).reshape(T, H, d)
    k = (h @ P[p + "k"].T).reshape(T, G, d)
    v = h @ P[p + "v"].T
    if mx.get("v_mix"):
        if "first" in shared:
            v = mixed_values(v, shared["first"], float(P[p + "vmix"]))
        else:
            shared["first"] = v
    v = v.reshape(T, G, dv)
    out = np.zeros((T, H, dv))
    for i in range(T):
        seen = [j for j in range(i + 1) if in_window(i, j, window, keep)]
        for hd in range(H):
            g = hd // (H // G)
            wts = softmax(score(q[i, hd], k[seen, g], mx["scale"], cap, distance_slope(hd, H), i - np.array(seen)))
            out[i, hd] = wts @ v[seen, g]
    return (out.reshape(T, -1) * sigmoid(h @ P[p + "g"].T)) @ P[p + "o"].T


def retention_head(q, k, v, decay):
    """S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t from S = 0.  q, k [T][d], v [T][dv]."""
    S = np.zeros((k.shape[1], v.shape[1]))
    out = np.zeros((len(q), v.shape[1]))
    for t in range(len(q)):
        S = decay * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def retention(mx, P, p, h, eps):
    T = h.shape[0]
    H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
    dims, base = int(mx["rot"]["dims"]), float(mx["rot"]["base"])
    q = (h @ P[p + "q"].T).reshape(T, H, d)
    k = (h @ P[p + "k"].T).reshape(T, H, d)
    v = (h @ P[p + "v"].T).reshape(T, H, dv)
    out = np.zeros((T, H, dv))
    for hd in range(H):
        qr = np.stack([rotate_halves(q[t, hd], t, dims, base) for t in range(T)])
        kr = np.stack([rotate_halves(k[t, hd], t, dims, base) for t in range(T)]) * d ** -0.5
        out[:, hd] = rms_unit(retention_head(qr, kr, v[:, hd], mx["decay"][hd]), eps)
    return (out.reshape(T, -1) * silu(h @ P[p + "g"].T)) @ P[p + "o"].T


def latent_attention(mx, P, p, h, eps):
    T = h.shape[0]
    H, d, dr, dv, r = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    dims, base = int(mx["rot"]["dims"]), float(mx["rot"]["base"])
    window = int((mx.get("mask") or {}).get("size", 0))
    if mx.get("q_rank"):
        q = rms_norm_plain(h @ P[p + "dq"].T, P[p + "dq.norm"], eps) @ P[p + "uq"].T
    else:
        q = h @ P[p + "q"].T
    q = q.reshape(T, H, d + dr)
    both = h @ P[p + "dkv"].T
    c = rms_norm_plain(both[:, :r], P[p + "dkv.norm"], eps)
    kr = np.stack([rotate_neighbours(both[t, r:], t, dims, base) for t in range(T)])
    k = (c @ P[p + "uk"].T).reshape(T, H, d)
    v = (c @ P[p + "uv"].T).reshape(T, H, dv)
    out = np.zeros((T, H, dv))
    for i in range(T):
        seen = [j for j in range(i + 1) if in_window(i, j, window)]
        for hd in range(H):
            qr = rotate_neighbours(q[i, hd, d:], i, dims, base)
            wts = softmax((k[seen, hd] @ q[i, hd, :d] + kr[seen] @ qr) * mx["scale"])
            out[i, hd] = wts @ v[seen, hd]
    return out.reshape(T, -1) @ P[p + "o"].T


def gated_unit(P, p, h):
    return (silu(h @ P[p + "gate"].T) * (h @ P[p + "up"].T)) @ P[p + "down"].T


def layer(ly, P, p, x, eps, mult, shared):
    """Both sublayers read the one norm's output; their sum, times the multiplier, joins the residual."""
    h = rms_norm_around_one(x, P[p + "norm1"], eps)
    if ly["type"] == "attention":
        y = attention(ly["mixer"], P, p + "mix.", h, shared)
    elif ly["type"] == "retention":
        y = retention(ly["mixer"], P, p + "mix.", h, eps)
    else:
        y = latent_attention(ly["mixer"], P, p + "mix.", h, eps)
    if ly.get("mlp"):
        y = y + gated_unit(P, p + "mlp.", h)
    return x + mult * y


def forward(cfg, P, tokens):
    """Logits [T][vocab] of one sequence and the residual after every layer."""
    P = {k: np.asarray(v, np.float64) for k, v in P.items()}
    eps, mult = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x = P["embed"][np.asarray(tokens)]
    shared, trail = {}, []
    for i, ly in enumerate(cfg["layers"]):
        x = layer(ly, P, f"l{i}.", x, eps, mult, shared)
        trail.append(x)
    return rms_norm_around_one(x, P["final.norm"], eps) @ P["head"].T, trail
