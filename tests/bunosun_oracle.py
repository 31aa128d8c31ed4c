"""Plain float64 restatement of the Bunosun design, one function per mechanism, written for the tests only.  It shares no code
with the engine: numpy on the CPU, the delta rule token by token over an explicit state, attention over explicit lists of visible
keys, the router by sorting.  Tensors come as a dict name -> array (names as in the model file).

Notation: W width, H heads, G key/value heads, d query/key size (of one map), dv value size, w window length, E experts.
"""
import numpy as np


def rms_unit(v, eps):
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    v = np.asarray(v, np.float64)
    return v / np.sqrt(np.mean(v * v, axis=-1, keepdims=True) + eps)


def rms_norm_around_one(v, w, eps):
    """The layer and final norms: the stored vector is the gain's distance from one."""
    return rms_unit(v, eps) * (1.0 + w)


def length_unit(v, eps=1e-6):
    """v / sqrt(sum(v^2) + eps) over the last axis."""
    return v / np.sqrt(np.sum(v * v, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    z = np.asarray(z, np.float64)
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return np.asarray(z, np.float64) * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def softmax(s):
    e = np.exp(s - np.max(s))
    return e / e.sum()


# ---------------------------------------------------------------------------------------------- differential attention
def rotate_neighbours(v, p, dims, base, factor=1.0):
    """Coordinate 2i turns with coordinate 2i + 1 by p base^(-2i/dims) / factor; coordinates from dims on stay.  v [..., d]."""
    out = np.array(v, np.float64)
    for i in range(dims // 2):
        a = p * (base ** (-2.0 * i / dims) / factor)
        x, y = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = x * np.cos(a) - y * np.sin(a), y * np.cos(a) + x * np.sin(a)
    return out


def in_window(i, j, window):
    """Causal; with a window w > 0 only the keys less than w positions back."""
    return 0 <= i - j and (window <= 0 or i - j < window)


def map_weight(P, p, diff):
    """The factor on the second map: one number per layer."""
    return float(np.exp(np.sum(P[p + "lq1"] * P[p + "lk1"])) - np.exp(np.sum(P[p + "lq2"] * P[p + "lk2"])) + diff)


def combine_maps(a1, a2, lam, diff, eps):
    """The maps' difference, divided by its root mean square over the value coordinates, times 1 - diff."""
    return rms_unit(a1 - lam * a2, eps) * (1.0 - diff)


def attention(mx, P, p, h, eps):
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    window = int((mx.get("mask") or {}).get("size", 0))
    rot = mx.get("rot") or {}
    dims, base = int(rot.get("dims", 0)), float(rot.get("base", 1.0))
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    q = (h @ P[p + "q"].T).reshape(T, H, 2, d)
    k = (h @ P[p + "k"].T).reshape(T, G, 2, d)
    v = (h @ P[p + "v"].T).reshape(T, G, dv)
    q = np.stack([rotate_neighbours(q[t], t, dims, base, factor) for t in range(T)])
    k = np.stack([rotate_neighbours(k[t], t, dims, base, factor) for t in range(T)])
    lam = map_weight(P, p, mx["diff"])
    out = np.zeros((T, H, dv))
    for i in range(T):
        seen = [j for j in range(i + 1) if in_window(i, j, window)]
        for hd in range(H):
            g = hd // (H // G)
            a = [softmax(k[seen, g, m] @ q[i, hd, m] * mx["scale"]) @ v[seen, g] for m in (0, 1)]
            out[i, hd] = combine_maps(a[0], a[1], lam, mx["diff"], eps)
    return out.reshape(T, -1) @ P[p + "o"].T


# ---------------------------------------------------------------------------------------------- gated delta rule
def causal_conv(x, w):
    """Per channel: y[t] = sum_j w[:, j] x[t - (taps - 1) + j], zeros before the start.  x [T][C], w [C][taps]."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return sum(w[:, j] * padded[j:j + len(x)] for j in range(taps))


def channel_decay(z, a_log, dt_bias):
    """exp(-exp(a_log) softplus(z + dt_bias)); z [..., H, d], a_log [H], dt_bias [H, d]."""
    return np.exp(-np.exp(a_log)[:, None] * softplus(z + dt_bias))


def delta_head(q, k, v, g, beta):
    """One head from a zero state: every row of S decays by its channel's factor, the value's distance from what the key reads
    back, times beta, is written at the key, and the query reads the state with the token's write in it."""
    S = np.zeros((k.shape[1], v.shape[1]))
    out = np.zeros((len(q), v.shape[1]))
    for t in range(len(q)):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def channel_delta(mx, P, p, h, eps):
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(h @ P[p + n].T, P[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = length_unit(q.reshape(T, G, d)) * d ** -0.5
    k = length_unit(k.reshape(T, G, d))
    v = v.reshape(T, H, dv)
    beta = sigmoid(h @ P[p + "b"].T)
    g = channel_decay(((h @ P[p + "a1"].T) @ P[p + "a2"].T).reshape(T, H, d), P[p + "A_log"], P[p + "dt_bias"].reshape(H, d))
    out = np.zeros((T, H, dv))
    for hd in range(H):
        kv = hd // (H // G)
        out[:, hd] = rms_unit(delta_head(q[:, kv], k[:, kv], v[:, hd], g[:, hd], beta[:, hd]), eps) * P[p + "norm"]
    gate = sigmoid((h @ P[p + "g1"].T) @ P[p + "g2"].T)
    return (out.reshape(T, -1) * gate) @ P[p + "o"].T


# ---------------------------------------------------------------------------------------------- mixture of experts
def gated_unit(P, p, h):
    return (silu(h @ P[p + "gate"].T) * (h @ P[p + "up"].T)) @ P[p + "down"].T


def choose(z, correction, top, groups, keep):
    """Experts of one token and their weights from its logits: softmax scores plus the correction rank the experts, a run of
    neighbours ranks by its best, experts outside the best runs are out; the weights are the plain scores of the chosen."""
    s = softmax(z)
    c = s + correction
    if groups and groups > 1:
        per = len(z) // groups
        best = [max(c[g * per:(g + 1) * per]) for g in range(groups)]
        kept = sorted(range(groups), key=lambda g: -best[g])[:keep]
        c = np.array([c[e] if e // per in kept else -np.inf for e in range(len(z))])
    ids = sorted(range(len(z)), key=lambda e: -c[e])[:top]
    return ids, s[ids] / (np.sum(s[ids]) + 1e-20)


def mixture(ml, P, p, h):
    r = ml["router"]
    gr = r.get("groups") or {}
    Z = h @ P[p + "router"].T
    out = np.zeros_like(h)
    chosen = [choose(Z[t], P[p + "correction"], r["top"], gr.get("count", 0), gr.get("keep", 0)) for t in range(len(h))]
    for e in range(r["experts"]):
        ts = [t for t in range(len(h)) if e in chosen[t][0]]
        if ts:
            y = gated_unit(P, f"{p}e{e}.", h[ts])
            for n, t in enumerate(ts):
                ids, w = chosen[t]
                out[t] += w[ids.index(e)] * y[n]
    if ml.get("shared"):
        out = out + gated_unit(P, p + "shared.", h)
    return out


# ---------------------------------------------------------------------------------------------- the model
def layer(ly, P, p, x, eps):
    """Both sublayers read x through norms of their own; each result is scaled per coordinate before the sum."""
    mix = attention if ly["type"] == "attention" else channel_delta
    y = mix(ly["mixer"], P, p + "mix.", rms_norm_around_one(x, P[p + "norm1"], eps), eps) * P[p + "ls1"]
    if ly.get("mlp"):
        y = y + mixture(ly["mlp"], P, p + "mlp.", rms_norm_around_one(x, P[p + "norm2"], eps)) * P[p + "ls2"]
    return x + y


def order_of_runs(cfg):
    """(layer, whether the embedding joins in front of it) of every layer run."""
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp or not lp.get("times"):
        return [(i, False) for i in range(n)]
    a, b, times = lp["start"], lp["stop"], lp["times"]
    return [(i, False) for i in range(a)] + [(i, t > 0 and i == a) for t in range(times) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def forward(cfg, P, tokens):
    """Logits [T][vocab] of one sequence and the residual after every layer run."""
    P = {k: np.asarray(v, np.float64) for k, v in P.items()}
    eps = float(cfg["norm"]["eps"])
    x0 = P["embed"][np.asarray(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    x, trail = x0, []
    for i, again in order_of_runs(cfg):
        if again:
            x = x + x0
        x = layer(cfg["layers"][i], P, f"l{i}.", x, eps)
        trail.append(x)
    return rms_norm_around_one(x, P["final.norm"], eps) @ P["head"].T, trail
