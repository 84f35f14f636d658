"""Plain float64 restatement of the Kugalorn design, one function per mechanism, written from the design's equations.  It shares no code
with the package; it is slow on purpose (explicit loops over tokens and heads) and runs on the CPU with numpy alone.

Notation: h [T, W] is a sublayer's input, weights are [out, in] and applied as h @ w.T; `w` dictionaries hold a sublayer's tensors under
their checkpoint names with the prefix removed ("q", "dkv.norm", "e0.gate", ...).  Every function takes one whole sequence whose first
token has position 0."""
import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose weight tensor holds the distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


# ----------------------------------------------------------------------------------------------------------- softmax attention
def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def head_slopes(H):
    """Slope of the distance penalty of every head."""
    return [2.0 ** (-8.0 * (h + 1) / H) for h in range(H)]


def window_keys(i, size):
    return list(range(max(0, i - size + 1), i + 1))


def windowed_attention(h, w, m, eps):
    """Grouped-query attention under a sliding window; unit-RMS queries and keys; a penalty that grows with the distance."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w["q"].T).reshape(T, H, d), eps)
    k = unit_rms((h @ w["k"].T).reshape(T, G, d), eps)
    v = (h @ w["v"].T).reshape(T, G, dv)
    slope = head_slopes(H)
    out = np.zeros((T, H, dv))
    for i in range(T):
        js = np.array(window_keys(i, m["mask"]["size"]))
        for a in range(H):
            g = a // (H // G)
            out[i, a] = softmax(k[js, g] @ q[i, a] * m["scale"] - slope[a] * (i - js)) @ v[js, g]
    return out.reshape(T, H * dv) @ w["o"].T


def turn_pairs(x, positions, base):
    """x [T, ..., d]: dimensions 2i and 2i + 1 turn by position * base^(-2i / d)."""
    d = x.shape[-1]
    y = x.copy()
    for t, p in enumerate(positions):
        for i in range(d // 2):
            a = p * base ** (-2.0 * i / d)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            y[t, ..., 2 * i] = u * c - v * s
            y[t, ..., 2 * i + 1] = v * c + u * s
    return y


def latent_attention(h, w, m, eps):
    """Causal attention whose keys and values come from one normed latent per token plus one rotated key part shared by the heads; one
    sigmoid gate per head."""
    T = h.shape[0]
    H, dn, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w["q"].T).reshape(T, H, dn + dr)
    both = h @ w["dkv"].T
    c = unit_rms(both[:, :r], eps) * w["dkv.norm"]
    pos, base = range(T), m["rot"]["base"]
    kr, qr = turn_pairs(both[:, r:], pos, base), turn_pairs(q[:, :, dn:], pos, base)
    kn = (c @ w["uk"].T).reshape(T, H, dn)
    v = (c @ w["uv"].T).reshape(T, H, dv)
    gate = sigmoid(h @ w["g"].T)
    out = np.zeros((T, H, dv))
    for i in range(T):
        for a in range(H):
            s = (kn[:i + 1, a] @ q[i, a, :dn] + kr[:i + 1] @ qr[i, a]) * m["scale"]
            out[i, a] = softmax(s) @ v[:i + 1, a] * gate[i, a]
    return out.reshape(T, H * dv) @ w["o"].T


# ----------------------------------------------------------------------------------------------------------- feed-forward
def clamped_unit(h, w, limit):
    g = np.minimum(h @ w["gate"].T, limit)
    u = np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


def choose(z, top):
    """[(expert, weight)] for one token's router logits: the largest `top`, weighted by a softmax over those alone."""
    order = np.argsort(-z, kind="stable")[:top]
    return list(zip(order.tolist(), softmax(z[order])))


def routed_experts(h, w, m):
    T = h.shape[0]
    z = h @ w["router"].T + w["router.b"]
    y = np.zeros((T, h.shape[1]))
    for t in range(T):
        for e, p in choose(z[t], m["router"]["top"]):
            y[t] += p * clamped_unit(h[t], sub(w, f"e{e}."), m["expert"]["limit"])
    if m.get("shared"):
        y = y + clamped_unit(h, sub(w, "shared."), m["shared"]["limit"])
    return y


# ----------------------------------------------------------------------------------------------------------- streams and layers
def read_streams(xs, a):
    """Sublayer input: sum_s a[s] x_s."""
    return sum(a[s] * xs[s] for s in range(len(xs)))


def write_streams(xs, mix, out, y):
    """New streams, all from the old ones: x_t <- sum_s mix[s, t] x_s + out[t] y."""
    n = len(xs)
    return [sum(mix[s, t] * xs[s] for s in range(n)) + out[t] * y for t in range(n)]


def layer_order(n, loop):
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def mixer(kind, h, w, m, eps):
    if kind == "attention":
        return windowed_attention(h, w, m, eps)
    if kind == "latent_attention":
        return latent_attention(h, w, m, eps)
    raise ValueError(kind)


def forward(cfg, weights, tokens, trace=None):
    """Logits [T, vocab] of one sequence; trace (a list) collects the sum of the streams after every layer run."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    xs = [w["embed"][np.asarray(tokens)]] * cfg["streams"]
    for i in layer_order(len(cfg["layers"]), cfg.get("loop")):
        L, p = cfg["layers"][i], f"l{i}."
        h = offset_norm(read_streams(xs, w[p + "hc1.in"]), w[p + "norm1"], eps)
        xs = write_streams(xs, w[p + "hc1.mix"], w[p + "hc1.out"], mixer(L["type"], h, sub(w, p + "mix."), L["mixer"], eps))
        if L.get("mlp"):
            h = offset_norm(read_streams(xs, w[p + "hc2.in"]), w[p + "norm2"], eps)
            xs = write_streams(xs, w[p + "hc2.mix"], w[p + "hc2.out"], routed_experts(h, sub(w, p + "mlp."), L["mlp"]))
        if trace is not None:
            trace.append(sum(xs))
    return offset_norm(sum(xs), w["final.norm"], eps) @ w["head"].T
