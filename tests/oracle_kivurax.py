"""Plain float64 restatement of the Kivurax design, one function per mechanism, written from the design's equations.  It shares no code with
the package; it is slow on purpose (explicit loops over tokens and heads) and runs on the CPU with numpy alone.

Notation: h [T, W] is a sublayer's input, weights are [out, in] and applied as h @ w.T; `w` dictionaries hold a sublayer's tensors under
their checkpoint names with the prefix removed ("q", "i.b", "left.q.norm", "e0.gate", ...).  Every function takes one whole sequence whose
first token has position 0."""
import math

import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm(x, w, eps):
    return unit_rms(x, eps) * w


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


# ----------------------------------------------------------------------------------------------------------- matrix memory
def memory_gates(h, w, cap):
    """(log input gate, log forget gate), [T, heads] each."""
    i = cap * np.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = -softplus(-cap * np.tanh((h @ w["f"].T + w["f.b"]) / cap))
    return i, f


def memory_read(S, n, q, m):
    return S.T @ q / (max(abs(n @ q), math.exp(-m)) + 1e-6)


def matrix_memory(h, w, c, eps):
    """mLSTM: a key-value matrix and a key sum per head, exponential gates, everything relative to a running maximum of the log gates."""
    T = h.shape[0]
    H, d, dv = c["heads"], c["dim"], c["vdim"]
    q = (h @ w["q"].T).reshape(T, H, d) * d ** -0.5
    k, v = (h @ w["k"].T).reshape(T, H, d), (h @ w["v"].T).reshape(T, H, dv)
    i, f = memory_gates(h, w, c["gate_cap"])
    o = np.zeros((T, H, dv))
    for a in range(H):
        S, n, m = np.zeros((d, dv)), np.zeros(d), 0.0
        for t in range(T):
            new = max(f[t, a] + m, i[t, a])
            keep, add = math.exp(f[t, a] + m - new), math.exp(i[t, a] - new)
            S = keep * S + add * np.outer(k[t, a], v[t, a])
            n = keep * n + add * k[t, a]
            m = new
            o[t, a] = memory_read(S, n, q[t, a], m)
    o = unit_rms(o, eps).reshape(T, H * dv) * w["norm"]
    return (o * sigmoid(h @ w["g"].T)) @ w["o"].T


# ----------------------------------------------------------------------------------------------------------- gated delta rule
def short_conv(x, taps):
    """x [T, C], taps [C, K]; the last column is the current token's."""
    T, K = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for t in range(T):
        for j in range(K):
            if t - j >= 0:
                y[t] += taps[:, K - 1 - j] * x[t - j]
    return y


def delta_decay(h, w):
    return np.exp(-np.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))


def delta_rule(h, w, c, eps):
    T = h.shape[0]
    H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(short_conv(h @ w[n].T, w[n + ".conv"])) for n in "qkv")
    q, k, v = q.reshape(T, G, d), k.reshape(T, G, d), v.reshape(T, H, dv)
    unit = lambda x: x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)
    q, k = unit(q) * d ** -0.5, unit(k)
    beta, g = sigmoid(h @ w["b"].T), delta_decay(h, w)
    o = np.zeros((T, H, dv))
    for a in range(H):
        S, b = np.zeros((d, dv)), a // (H // G)
        for t in range(T):
            S = g[t, a] * S
            u = beta[t, a] * (v[t, a] - S.T @ k[t, b])
            S = S + np.outer(k[t, b], u)
            o[t, a] = S.T @ q[t, b]
    o = norm(o, w["norm"], eps) * silu(h @ w["g"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ w["o"].T


# ----------------------------------------------------------------------------------------------------------- attention
def pair_frequencies(rot):
    """(frequency per pair, factor on cos and sin)."""
    n, base, y = rot["dims"], rot["base"], rot.get("scaling")
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    if not y:
        return f, 1.0
    where = lambda turns: n * math.log(y["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(where(y["fast"])), 0), min(math.ceil(where(y["slow"])), n - 1)
    ramp = np.array([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(n // 2)])
    return f / y["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(y["factor"]) + 1.0


def turn_pairs(x, rot):
    """x [T, heads, d] by token positions; dimensions 2i and 2i + 1 of the first rot.dims turn together."""
    f, amp = pair_frequencies(rot)
    y = x.copy()
    for p in range(x.shape[0]):
        for i in range(rot["dims"] // 2):
            c, s = amp * math.cos(p * f[i]), amp * math.sin(p * f[i])
            u, v = x[p, :, 2 * i], x[p, :, 2 * i + 1]
            y[p, :, 2 * i] = u * c - v * s
            y[p, :, 2 * i + 1] = v * c + u * s
    return y


def window_keys(i, size):
    return list(range(max(0, i - size + 1), i + 1))


def softmax_plus_one(s):
    """exp(s) / (1 + sum exp(s))."""
    m = max(s.max(), 0.0)
    e = np.exp(s - m)
    return e / (math.exp(-m) + e.sum())


def key_value_attention(h, w, c, eps):
    """Windowed grouped-query attention whose values are the projected keys, ahead of norm and rotation."""
    T = h.shape[0]
    H, G, d = c["heads"], c["kv_heads"], c["dim"]
    v = (h @ w["k"].T).reshape(T, G, d)
    q = turn_pairs(norm((h @ w["q"].T).reshape(T, H, d), w["q.norm"], eps), c["rot"])
    k = turn_pairs(norm(v, w["k.norm"], eps), c["rot"])
    out = np.zeros((T, H, d))
    for i in range(T):
        js = window_keys(i, c["mask"]["size"])
        for a in range(H):
            g = a // (H // G)
            out[i, a] = softmax_plus_one(k[js, g] @ q[i, a] * c["scale"]) @ v[js, g]
    return out.reshape(T, H * d) @ w["o"].T


# ----------------------------------------------------------------------------------------------------------- gated linear unit recurrence
def block_product(u, w):
    """u [T, B n] cut into B parts, w [B, n, n] one matrix per part."""
    B, n = w.shape[0], w.shape[1]
    return np.concatenate([u[:, b * n:(b + 1) * n] @ w[b].T for b in range(B)], 1)


def recurrent_block(h, w, c):
    """Griffin's block: a convolved branch through a real-gated diagonal recurrence, times a gelu branch."""
    T = h.shape[0]
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = short_conv(h @ w["x"].T + w["x.b"], w["conv"]) + w["conv.b"]
    r = sigmoid(block_product(u, w["ra"]) + w["ra.b"].reshape(-1))
    i = sigmoid(block_product(u, w["ri"]) + w["ri.b"].reshape(-1))
    la = -8.0 * r * softplus(w["lam"])
    S, out = np.zeros(c["width"]), np.zeros((T, c["width"]))
    for t in range(T):
        S = np.exp(la[t]) * S + np.sqrt(-np.expm1(2.0 * la[t])) * i[t] * u[t]
        out[t] = S * y[t]
    return out @ w["o"].T


def parallel(h, w, c, eps):
    return (c["left_scale"] * key_value_attention(h, sub(w, "left."), c["left"], eps)
            + c["right_scale"] * recurrent_block(h, sub(w, "right."), c["right"]))


# ----------------------------------------------------------------------------------------------------------- feed-forward
def dense(h, w):
    return (silu(h @ w["gate"].T + w["gate.b"]) * (h @ w["up"].T + w["up.b"])) @ w["down"].T + w["down.b"]


def choose(z, top):
    """[(expert, weight)] of one token's router logits."""
    s = sigmoid(z)
    return [(int(e), s[e]) for e in np.argsort(-s, kind="stable")[:top]]


def expert(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def routed_experts(h, w, c):
    """The weight multiplies what an expert reads."""
    z, y = h @ w["router"].T, np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in choose(z[t], c["router"]["top"]):
            y[t] += expert(p * h[t], sub(w, f"e{e}."))
    return y


def feed_forward(h, w, c):
    return dense(h, w) if c["kind"] == "dense" else routed_experts(h, w, c)


# ----------------------------------------------------------------------------------------------------------- layers
def mixer(kind, h, w, c, eps):
    if kind == "mlstm":
        return matrix_memory(h, w, c, eps)
    if kind == "parallel":
        return parallel(h, w, c, eps)
    if kind == "delta":
        return delta_rule(h, w, c, eps)
    raise ValueError(kind)


def forward(cfg, weights, tokens, trace=None):
    """Logits [T, vocab] of one sequence; trace (a list) collects the residual stream after every layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][np.asarray(tokens)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + m * norm(mixer(L["type"], x, sub(w, p + "mix."), L["mixer"], eps), w[p + "norm1"], eps)
        if L.get("mlp"):
            x = x + m * norm(feed_forward(x, sub(w, p + "mlp."), L["mlp"]), w[p + "norm2"], eps)
        if trace is not None:
            trace.append(x)
    return norm(x, w["final.norm"], eps) @ w["embed"].T
