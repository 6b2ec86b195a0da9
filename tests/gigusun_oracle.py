"""Plain statement of the Gigusun decoder in float64 numpy: one function per mechanism, token by token,
no caches and no chunking.  It shares no code with the product path; the tests compare the library with
it.  Weights are a dict of float64 arrays under the model's tensor names, the configuration is the parsed
config.json."""
from __future__ import annotations

import numpy as np


def rms(x: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(x):
    return 0.5 * (1.0 + np.tanh(0.5 * x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def centred_rms_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    """RMS norm whose gain is stored around zero."""
    return rms(x, eps) * (1.0 + w)


def embed(tokens, table: np.ndarray, positions: np.ndarray, gain: np.ndarray, eps: float, first: int = 0) -> np.ndarray:
    tokens = np.asarray(tokens)
    return centred_rms_norm(table[tokens] + positions[first:first + len(tokens)], gain, eps)


def poly_norm(z: np.ndarray, coefficients: np.ndarray, eps: float) -> np.ndarray:
    a, b, c, e = coefficients
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def window_scores(q: np.ndarray, k: np.ndarray, i: int, visible: np.ndarray, scale: float, softcap: float,
                  r1: float, r2: float) -> np.ndarray:
    """Scores of the query at position i against the visible key positions."""
    s = (k[visible] @ q) * scale
    s = softcap * np.tanh(s / softcap)
    return s - r1 * np.log1p(r2 * (i - visible))


def visible_keys(i: int, size: int, keep_first: int) -> np.ndarray:
    j = np.arange(i + 1)
    return j[(i - j < size) | (j < keep_first)]


def softmax_with_sink(s: np.ndarray) -> np.ndarray:
    m = max(0.0, float(s.max()))
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum())


def attention(q, k, v, *, scale, softcap, r1, r2, size, keep_first) -> np.ndarray:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]."""
    T, H = q.shape[:2]
    group = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        seen = visible_keys(i, size, keep_first)
        for h in range(H):
            s = window_scores(q[i, h], k[:, h // group], i, seen, scale, softcap, r1[h], r2[h])
            out[i, h] = softmax_with_sink(s) @ v[seen, h // group]
    return out


def attention_mixer(h: np.ndarray, w: dict, p: str, m: dict, eps: float) -> np.ndarray:
    T = len(h)
    H, G = m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].T).reshape(T, H, m["dim"])
    k = (h @ w[p + "k"].T).reshape(T, G, m["dim"])
    v = (h @ w[p + "v"].T).reshape(T, G, m["vdim"])
    q, k = rms(q, eps) * w[p + "q.norm"], rms(k, eps) * w[p + "k.norm"]
    o = attention(q, k, v, scale=m["scale"], softcap=m["softcap"], r1=w[p + "r1"], r2=w[p + "r2"],
                  size=m["mask"]["size"], keep_first=m["mask"]["keep_first"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].T


def gated_linear_attention(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, dim], v [T, H, vdim] -> (o [T, H, vdim], final state [H, dim, vdim])."""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2])) if state is None else state.copy()
    out = np.zeros(v.shape)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out, S


def gla_decay(h: np.ndarray, w: dict, p: str, m: dict) -> np.ndarray:
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return np.exp(-softplus(-z) / m["tau"]).reshape(len(h), m["heads"], m["dim"])


def gla_mixer(h: np.ndarray, w: dict, p: str, m: dict, eps: float) -> np.ndarray:
    T, H = len(h), m["heads"]
    q = (h @ w[p + "q"].T).reshape(T, H, m["dim"]) * m["dim"] ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, m["dim"])
    v = (h @ w[p + "v"].T).reshape(T, H, m["vdim"])
    o, _ = gated_linear_attention(q, k, v, gla_decay(h, w, p, m))
    o = rms(o, eps) * w[p + "norm"]
    return (o.reshape(T, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def causal_convolution(x: np.ndarray, taps: np.ndarray) -> np.ndarray:
    """x [T, channels], taps [channels, n], the last tap meets the current token."""
    n = taps.shape[1]
    padded = np.concatenate([np.zeros((n - 1, x.shape[1])), x])
    return sum(padded[j:j + len(x)] * taps[:, j] for j in range(n))


def unit_vectors(x: np.ndarray) -> np.ndarray:
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def gated_delta_rule(q, k, v, beta, g, state=None):
    """q, k [T, G, dim], v [T, H, vdim], beta, g [T, H] -> (o [T, H, vdim], state [H, dim, vdim])."""
    T, H, vdim = v.shape
    group = H // k.shape[1]
    S = np.zeros((H, k.shape[2], vdim)) if state is None else state.copy()
    out = np.zeros((T, H, vdim))
    for t in range(T):
        for h in range(H):
            key, query = k[t, h // group], q[t, h // group]
            S[h] *= g[t, h]
            u = beta[t, h] * (v[t, h] - S[h].T @ key)
            S[h] += np.outer(key, u)
            out[t, h] = S[h].T @ query
    return out, S


def delta_gates(h: np.ndarray, w: dict, p: str):
    beta = sigmoid(h @ w[p + "b"].T)
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    return beta, g


def delta_mixer(h: np.ndarray, w: dict, p: str, m: dict, eps: float) -> np.ndarray:
    T, H, G = len(h), m["heads"], m["kv_heads"]
    q, k, v = (silu(causal_convolution(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q = unit_vectors(q.reshape(T, G, m["dim"])) * m["dim"] ** -0.5
    k = unit_vectors(k.reshape(T, G, m["dim"]))
    beta, g = delta_gates(h, w, p)
    o, _ = gated_delta_rule(q, k, v.reshape(T, H, m["vdim"]), beta, g)
    o = rms(o, eps) * w[p + "norm"] * silu((h @ w[p + "g"].T).reshape(T, H, m["vdim"]))
    return o.reshape(T, -1) @ w[p + "o"].T


MIXERS = {"attention": attention_mixer, "gla": gla_mixer, "delta": delta_mixer}


def feed_forward(h: np.ndarray, w: dict, p: str, eps: float) -> np.ndarray:
    return poly_norm(h @ w[p + "up"].T, w[p + "act"], eps) @ w[p + "down"].T


def forward(config: dict, w: dict, tokens, residuals: list | None = None) -> np.ndarray:
    """Logits [T, vocab] of one sequence; `residuals` collects the stream after every layer."""
    eps = config["norm"]["eps"]
    x = embed(tokens, w["embed"], w["pos"], w["embed.norm"], eps)
    for i, layer in enumerate(config["layers"]):
        h = centred_rms_norm(x, w[f"l{i}.norm1"], eps)
        x = x + MIXERS[layer["type"]](h, w, f"l{i}.mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + feed_forward(centred_rms_norm(x, w[f"l{i}.norm2"], eps), w, f"l{i}.mlp.", eps)
        if residuals is not None:
            residuals.append(x.copy())
    return centred_rms_norm(x, w["final.norm"], eps) @ w["head"].T
