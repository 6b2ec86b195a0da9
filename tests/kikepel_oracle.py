"""Plain statement of the Kikepel decoder in float64 numpy: one function per mechanism, query by query, no
caches, no absorbed products and no grouping of tokens.  It shares no code with the product path; the tests
compare the library with it.  Weights are a dict of float64 arrays under the model's tensor names, the
configuration is the parsed config.json."""
from __future__ import annotations

import numpy as np


def rms(x: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    centred = x - np.mean(x, axis=-1, keepdims=True)
    return rms(centred, eps) * w


def sigmoid(x):
    return 0.5 * (1.0 + np.tanh(0.5 * x))


# ---------------------------------------------------------------- latent attention
def latent_rows(h: np.ndarray, down: np.ndarray, gain: np.ndarray, eps: float) -> np.ndarray:
    """The normalised latent of each token: [T, rank]."""
    return rms(h @ down.T, eps) * gain


def visible_keys(i: int, size: int) -> np.ndarray:
    return np.arange(max(0, i - size + 1), i + 1)


def softmax(s: np.ndarray, sink: float | None) -> np.ndarray:
    """Weights of the keys; a sink has a place in the denominator and none among the weights."""
    m = float(s.max()) if sink is None else max(float(s.max()), sink)
    e = np.exp(s - m)
    return e / (e.sum() + (0.0 if sink is None else np.exp(sink - m)))


def attention(q, k, v, *, scale: float, size: int, sink=None) -> np.ndarray:
    """q, k [T, H, dim], v [T, H, vdim], sink [H] or None -> [T, H, vdim]."""
    T, H = q.shape[:2]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        seen = visible_keys(i, size)
        for h in range(H):
            weights = softmax((k[seen, h] @ q[i, h]) * scale, None if sink is None else float(sink[h]))
            out[i, h] = weights @ v[seen, h]
    return out


def latent_attention_mixer(h: np.ndarray, w: dict, p: str, m: dict, eps: float, sinks: bool) -> np.ndarray:
    T, H = len(h), m["heads"]
    q = latent_rows(h, w[p + "dq"], w[p + "dq.norm"], eps) @ w[p + "uq"].T
    c = latent_rows(h, w[p + "dkv"], w[p + "dkv.norm"], eps)
    k, v = c @ w[p + "uk"].T, c @ w[p + "uv"].T
    o = attention(q.reshape(T, H, m["dim"]), k.reshape(T, H, m["dim"]), v.reshape(T, H, m["vdim"]), scale=m["scale"],
                  size=m["mask"]["size"], sink=w[p + "sink"] if sinks else None)
    return o.reshape(T, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forwards
def dense(h: np.ndarray, w: dict, p: str) -> np.ndarray:
    gate = np.maximum(h @ w[p + "gate"].T + w[p + "gate.b"], 0.0)
    return (gate * (h @ w[p + "up"].T + w[p + "up.b"])) @ w[p + "down"].T + w[p + "down.b"]


def expert(h: np.ndarray, gate: np.ndarray, up: np.ndarray, down: np.ndarray, limit: float) -> np.ndarray:
    g = np.minimum(gate @ h, limit)
    u = np.clip(up @ h, -limit, limit)
    return down @ (g * sigmoid(1.702 * g) * (u + 1.0))


def route(h: np.ndarray, router: np.ndarray, top: int):
    """One token's experts, best first, and their weights."""
    scores = sigmoid(router @ h)
    chosen = np.argsort(-scores, kind="stable")[:top]
    return chosen, scores[chosen]


def mixture(h: np.ndarray, w: dict, p: str, mlp: dict) -> np.ndarray:
    out = np.zeros_like(h)
    for t, row in enumerate(h):
        for e, weight in zip(*route(row, w[p + "router"], mlp["router"]["top"])):
            out[t] += expert(weight * row, w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"], mlp["expert"]["limit"])
    return out


def feed_forward(h: np.ndarray, w: dict, p: str, mlp: dict) -> np.ndarray:
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp)


# ---------------------------------------------------------------- the model
def capped_logits(h: np.ndarray, head: np.ndarray, scale: float, softcap: float) -> np.ndarray:
    return softcap * np.tanh((h @ head.T) * scale / softcap)


def forward(config: dict, w: dict, tokens, residuals: list | None = None) -> np.ndarray:
    """Logits [T, vocab] of one sequence; `residuals` collects the stream after every layer."""
    eps = config["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    for i, layer in enumerate(config["layers"]):
        mixed = latent_attention_mixer(x, w, f"l{i}.mix.", layer["mixer"], eps, sinks=layer["type"] == "latent_attention")
        x = x + layer_norm(mixed, w[f"l{i}.norm1"], eps)
        if layer["mlp"] is not None:
            x = x + layer_norm(feed_forward(x, w, f"l{i}.mlp.", layer["mlp"]), w[f"l{i}.norm2"], eps)
        if residuals is not None:
            residuals.append(x.copy())
    return capped_logits(layer_norm(x, w["final.norm"], eps), w["head"], config["logit_scale"], config["logit_softcap"])
