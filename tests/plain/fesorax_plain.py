"""Plain float64 implementation of the Fesorax decoder: the oracle of the tests.

Whole sequences, no cache, no batching, one function per mechanism, numpy only; it shares no code
with the package.  ``weights`` maps tensor names to arrays, ``config`` is the parsed config.json.

    x = E[token] * s                                    (s = embedding.scale)
    a layer:  x <- n1(a x + mixer(x));  x <- n2(a x + ff(x))     n(x) = x / sqrt(mean(x^2) + eps) * w, a = postln_alpha
    logits = W_head n_final(x)

Mixers: "attention" (unit-RMS q and k per head, a learned bias by distance, a window beside which the first tokens
stay visible, one gate per head, keys and values that may be an earlier layer's), "mlstm" (a matrix memory with
exponential input gates, a normaliser and a running maximum).  Feed-forward: a mixture of clamped gated experts with
logistic scores that multiply the experts' inputs, and one that every token uses.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np

F = np.float64


def unit_rms(x: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def rms_norm(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    return unit_rms(x.astype(F), eps) * weight.astype(F)


def sigmoid(z: np.ndarray) -> np.ndarray:
    return np.exp(-np.logaddexp(0.0, -z))


def log_sigmoid(z: np.ndarray) -> np.ndarray:
    return -np.logaddexp(0.0, -z)


def soft_cap(z: np.ndarray, cap: float) -> np.ndarray:
    return cap * np.tanh(z / cap)


def distance_bucket(n: int, rows: int, far: float) -> int:
    """Distances below rows/2 have a row each; beyond, rows are spaced evenly in the logarithm up to ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


def sees(i: int, j: int, window: Optional[int], keep: int) -> bool:
    """Whether the query at i may read the key at j: the last ``window`` positions (None: all) and the first ``keep``."""
    return j <= i and (window is None or i - j < window or j < keep)


def attend(q: np.ndarray, k: np.ndarray, v: np.ndarray, scale: float, bias: np.ndarray, far: float,
           window: Optional[int], keep: int) -> np.ndarray:
    """q [T, H, d], k [T, G, d], v [T, G, dv]; ``bias`` [rows, H] by the bucket of i - j, not scaled.  [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=F)
    buckets = np.array([distance_bucket(n, bias.shape[0], far) for n in range(T)])
    for i in range(T):
        js = np.array([j for j in range(i + 1) if sees(i, j, window, keep)])
        for h in range(H):
            g = h // (H // G)
            s = (k[js, g] @ q[i, h]) * scale + bias[buckets[i - js], h]
            w = np.exp(s - s.max())
            out[i, h] = (w / w.sum()) @ v[js, g]
    return out


def attention_mixer(h: np.ndarray, W: Dict[str, np.ndarray], p: str, m: dict, eps: float, kept: Dict[int, tuple],
                    layer: int) -> np.ndarray:
    """``kept``: layer -> (keys after their norm, values) of this sequence."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ W[p + "q"].astype(F).T).reshape(T, H, d), eps)
    if m.get("kv_from") is None:
        k = unit_rms((h @ W[p + "k"].astype(F).T).reshape(T, G, d), eps)
        v = (h @ W[p + "v"].astype(F).T).reshape(T, G, dv)
        kept[layer] = (k, v)
    else:
        k, v = kept[m["kv_from"]]
    mask = m.get("mask") or {}
    a = attend(q, k, v, m["scale"], W[p + "rel"].astype(F), float(m["bias_max"]), mask.get("size"), mask.get("keep_first") or 0)
    gate = sigmoid(h @ W[p + "g"].astype(F).T)                       # one number per head
    return (a * gate[:, :, None]).reshape(T, H * dv) @ W[p + "o"].astype(F).T


def mlstm_memory(q: np.ndarray, k: np.ndarray, v: np.ndarray, log_i: np.ndarray, log_f: np.ndarray) -> np.ndarray:
    """One head: q, k [T, d], v [T, dv], log gates [T].  The maximum starts at 0."""
    T, d = q.shape
    S, n, m = np.zeros((d, v.shape[1]), dtype=F), np.zeros(d, dtype=F), 0.0
    out = np.zeros((T, v.shape[1]), dtype=F)
    for t in range(T):
        m_new = max(log_f[t] + m, log_i[t])
        keep, write = math.exp(log_f[t] + m - m_new), math.exp(log_i[t] - m_new)
        S = keep * S + write * np.outer(k[t], v[t])
        n = keep * n + write * k[t]
        m = m_new
        out[t] = (S.T @ q[t]) / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6)
    return out


def mlstm_gates(h: np.ndarray, W: Dict[str, np.ndarray], p: str, cap: float):
    """(log input gate, log forget gate), each [T, heads]."""
    i = soft_cap(h @ W[p + "i"].astype(F).T + W[p + "i.b"].astype(F), cap)
    f = log_sigmoid(soft_cap(h @ W[p + "f"].astype(F).T + W[p + "f.b"].astype(F), cap))
    return i, f


def mlstm_mixer(h: np.ndarray, W: Dict[str, np.ndarray], p: str, m: dict, eps: float) -> np.ndarray:
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].astype(F).T).reshape(T, H, d) * d ** -0.5
    k = (h @ W[p + "k"].astype(F).T).reshape(T, H, d)
    v = (h @ W[p + "v"].astype(F).T).reshape(T, H, dv)
    log_i, log_f = mlstm_gates(h, W, p, m["gate_cap"])
    o = np.stack([mlstm_memory(q[:, n], k[:, n], v[:, n], log_i[:, n], log_f[:, n]) for n in range(H)], axis=1)
    o = unit_rms(o, eps).reshape(T, H * dv) * W[p + "norm"].astype(F) * sigmoid(h @ W[p + "g"].astype(F).T)
    return o @ W[p + "o"].astype(F).T


def expert(h: np.ndarray, W: Dict[str, np.ndarray], p: str, limit: float) -> np.ndarray:
    g = np.minimum(h @ W[p + "gate"].astype(F).T, limit)
    u = np.clip(h @ W[p + "up"].astype(F).T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].astype(F).T


def route(h: np.ndarray, W: Dict[str, np.ndarray], p: str, top: int, margins: Optional[list] = None,
          choice: Optional[np.ndarray] = None):
    """(chosen experts [T, top], their logistic scores [T, top]).  ``margins`` collects, per token, how far the last
    chosen logit lies above the first one left out.  ``choice`` [T, top]: take these experts instead (another program's
    choice, whose rounding may have turned a close call); ``margins`` then collects how far its worst expert lies below
    the best one it left out, as a negative number, or the distance as above where it took the largest."""
    z = h @ W[p + "router"].astype(F).T
    ids = np.argsort(-z, axis=-1, kind="stable")[:, :top] if choice is None else np.asarray(choice)
    if margins is not None:
        left_out = z.copy()
        np.put_along_axis(left_out, ids, -np.inf, axis=-1)
        margins.append(np.take_along_axis(z, ids, axis=-1).min(axis=-1) - left_out.max(axis=-1))
    return ids, sigmoid(np.take_along_axis(z, ids, axis=-1))


def moe_ff(h: np.ndarray, W: Dict[str, np.ndarray], p: str, mlp: dict, margins: Optional[list] = None,
           choice: Optional[np.ndarray] = None) -> np.ndarray:
    """The weight multiplies the expert's input."""
    ids, w = route(h, W, p, mlp["router"]["top"], margins, choice)
    out = np.zeros(h.shape, dtype=F)
    for e in range(mlp["router"]["experts"]):
        for j in range(ids.shape[1]):
            mine = np.nonzero(ids[:, j] == e)[0]
            if mine.size:
                out[mine] += expert(h[mine] * w[mine, j][:, None], W, f"{p}e{e}.", mlp["expert"]["limit"])
    if mlp.get("shared") is not None:
        out += expert(h, W, p + "shared.", mlp["shared"]["limit"])
    return out


def forward(config: dict, W: Dict[str, np.ndarray], tokens, streams: Optional[list] = None,
            margins: Optional[list] = None, choices: Optional[list] = None) -> np.ndarray:
    """Logits [T, vocab] of one sequence; ``streams`` collects the stream after every layer, ``margins`` every routed layer's
    distances from another choice of experts; ``choices``: per routed layer, the experts to take (see ``route``)."""
    choices = iter(choices) if choices is not None else None
    eps, alpha = config["norm"]["eps"], config["postln_alpha"]
    x = W["embed"].astype(F)[np.asarray(tokens)] * (config.get("embedding") or {}).get("scale", 1.0)
    kept: Dict[int, tuple] = {}
    for n, layer in enumerate(config["layers"]):
        p, m = f"l{n}.", layer["mixer"]
        if layer["type"] == "attention":
            y = attention_mixer(x, W, p + "mix.", m, eps, kept, n)
        elif layer["type"] == "mlstm":
            y = mlstm_mixer(x, W, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = rms_norm(alpha * x + y, W[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = rms_norm(alpha * x + moe_ff(x, W, p + "mlp.", layer["mlp"], margins, next(choices) if choices is not None else None), W[p + "norm2"], eps)
        if streams is not None:
            streams.append(x.copy())
    return rms_norm(x, W["final.norm"], eps) @ W["head"].astype(F).T
