"""Plain float64 implementation of the Tazizen decoder: the oracle of the tests.

Whole sequences, no cache, no batching, one function per mechanism, numpy only; it shares no code
with the package.  ``weights`` maps tensor names to arrays, ``config`` is the parsed config.json.

The residual is a set of S streams X_1 .. X_S (rows of ``X`` [T, S, width]), all E[token] at the start.  A sublayer f with
its norm n and its connection (a [S], B [S, S], c [S]) acts on all of them at once:

    u = sum_s a_s X_s        y = f(n(u))        X'_t = sum_s B_st X_s + c_t y        n(u) = u / sqrt(mean(u^2) + eps) * (1 + w)

A layer is two such sublayers, a mixer and a feed-forward (or the mixer alone); a run of layers may be passed several
times.  logits = W_head n_final(sum_s X_s).

Mixers: "attention" (grouped heads, half rotation with frequencies stretched for long contexts, q and k over their root
mean square after the rotation, a sliding window, one added to the softmax's denominator, a gate per output element) and
"latent_attention" (keys and values from a narrow latent, one rotated key part for all heads, a sliding window).
Feed-forward: gated experts chosen inside the best groups, and a gated one that every token uses, times a gate per token.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np

F = np.float64


# ----------------------------------------------------------------------------------------------- norms and activations
def unit_rms(x: np.ndarray, eps: float) -> np.ndarray:
    x = np.asarray(x, dtype=F)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def norm_around_one(x: np.ndarray, w: np.ndarray, eps: float) -> np.ndarray:
    return unit_rms(x, eps) * (1.0 + np.asarray(w, dtype=F))


def sigmoid(z: np.ndarray) -> np.ndarray:
    return np.exp(-np.logaddexp(0.0, -np.asarray(z, dtype=F)))


def silu(z: np.ndarray) -> np.ndarray:
    return z * sigmoid(z)


# ----------------------------------------------------------------------------------------------- residual streams
def streams_in(X: np.ndarray, a: np.ndarray) -> np.ndarray:
    """[T, S, width] -> [T, width]: what a sublayer's norm reads."""
    return np.einsum("tsw,s->tw", np.asarray(X, dtype=F), np.asarray(a, dtype=F))


def streams_out(X: np.ndarray, y: np.ndarray, mix: np.ndarray, out: np.ndarray) -> np.ndarray:
    """X'_t = sum_s mix[s, t] X_s + out[t] y (mix is indexed [from, to])."""
    mixed = np.einsum("tsw,sr->trw", np.asarray(X, dtype=F), np.asarray(mix, dtype=F))
    return mixed + np.asarray(out, dtype=F)[None, :, None] * y[:, None, :]


# ----------------------------------------------------------------------------------------------- rotation
def frequencies(rot: dict) -> np.ndarray:
    """dims/2 frequencies.  With a scaling {factor, original, fast, slow}: those that turn more than ``fast`` times over
    ``original`` positions stay, those that turn less than ``slow`` times are divided by ``factor``, a ramp in between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    half = dims // 2
    f = np.array([base ** (-2.0 * i / dims) for i in range(half)], dtype=F)
    s = rot.get("scaling")
    if s is None:
        return f
    def place(turns: float) -> float:
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(place(s["fast"])), 0)
    hi = min(math.ceil(place(s["slow"])), dims - 1)
    out = np.zeros(half, dtype=F)
    for i in range(half):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / s["factor"] * ramp + f[i] * (1.0 - ramp)
    return out


def amplitude(rot: dict) -> float:
    s = rot.get("scaling")
    return 1.0 if s is None else 0.1 * math.log(s["factor"]) + 1.0


def rotate_halves(x: np.ndarray, rot: dict, first_position: int = 0) -> np.ndarray:
    """x [T, ..., d]: element i < dims/2 is paired with i + dims/2; elements from dims on pass unchanged."""
    dims = int(rot["dims"])
    half = dims // 2
    out = np.array(x, dtype=F)
    if half == 0:
        return out
    f, m = frequencies(rot), amplitude(rot)
    for t in range(x.shape[0]):
        angle = (first_position + t) * f
        cos, sin = m * np.cos(angle), m * np.sin(angle)
        u, v = np.array(x[t, ..., :half], dtype=F), np.array(x[t, ..., half:dims], dtype=F)
        out[t, ..., :half] = u * cos - v * sin
        out[t, ..., half:dims] = v * cos + u * sin
    return out


# ----------------------------------------------------------------------------------------------- attention
def window_attention(q: np.ndarray, k: np.ndarray, v: np.ndarray, scale: float, window: Optional[int],
                     extra: float) -> np.ndarray:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; the query at i reads 0 <= i - j < window (None: all j <= i);
    ``extra`` is added to the sum of the exponentials."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), dtype=F)
    for i in range(T):
        first = 0 if window is None else max(i - window + 1, 0)
        for h in range(H):
            g = h // (H // G)
            s = (k[first:i + 1, g] @ q[i, h]) * scale
            top = max(s.max(), 0.0)
            p = np.exp(s - top)
            out[i, h] = (p @ v[first:i + 1, g]) / (p.sum() + extra * math.exp(-top))
    return out


def attention(h: np.ndarray, W: Dict[str, np.ndarray], p: str, m: dict, eps: float) -> np.ndarray:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, d)
    k = (h @ W[p + "k"].T).reshape(T, G, d)
    v = (h @ W[p + "v"].T).reshape(T, G, dv)
    q, k = unit_rms(rotate_halves(q, m["rot"]), eps), unit_rms(rotate_halves(k, m["rot"]), eps)
    window = (m.get("mask") or {}).get("size")
    o = window_attention(q, k, v, m["scale"], window, 1.0).reshape(T, H * dv)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def latent_attention(h: np.ndarray, W: Dict[str, np.ndarray], p: str, m: dict, eps: float) -> np.ndarray:
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (unit_rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T
    q = q.reshape(T, H, d + r)
    q = np.concatenate([q[..., :d], rotate_halves(q[..., d:], m["rot"])], axis=-1)
    down = h @ W[p + "dkv"].T
    c = unit_rms(down[:, :rank], eps) * W[p + "dkv.norm"]
    shared = rotate_halves(down[:, rank:], m["rot"])
    k = np.concatenate([(c @ W[p + "uk"].T).reshape(T, H, d), np.repeat(shared[:, None, :], H, axis=1)], axis=-1)
    v = (c @ W[p + "uv"].T).reshape(T, H, dv)
    window = (m.get("mask") or {}).get("size")
    return window_attention(q, k, v, m["scale"], window, 0.0).reshape(T, H * dv) @ W[p + "o"].T


# ----------------------------------------------------------------------------------------------- feed-forward
def gated(h: np.ndarray, W: Dict[str, np.ndarray], p: str) -> np.ndarray:
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def group_values(choice: np.ndarray, count: int) -> np.ndarray:
    """[outputs] -> [count]: the sum of each group's two largest choice scores (of the only one in a group of one)."""
    return np.array([np.sort(part)[::-1][:2].sum() for part in choice.reshape(count, -1)])


def route(h: np.ndarray, router: np.ndarray, correction: np.ndarray, top: int, count: int, keep: int, scale: float,
          margins: Optional[List[float]] = None, choices: Optional[np.ndarray] = None):
    """-> (ids [T, top], weights [T, top]).  ``margins`` receives per token how far the choice is from another one.
    ``choices`` [T, top]: these experts instead, with their own scores; a margin is then negative by how much the choice
    scores (or group values) would have to move for it."""
    s = sigmoid(h @ router.T)
    ids, weights = [], []
    for t in range(h.shape[0]):
        choice = s[t] + correction
        per = choice.size // count
        values = group_values(choice, count)
        order = list(np.argsort(-values, kind="stable"))
        if choices is not None:
            taken = {int(e) // per for e in choices[t]}
            order.sort(key=lambda g: g not in taken)               # the groups of the experts taken first
        allowed = np.full(choice.size, -np.inf)
        for g in order[:keep]:
            allowed[g * per:(g + 1) * per] = choice[g * per:(g + 1) * per]
        chosen = np.argsort(-allowed, kind="stable")[:top] if choices is None else np.asarray(choices[t], dtype=np.int64)
        ids.append(chosen)
        w = s[t, chosen]
        weights.append(w / (w.sum() + 1e-20) * scale)
        if margins is not None:
            gap = np.inf if keep >= count else values[order[:keep]].min() - values[order[keep:]].max()
            left = np.delete(allowed, chosen)
            if left.size and np.isfinite(left.max()):
                gap = min(gap, allowed[chosen].min() - left.max())
            margins.append(float(gap))
    return np.array(ids), np.array(weights)


def experts(h: np.ndarray, W: Dict[str, np.ndarray], p: str, mlp: dict, margins: Optional[List[float]] = None,
            choices: Optional[np.ndarray] = None) -> np.ndarray:
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    ids, weights = route(h, W[p + "router"], W[p + "correction"], r["top"], groups["count"], groups["keep"], r.get("scale", 1.0),
                         margins, choices)
    out = np.zeros_like(h)
    for e in range(r["experts"]):
        rows, places = np.nonzero(ids == e)
        if rows.size:
            out[rows] += weights[rows, places][:, None] * gated(h[rows], W, f"{p}e{e}.")
    if mlp.get("shared") is not None:
        out = out + sigmoid(h @ W[p + "shared.sg"].T) * gated(h, W, p + "shared.")
    return out


# ----------------------------------------------------------------------------------------------- the model
def run_order(config: dict) -> List[int]:
    n, loop = len(config["layers"]), config.get("loop")
    if loop is None:
        return list(range(n))
    once = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + once * loop["times"] + list(range(loop["stop"], n))


def forward(config: dict, weights: Dict[str, np.ndarray], tokens, return_layers: bool = False, margins: Optional[list] = None,
            choices: Optional[list] = None):
    """Logits [T, vocab] of a whole sequence (and, on request, the sum of the streams after every layer run [runs, T,
    width]).  ``margins``: a list that receives the [T] choice margins of every routed layer run; ``choices``: the experts
    every routed layer run takes, [T, top] each."""
    W = {name: np.asarray(t, dtype=F) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    X = np.repeat(W["embed"][np.asarray(tokens)][:, None, :], config["streams"], axis=1)
    kept, routed = [], 0
    for n in run_order(config):
        layer, p = config["layers"][n], f"l{n}."
        mixer = {"attention": attention, "latent_attention": latent_attention}[layer["type"]]
        y = mixer(norm_around_one(streams_in(X, W[p + "hc1.in"]), W[p + "norm1"], eps), W, p + "mix.", layer["mixer"], eps)
        X = streams_out(X, y, W[p + "hc1.mix"], W[p + "hc1.out"])
        if layer.get("mlp") is not None:
            found = None if margins is None else []
            y = experts(norm_around_one(streams_in(X, W[p + "hc2.in"]), W[p + "norm2"], eps), W, p + "mlp.", layer["mlp"], found,
                        None if choices is None else choices[routed])
            routed += 1
            X = streams_out(X, y, W[p + "hc2.mix"], W[p + "hc2.out"])
            if margins is not None:
                margins.append(np.array(found))
        kept.append(X.sum(axis=1))
    logits = norm_around_one(X.sum(axis=1), W["final.norm"], eps) @ W["head"].T
    return (logits, np.stack(kept)) if return_layers else logits
