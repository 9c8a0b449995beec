"""Pekerax, plain and slow: NumPy float64, one whole sequence at a time, no
cache (every attention position looks at its whole prefix) and the recurrence
walked token by token from a zero state, one function per mechanism.  It
shares nothing with the package: it reads config.json as a dict and
model.safetensors with its own few lines."""
import json
import math
import struct
from pathlib import Path

import numpy as np


def load(folder):
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    meta = json.loads(raw[8 : 8 + n])
    data = raw[8 + n :]
    w = {}
    for name, m in meta.items():
        if name == "__metadata__":
            continue
        lo, hi = m["data_offsets"]
        if m["dtype"] == "BF16":
            arr = (np.frombuffer(data[lo:hi], dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif m["dtype"] == "F32":
            arr = np.frombuffer(data[lo:hi], dtype="<f4").astype(np.float64)
        else:
            raise ValueError(m["dtype"])
        w[name] = arr.reshape(m["shape"])
    return w, cfg


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, dtype=np.float64)))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_norm(x, weight, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * weight


def layer_norm(x, weight, bias, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * weight + bias


# ---- attention -------------------------------------------------------------------------------------------------
def slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def window_mask(T, size=None, keep_first=0):
    """[i, j]: position i sees j."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & ((i - j < size) | (j < keep_first))
    return seen


def sink_softmax(scores, mask, sink):
    """Rows of weights over the keys; exp(sink) stands in the denominator only."""
    s = np.where(mask, scores, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def biased_attention(q, k, v, scale, mask, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    distance = np.arange(T)[:, None] - np.arange(T)[None, :]
    out = np.zeros((T, H, v.shape[-1]))
    for h, slope in enumerate(slopes(H)):
        g = h // (H // G)
        out[:, h] = sink_softmax((q[:, h] @ k[:, g].T) * scale - slope * distance, mask, sink[h]) @ v[:, g]
    return out


def mixed_values(v, v_first, lam):
    return v if v_first is None else (1.0 - lam) * v + lam * v_first


def attention(w, p, m, h, eps, v_first=None):
    """(the mixer's output, its values as projected).  ``v_first``: the values that the layer's own are mixed with, or None."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, H, d)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, G, d)
    own = h @ w[p + "v"].T
    v = mixed_values(own, v_first, float(w[p + "vmix"]) if v_first is not None else 0.0).reshape(T, G, dv)
    mask = m.get("mask") or {}
    o = biased_attention(q, k, v, m["scale"], window_mask(T, mask.get("size"), mask.get("keep_first", 0)), w[p + "sink"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T, own


# ---- the gated delta rule ----------------------------------------------------------------------------------------
def causal_conv(x, taps):
    """x [T, C], taps [C, K] (last column: the current token), zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    out = np.zeros_like(x)
    for j in range(K):
        back = K - 1 - j
        if back < T:
            out[back:] += x[: T - back] * taps[:, j]
    return out


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def delta_recurrence(q, k, v, beta, decay):
    """q, k [T, G, n], v [T, H, p], beta, decay [T, H] -> [T, H, p]."""
    T, H, P = v.shape
    G, N = k.shape[1], k.shape[2]
    out = np.zeros((T, H, P))
    S = np.zeros((H, N, P))
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] *= decay[t, h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, g])
            S[h] += np.outer(k[t, g], u)
            out[t, h] = S[h].T @ q[t, g]
    return out


def delta(w, p, m, h, eps):
    T = h.shape[0]
    H, G, n, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def short(name):
        return silu(causal_conv(h @ w[p + name].T, w[p + name + ".conv"]))

    q = unit(short("q").reshape(T, G, n)) / math.sqrt(n)
    k = unit(short("k").reshape(T, G, n))
    v = short("v").reshape(T, H, P)
    beta = sigmoid(h @ w[p + "b"].T)
    decay = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = rms_norm(delta_recurrence(q, k, v, beta, decay), w[p + "norm"], eps)
    o = o.reshape(T, H * P) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---- feed-forwards -----------------------------------------------------------------------------------------------
def clamped_gated(w, p, h, limit):
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(w, p, r, h):
    """(chosen experts [T, top], their weights [T, top], margin [T]) for every token; ``margin`` is the smallest relative
    gap between what was taken and what was not (scores of experts, scores of groups), so that tests know a close call."""
    E, top = r["experts"], r["top"]
    z = h @ w[p + "router"].T
    s = np.exp(z - z.max(axis=-1, keepdims=True))
    s = s / s.sum(axis=-1, keepdims=True)
    c = s
    margin = np.full(len(s), np.inf)
    groups = r.get("groups")
    if groups:
        per = E // groups["count"]
        gscore = s.reshape(-1, groups["count"], per).max(axis=-1)
        order = np.argsort(-gscore, axis=-1, kind="stable")
        allowed = np.zeros_like(gscore, dtype=bool)
        np.put_along_axis(allowed, order[:, : groups["keep"]], True, axis=-1)
        if groups["keep"] < groups["count"]:
            ranked = -np.sort(-gscore, axis=-1)
            margin = 1.0 - ranked[:, groups["keep"]] / ranked[:, groups["keep"] - 1]
        c = np.where(np.repeat(allowed, per, axis=-1), s, 0.0)
    chosen = np.argsort(-c, axis=-1, kind="stable")[:, :top]
    picked = np.take_along_axis(s, chosen, axis=-1)
    weights = picked / (picked.sum(axis=-1, keepdims=True) + 1e-20)
    if top < E:
        ranked = -np.sort(-c, axis=-1)
        margin = np.minimum(margin, 1.0 - ranked[:, top] / ranked[:, top - 1])
    return chosen, weights, margin


def routed(w, p, mlp, h):
    chosen, weights, _ = route(w, p, mlp["router"], h)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(chosen[t], weights[t]):
            out[t] += g * clamped_gated(w, f"{p}e{e}.", h[t : t + 1], mlp["expert"].get("limit", np.inf))[0]
    return out


# ---- the model ----------------------------------------------------------------------------------------------------
def forward(w, cfg, tokens, streams=False, margins=False):
    """Logits [T, vocab] of one whole sequence; with ``streams`` also the residual stream after every layer, with
    ``margins`` also the smallest router margin at every position over all routed layers (inf without one)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    after, worst = [], np.full(len(tokens), np.inf)
    v_first = None
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        if spec["type"] == "delta":
            x = x + delta(w, p + "mix.", m, h, eps)
        elif spec["type"] == "attention":
            y, own = attention(w, p + "mix.", m, h, eps, v_first if m.get("v_mix") else None)
            if m.get("v_mix") and v_first is None:
                v_first = own
            x = x + y
        else:
            raise ValueError(spec["type"])
        mlp = spec.get("mlp")
        if mlp:
            h = layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps)
            if mlp["kind"] == "dense":
                x = x + clamped_gated(w, p + "mlp.", h, mlp.get("limit", np.inf))
            else:
                worst = np.minimum(worst, route(w, p + "mlp.", mlp["router"], h)[2])
                x = x + routed(w, p + "mlp.", mlp, h)
        after.append(x.copy())
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
    out = (logits,) + ((np.stack(after),) if streams else ()) + ((worst,) if margins else ())
    return out if len(out) > 1 else logits


def sure_prefix(margins, least=0.02):
    """How many leading positions come before the first close call of any router (a margin below ``least``)."""
    close = np.asarray(margins) < least
    return int(np.argmax(close)) if close.any() else len(close)


def greedy(w, cfg, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(np.argmax(forward(w, cfg, seq)[-1])))
    return seq[len(prompt):]
