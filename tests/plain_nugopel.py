"""Nugopel, plain and slow: NumPy float64, one whole sequence at a time, no
cache (every attention position looks at its whole prefix), one function per
mechanism.  It shares nothing with the package: it reads config.json as a dict
and model.safetensors with its own few lines."""
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
        if m["dtype"] != "BF16":
            raise ValueError(m["dtype"])
        w[name] = (np.frombuffer(data[lo:hi], dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64).reshape(m["shape"])
    return w, cfg


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, dtype=np.float64)))


def rms_norm(x, weight, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * weight


def offset_norm(x, stored, eps):
    """The stored numbers lie around zero: the norm's weight is one more."""
    return rms_norm(x, 1.0 + stored, eps)


# ---- positions ---------------------------------------------------------------------------------------------------
def frequencies(rot):
    """Turns per token (times 2 pi) of the pairs of a head.  With scaling, by the wavelength: short ones stay, long ones are
    stretched by the factor, and those between are a mixture of the two."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return np.array(out)


def rotate(x, rot):
    """x [T, heads, d]: the first ``dims`` numbers of every head, number i with number i + dims / 2."""
    half = rot["dims"] // 2
    a = np.arange(x.shape[0])[:, None, None] * frequencies(rot)
    u, v = x[:, :, :half], x[:, :, half : 2 * half]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[:, :, 2 * half :]], axis=-1)


# ---- attention over a window, with one added to the softmax's denominator ------------------------------------------
def causal_mask(T, window=None):
    """[i, j]: position i sees j."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = j <= i
    return seen if window is None else seen & (i - j < window)


def softmax(scores, mask, one_more=False):
    """Rows of weights over the keys; ``one_more``: a term of score 0 that has no value stands in the denominator too."""
    s = np.where(mask, scores, -np.inf)
    m = s.max(axis=-1, keepdims=True)
    if one_more:
        m = np.maximum(m, 0.0)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + (np.exp(-m) if one_more else 0.0))


def attend(q, k, v, scale, mask, one_more):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[-1]))
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax((q[:, h] @ k[:, g].T) * scale, mask, one_more) @ v[:, g]
    return out


def attention(w, p, m, h, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, H, d), m["rot"])
    k = rotate(rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, G, d), m["rot"])
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    mask = causal_mask(T, m["mask"]["size"] if m.get("mask") else None)
    return attend(q, k, v, m["scale"], mask, True).reshape(T, H * dv) @ w[p + "o"].T


# ---- latent attention ----------------------------------------------------------------------------------------------
def latent(w, p, h, eps):
    return rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)


def latent_attention(w, p, m, h, c):
    """``c`` [T, kv_rank]: this layer's latent or another layer's."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, d)
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    o = attend(q, k, v, m["scale"], causal_mask(T), False).reshape(T, H * dv)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward --------------------------------------------------------------------------------------------------
def expert(w, p, h):
    return np.maximum(h @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def route(w, p, r, h):
    """(chosen experts [T, top], their weights [T, top], margin [T]): ``margin`` is by how much the last chosen logit leads
    the first one left out, so that tests know a close call."""
    z = h @ w[p + "router"].T
    chosen = np.argsort(-z, axis=-1, kind="stable")[:, : r["top"]]
    picked = np.take_along_axis(z, chosen, axis=-1)
    e = np.exp(picked - picked.max(axis=-1, keepdims=True))
    margin = np.full(len(z), np.inf)
    if r["top"] < r["experts"]:
        ranked = -np.sort(-z, axis=-1)
        margin = ranked[:, r["top"] - 1] - ranked[:, r["top"]]
    return chosen, e / e.sum(axis=-1, keepdims=True), margin


def routed(w, p, mlp, h):
    chosen, weights, _ = route(w, p, mlp["router"], h)
    out = expert(w, p + "shared.", h) if mlp.get("shared") else np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(chosen[t], weights[t]):
            out[t] += g * expert(w, f"{p}e{e}.", h[t : t + 1])[0]
    return out


# ---- the model -----------------------------------------------------------------------------------------------------
def forward(w, cfg, tokens, streams=False, margins=False):
    """Logits [T, vocab] of one whole sequence; with ``streams`` also the residual stream after every layer, with
    ``margins`` also the smallest router margin at every position over all layers (inf without a router)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    after, worst, latents = [], np.full(len(tokens), np.inf), {}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        h = offset_norm(x, w[p + "norm1"], eps)
        if spec["type"] == "latent_attention":
            if m.get("kv_from") is None:
                latents[i] = latent(w, p + "mix.", h, eps)
            y = latent_attention(w, p + "mix.", m, h, latents[i if m.get("kv_from") is None else m["kv_from"]])
        elif spec["type"] == "attention":
            y = attention(w, p + "mix.", m, h, eps)
        else:
            raise ValueError(spec["type"])
        x = x + offset_norm(y, w[p + "norm1b"], eps)
        mlp = spec.get("mlp")
        if mlp:
            h = offset_norm(x, w[p + "norm2"], eps)
            worst = np.minimum(worst, route(w, p + "mlp.", mlp["router"], h)[2])
            x = x + offset_norm(routed(w, p + "mlp.", mlp, h), w[p + "norm2b"], eps)
        after.append(x.copy())
    logits = offset_norm(x, w["final.norm"], eps) @ w["head"].T
    out = (logits,) + ((np.stack(after),) if streams else ()) + ((worst,) if margins else ())
    return out if len(out) > 1 else logits


def sure_prefix(margins, least=0.05):
    """How many leading positions come before the first close call of any router (a margin below ``least``)."""
    close = np.asarray(margins) < least
    return int(np.argmax(close)) if close.any() else len(close)


def greedy(w, cfg, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(np.argmax(forward(w, cfg, seq)[-1])))
    return seq[len(prompt):]
