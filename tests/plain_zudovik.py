"""Zudovik, written plainly from its equations: float64 numpy, one function per mechanism, token by token where the design
is a recurrence.  It shares no code with the library; the tests compare the library with it.

A model is a config (a dict as config.json holds it) and a dict name -> numpy array of weights.  `forward` runs a whole
sequence and returns the logits at every position and, if asked, the residual stream after every layer.
"""
import json
import math
import os
import struct

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def rms(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def embed(tokens, table, scale):
    return table[np.asarray(tokens)] * scale


# ---- linear attention with a constant decay per head
def decayed_states(k, v, decay):
    """States after every token: S_t = decay S_(t-1) + k_t v_t^T, S before the first token zero.  k [T, d], v [T, dv]."""
    S = np.zeros((k.shape[1], v.shape[1]))
    out = []
    for t in range(k.shape[0]):
        S = decay * S + np.outer(k[t], v[t])
        out.append(S.copy())
    return out


def lightning(h, W, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W["q"].T).reshape(T, H, d)
    k = silu(h @ W["k"].T).reshape(T, H, d)
    v = silu(h @ W["v"].T).reshape(T, H, dv)
    o = np.zeros((T, H, dv))
    for a in range(H):
        for t, S in enumerate(decayed_states(k[:, a], v[:, a], m["decay"][a])):
            o[t, a] = q[t, a] @ S
    y = rms(o.reshape(T, H * dv), W["norm"], eps)          # one norm over all heads' results
    return (y * sigmoid(h @ W["g"].T)) @ W["o"].T


# ---- attention
def rotate_neighbours(x, rot):
    """x [T, heads, d]: dimensions 2i and 2i + 1 among the first `dims` turn by position * base^(-2i / dims)."""
    dims, base = rot["dims"], rot["base"]
    out = x.copy()
    for p in range(x.shape[0]):
        for i in range(dims // 2):
            a = p * base ** (-2.0 * i / dims)
            u, v = x[p, :, 2 * i], x[p, :, 2 * i + 1]
            out[p, :, 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[p, :, 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def cap(s, limit):
    return limit * np.tanh(s / limit)


def softmax_with_sink(scores, sink):
    """Causal softmax of scores [T, T] whose denominator also holds exp(sink)."""
    out = np.zeros_like(scores)
    for i in range(scores.shape[0]):
        s = scores[i, :i + 1]
        top = max(s.max(), sink)
        e = np.exp(s - top)
        out[i, :i + 1] = e / (e.sum() + math.exp(sink - top))
    return out


def keys_and_values(h, W, m, eps):
    T = h.shape[0]
    G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
    k = rms(h @ W["k"].T + W["k.b"], W["k.norm"], eps).reshape(T, G, d)
    v = (h @ W["v"].T + W["v.b"]).reshape(T, G, dv)
    return rotate_neighbours(k, m["rot"]), v


def attention(h, W, m, eps, shared):
    """`shared`: the keys and values of another layer, or None; returns the result and the keys and values it used."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ W["q"].T + W["q.b"], W["q.norm"], eps).reshape(T, H, d)
    q = rotate_neighbours(q, m["rot"])
    k, v = shared if shared is not None else keys_and_values(h, W, m, eps)
    out = np.zeros((T, H, dv))
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * m["scale"]
        out[:, a] = softmax_with_sink(cap(s, m["softcap"]), float(W["sink"][a])) @ v[:, g]
    out = out * sigmoid(h @ W["g"].T)[:, :, None]          # one number per head
    return out.reshape(T, H * dv) @ W["o"].T, (k, v)


# ---- feed-forwards
def dense(h, W):
    return np.maximum(h @ W["up"].T, 0.0) ** 2 @ W["down"].T


def clipped_glu(h, W, limit):
    g = np.minimum(h @ W["gate"].T, limit)
    u = np.clip(h @ W["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W["down"].T


def choose(z, correction, top):
    """Ids and weights of one token's experts: softmax scores over everything the router knows, chosen by score plus
    correction, weighted by the scores alone."""
    e = np.exp(z - z.max())
    s = e / e.sum()
    ids = np.argsort(-(s + correction), kind="stable")[:top]
    return ids, s[ids] / (s[ids].sum() + 1e-20)


def experts(h, W, mlp):
    r = mlp["router"]
    n, top = r["experts"], r["top"]
    z = h @ W["router"].T
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        ids, weights = choose(z[t], W["correction"], top)
        for e, w in zip(ids, weights):
            if e >= n:
                out[t] += w * h[t]                         # an identity expert
            else:
                out[t] += w * clipped_glu(h[t], sub(W, "e%d." % e), mlp["expert"]["limit"])
    if mlp.get("shared"):
        out += sigmoid(h @ W["shared.sg"].T) * clipped_glu(h, sub(W, "shared."), mlp["shared"]["limit"])
    return out


def sub(weights, prefix):
    return {n[len(prefix):]: x for n, x in weights.items() if n.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out (a list) receives the stream after every layer."""
    W = {n: np.asarray(x, dtype=np.float64) for n, x in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, W["embed"], cfg["embedding"]["scale"])
    held = {}
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % i
        m, mix = L["mixer"], sub(W, p + "mix.")
        if L["type"] == "lightning":
            y = lightning(x, mix, m, eps)
        elif L["type"] == "attention":
            j = m.get("kv_from")
            y, held[i] = attention(x, mix, m, eps, None if j is None else held[j])
        else:
            raise ValueError("no mixer of type %r" % L["type"])
        x = x + rms(y, W[p + "norm1"], eps)
        mlp = L.get("mlp")
        if mlp:
            ff = sub(W, p + "mlp.")
            x = x + rms(dense(x, ff) if mlp["kind"] == "dense" else experts(x, ff, mlp), W[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms(x, W["final.norm"], eps) @ W["head"].T


def load(model_dir):
    """config.json and every tensor of model.safetensors (BF16, F32 or I32) as float64 / int arrays."""
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(model_dir, "model.safetensors"), "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        meta = json.loads(f.read(n))
        blob = f.read()
    out = {}
    for name, m in meta.items():
        if name == "__metadata__":
            continue
        a, b = m["data_offsets"]
        raw = np.frombuffer(blob[a:b], dtype=np.uint8)
        if m["dtype"] == "BF16":
            x = (raw.view("<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif m["dtype"] == "F32":
            x = raw.view("<f4").astype(np.float64)
        elif m["dtype"] == "I32":
            x = raw.view("<i4")
        else:
            raise ValueError("tensor %s: dtype %s" % (name, m["dtype"]))
        out[name] = x.reshape(m["shape"])
    return cfg, out


def greedy(cfg, weights, prompt, n):
    """The n tokens that follow `prompt` when the largest logit is taken every time (the first of equal ones)."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, weights, toks)[-1])))
    return toks[len(prompt):]
