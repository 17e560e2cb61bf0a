"""Dapozen, written plainly from its equations: float64 numpy, one function per mechanism, token by token where the design
is a recurrence.  It shares no code with the library; the tests compare the library with it.

A model is a config (a dict as config.json holds it) and a dict name -> numpy array of weights.  `forward` runs a whole
sequence and returns the logits at every position and, if asked, the residual stream after every layer run.
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


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(x, eps):
    """x divided by its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms(x, w, eps):
    return unit_rms(x, eps) * w


def embed(tokens, table, scale):
    return table[np.asarray(tokens)] * scale


def causal_conv(u, taps):
    """y_t = sum_j taps[:, j] u_(t - n + 1 + j) for u [T, channels] and taps [channels, n]; zeros before the start."""
    n = taps.shape[1]
    y = np.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(n):
            s = t - n + 1 + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


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


def chunk_softmax(scores, size):
    """Row i of scores [T, T] over the columns j <= i of the same chunk of `size` positions; zero elsewhere."""
    out = np.zeros_like(scores)
    for i in range(scores.shape[0]):
        first = i // size * size
        e = np.exp(scores[i, first:i + 1] - scores[i, first:i + 1].max())
        out[i, first:i + 1] = e / e.sum()
    return out


def projected(h, W, name):
    return causal_conv(h @ W[name].T + W[name + ".b"], W[name + ".conv"])


def attention(h, W, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms(rotate_neighbours(projected(h, W, "q").reshape(T, H, d), m["rot"]), eps)
    k = unit_rms(rotate_neighbours(projected(h, W, "k").reshape(T, G, d), m["rot"]), eps)
    v = projected(h, W, "v").reshape(T, G, dv)
    out = np.zeros((T, H, dv))
    for a in range(H):
        g = a // (H // G)
        out[:, a] = chunk_softmax((q[:, a] @ k[:, g].T) * m["scale"], m["mask"]["size"]) @ v[:, g]
    return (out.reshape(T, H * dv) * sigmoid(h @ W["g"].T)) @ W["o"].T


# ---- state space duality
def ssd_states(x, B, dt, a_log):
    """States after every token of one head: S_t = exp(-exp(a_log) dt_t) S_(t-1) + dt_t B_t x_t^T, zero before the first.
    x [T, dv], B [T, N], dt [T]."""
    S = np.zeros((B.shape[1], x.shape[1]))
    out = []
    for t in range(x.shape[0]):
        S = math.exp(-math.exp(a_log) * dt[t]) * S + dt[t] * np.outer(B[t], x[t])
        out.append(S.copy())
    return out


def group_norm(y, parts, w, eps):
    """Each of `parts` equal runs of a row divided by its own root mean square, then times w [row]."""
    T, n = y.shape
    return unit_rms(y.reshape(T, parts, n // parts), eps).reshape(T, n) * w


def mamba2(h, W, m, eps):
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, gn = H * dv, G * N
    p = h @ W["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * gn], p[:, 2 * inner + 2 * gn:]
    xbc = silu(causal_conv(xbc, W["conv"]) + W["conv.b"])
    x = xbc[:, :inner].reshape(T, H, dv)
    B = xbc[:, inner:inner + gn].reshape(T, G, N)
    C = xbc[:, inner + gn:].reshape(T, G, N)
    dt = softplus(dt + W["dt_bias"])
    y = np.zeros((T, H, dv))
    for a in range(H):
        g = a // (H // G)
        for t, S in enumerate(ssd_states(x[:, a], B[:, g], dt[:, a], float(W["A_log"][a]))):
            y[t, a] = S.T @ C[t, g] + W["D"][a] * x[t, a]
    return group_norm(y.reshape(T, inner) * silu(z), m["norm_groups"], W["norm"], eps) @ W["o"].T


# ---- feed-forwards
def dense(h, W):
    return (silu(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def clipped_glu(h, W, limit):
    g = np.minimum(h @ W["gate"].T, limit)
    u = np.clip(h @ W["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W["down"].T


def experts(h, tokens, W, mlp):
    """The experts that the table gives each token's id, all with the weight 1 / top, and the shared one for every token."""
    top = mlp["router"]["top"]
    out = np.zeros_like(h)
    for t, token in enumerate(tokens):
        for e in W["table"][token]:
            out[t] += clipped_glu(h[t], sub(W, "e%d." % int(e)), mlp["expert"]["limit"]) / top
    if mlp.get("shared"):
        out += clipped_glu(h, sub(W, "shared."), mlp["shared"]["limit"])
    return out


def sub(weights, prefix):
    return {n[len(prefix):]: x for n, x in weights.items() if n.startswith(prefix)}


def run_order(cfg):
    """Layer numbers in the order in which they run: the loop's span `times` times in a row."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out (a list) receives the stream after every layer run."""
    W = {n: np.asarray(x, dtype=np.float64) for n, x in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, W["embed"], cfg["embedding"]["scale"])
    for i in run_order(cfg):
        L, p = cfg["layers"][i], "l%d." % i
        mixers = {"attention": attention, "mamba2": mamba2}
        y = mixers[L["type"]](rms(x, W[p + "norm1"], eps), sub(W, p + "mix."), L["mixer"], eps)
        x = x + rms(y, W[p + "norm1b"], eps)
        mlp = L.get("mlp")
        if mlp:
            ff, h = sub(W, p + "mlp."), rms(x, W[p + "norm2"], eps)
            y = dense(h, ff) if mlp["kind"] == "dense" else experts(h, tokens, ff, mlp)
            x = x + rms(y, W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    logits = rms(x, W["final.norm"], eps) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(logits / cap) if cap else logits


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
