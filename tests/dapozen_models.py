"""Small Dapozen configurations of the tests' own and weights drawn so that faults show.

N(0, 0.02) everywhere would hide faults: a flat softmax does not care which keys it sees, a convolution whose taps vanish loses
no history, a state that forgets at once cannot be lost.  So: scores of unit heads are a few units, the taps of a convolution are
of one size, some heads forget within a few tokens and some remember for hundreds, the clipped units' inputs reach their limits, and
the logits come near their cap.

`standout` rewrites a folder's tensors so that one token's key outweighs every other in every head of the first layer: whether
that token is seen decides the result, so a key just inside or just outside a run of positions changes the logits by as much as they
vary at all.
"""
import json
import os

import numpy as np

import harness


def attention(heads, kv, dim, vdim, dims, size, conv=4, base=10000.0, amount=3.0):
    """`amount`: how large a score of two random unit heads is."""
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "scale": amount / dim ** 0.5,
                                           "rot": {"base": base, "dims": dims}, "mask": {"size": size}}}


def mamba2(heads, vdim, state, groups=1, norm_groups=1, conv=4):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def config(width, vocab, layers, mlps, loop=None, scale=1.0, eps=1e-5, cap=12.0):
    c = {"architecture": "Dapozen", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
         "layers": [dict(L, mlp=f) for L, f in zip(layers, mlps)]}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    if cap:
        c["logit_softcap"] = cap
    return c


CONFIGS = {
    # every kind of layer, values of another size than the keys, a layer without feed-forward, part of a head rotated, a loop in the
    # middle, convolutions of two, three and four taps, runs of positions that are no pages
    "P": config(96, 300, [attention(4, 2, 16, 24, 8, 10), mamba2(6, 8, 16, 2, 3, 3), attention(6, 3, 20, 12, 20, 37, 2, 500.0, 2.0), mamba2(4, 24, 12, 4, 2)],
                [dense(40), moe(6, 3, 24, 0.8, (40, 1.3)), None, moe(5, 2, 16, 1.5)], (1, 3, 2), scale=2.5, eps=3e-6),
    # one of everything: one head, one group, one expert, one tap, a run of one position; no loop, no cap
    "Q": config(64, 200, [mamba2(1, 32, 8, conv=1), attention(1, 1, 16, 16, 2, 1, 1, 30.0), attention(1, 1, 16, 16, 16, 64, 2)],
                [moe(1, 1, 16, 1.0), None, moe(2, 1, 8, 2.0, (8, 0.5))], cap=None),
    # sizes that the tensor-core kernels like; many experts; a value size that is not the keys' and is no power of two; the first
    # layers three times
    "R": config(128, 512, [attention(8, 2, 32, 32, 16, 64, base=20000.0), mamba2(4, 32, 64, 2, 2), attention(4, 4, 48, 80, 48, 100, base=1000.0), mamba2(8, 64, 32, 1, 4)],
                [dense(128), moe(16, 4, 64, 1.0, (96, 1.5)), moe(8, 3, 32, 0.7), dense(64)], (0, 2, 3), scale=1.5),
    # sizes that fit no tile: a width that is no multiple of 8, odd head counts, five and six taps, every expert for every token
    "S": config(100, 333, [attention(5, 5, 10, 14, 6, 33, 5, 77.0), mamba2(5, 10, 12, 5, 2, 6), attention(6, 2, 24, 40, 2, 129, 4, 777.0)],
                [moe(5, 5, 22, 0.9, (30, 1.1)), dense(50), moe(9, 3, 10, 1.4)], scale=0.7, eps=1e-6, cap=8.0),
    "T": config(52, 97, [mamba2(3, 7, 5, 1, 7, 2), attention(3, 1, 7, 9, 6, 5, 3, 200.0), attention(10, 5, 6, 11, 4, 70, 4, 900.0), mamba2(2, 9, 7, 2, 1, 5)],
                [dense(22), None, moe(4, 4, 6, 1.0, (14, 2.0)), None], (1, 4, 2), scale=3.0),
    # heads as large as real models have them
    "U": config(256, 200, [attention(4, 2, 128, 128, 64, 96), mamba2(8, 64, 128, 2, 2), attention(4, 1, 64, 64, 64, 150, 4)],
                [moe(4, 2, 64, 1.0, (64, 1.0)), dense(128), None]),
    # heads larger than the tensor-core kernels take, a value size beyond their tile, a state of more rows than they hold
    "V": config(72, 120, [mamba2(2, 160, 24), attention(2, 1, 144, 136, 100, 70, 4, 5000.0), mamba2(2, 24, 200, 1, 2), attention(3, 1, 24, 200, 24, 45, 3)],
                [None, dense(24), None, None], scale=2.0),
    # single mechanisms
    "attention_only": config(64, 100, [attention(4, 2, 16, 24, 8, 23)], [None]),
    "mamba2_only": config(64, 100, [mamba2(6, 16, 24, 2, 3)], [None]),
    "dense_only": config(64, 100, [mamba2(1, 8, 8)], [dense(48)], scale=1.7),
    "experts_only": config(64, 100, [mamba2(1, 8, 8)], [moe(8, 3, 16, 0.9, (24, 1.2))]),
    "loop_only": config(64, 100, [mamba2(2, 16, 8), attention(2, 2, 16, 16, 8, 19)], [None, None], (0, 2, 4)),
    # scores that let one key stand out; runs of 50 positions begin and end in the middle of a page, runs of 128 at a page's
    "far": config(64, 30, [attention(4, 2, 16, 16, 8, 50), attention(4, 2, 16, 16, 8, 50)], [None, dense(32)], cap=30.0),
    "far_pages": config(64, 30, [attention(4, 2, 32, 32, 8, 128), attention(4, 2, 32, 32, 8, 128)], [None, dense(32)], cap=30.0),
    # states and runs that reach back over hundreds of tokens
    "long": config(64, 120, [mamba2(4, 16, 16, 1, 2), attention(4, 2, 32, 32, 16, 192)], [dense(48), None], (0, 2, 2)),
}
SEEDS = {name: 310 + i for i, name in enumerate(CONFIGS)}


def tensors_of(cfg, rng):
    """Every tensor of the design by name: float32, or int32 for tables."""
    w = cfg["width"]
    out = {}

    def normal(shape, std=0.02, mean=0.0):
        return (rng.standard_normal(shape) * std + mean).astype(np.float32)

    def taps(channels, n):
        return normal((channels, n), 0.6 / np.sqrt(n), 0.3 / np.sqrt(n))

    unit = 1.0 / np.sqrt(w)                       # sublayers read normed rows: products of entries of about 1
    out["embed"] = normal((cfg["vocab"], w), 1.2 / cfg["embedding"]["scale"])
    out["head"] = normal((cfg["vocab"], w), 5.0 * unit)
    out["final.norm"] = normal((w,), 0.1, 1.0)
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        H, dv = m["heads"], m["vdim"]
        out[p + "norm1"], out[p + "norm1b"] = normal((w,), 0.1, 1.0), normal((w,), 0.2, 0.8)
        out[p + "mix.o"] = normal((w, H * dv), 1.0 / np.sqrt(H * dv))
        if L["type"] == "attention":
            G, d, n = m["kv_heads"], m["dim"], m["conv"]
            for name, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                out[p + "mix." + name], out[p + "mix.%s.b" % name] = normal((rows, w), unit), normal((rows,), 0.3)
                out[p + "mix.%s.conv" % name] = taps(rows, n)
            out[p + "mix.g"] = normal((H * dv, w), 1.5 * unit)
        else:
            inner, gn = H * dv, m["groups"] * m["state"]
            out[p + "mix.in"] = normal((2 * inner + 2 * gn + H, w), unit)
            out[p + "mix.conv"], out[p + "mix.conv.b"] = taps(inner + 2 * gn, m["conv"]), normal((inner + 2 * gn,), 0.2)
            out[p + "mix.dt_bias"] = normal((H,), 0.5, -0.5)
            out[p + "mix.A_log"] = np.linspace(np.log(2.0), np.log(0.004), H).astype(np.float32) if H > 1 else np.array([-3.0], dtype=np.float32)
            out[p + "mix.D"] = normal((H,), 0.5, 1.0)
            out[p + "mix.norm"] = normal((inner,), 0.2, 1.0)
        mlp = L.get("mlp")
        if not mlp:
            continue
        out[p + "norm2"], out[p + "norm2b"] = normal((w,), 0.1, 1.0), normal((w,), 0.2, 0.8)
        if mlp["kind"] == "dense":
            units = [("", mlp["ff"])]
        else:
            r = mlp["router"]
            out[p + "mlp.table"] = np.stack([rng.permutation(r["experts"])[:r["top"]] for _ in range(cfg["vocab"])]).astype(np.int32)
            units = [("e%d." % e, mlp["expert"]["ff"]) for e in range(r["experts"])]
            if mlp.get("shared"):
                units.append(("shared.", mlp["shared"]["ff"]))
        for n, f in units:
            out[p + "mlp." + n + "gate"], out[p + "mlp." + n + "up"] = normal((f, w), 1.2 * unit), normal((f, w), 1.2 * unit)
            out[p + "mlp." + n + "down"] = normal((w, f), 1.0 / np.sqrt(f))
    return out


def standout(cfg, t, token, gain=40.0):
    """Changes the first layer (attention) of the tensors `t` in place: the last channel of every key head, which no rotation
    reaches and whose convolution passes the present token only, is large for `token` and nothing for every other one, and every query
    has a large fixed part there, so that the score against that token's key stands out; its value is large too, and stays where it
    is."""
    m = cfg["layers"][0]["mixer"]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    assert m["rot"]["dims"] < d
    assert cfg["vocab"] <= cfg["width"]
    x = t["embed"].astype(np.float64) * cfg["embedding"]["scale"]
    rows = x / np.sqrt(np.mean(x * x, axis=1, keepdims=True) + cfg["norm"]["eps"]) * t["l0.norm1"]      # what the layer reads for each id
    only = np.linalg.pinv(rows)[:, token]          # one for `token`, zero for every other id
    rng = np.random.default_rng(5)
    now = np.zeros(m["conv"], dtype=np.float32)
    now[-1] = 1.0
    for g in range(G):
        t["l0.mix.k"][g * d + d - 1] = gain * only
        t["l0.mix.k.b"][g * d + d - 1] = 0.0
        t["l0.mix.k.conv"][g * d + d - 1] = now
    t["l0.mix.q.b"][d - 1::d] = 10.0
    t["l0.mix.q.conv"][d - 1::d] = now
    t["l0.mix.v.conv"][:] = now
    t["l0.mix.v"] += (8.0 * np.outer(rng.standard_normal(G * dv), only)).astype(np.float32)
    return t


def write_folder(path, cfg, tensors):
    from friday_inference_engine_b200.weights import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)

    def stored(n, x):
        if x.dtype == np.int32:
            return (n, "I32", list(x.shape), x.astype("<i4").tobytes())
        return (n, "BF16", list(x.shape), harness.f32_to_bf16_bytes(x))
    write_safetensors(os.path.join(path, "model.safetensors"), [stored(n, x) for n, x in tensors.items()])
    return path
