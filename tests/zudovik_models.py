"""Small Zudovik configurations of the tests' own and weights drawn so that faults show.

N(0, 0.02) everywhere would hide faults: a flat softmax does not care which keys it sees, a cap far above the scores caps
nothing, a state that forgets at once cannot be lost.  So: normed queries and keys give scores of a few units, of the size of
the caps and the sinks; decays lie between one half and one (one included); the clipped units' inputs reach their limits; the
routers' scores and the corrections are of the size of the scores' differences.

`standout` rewrites a folder's tensors so that one token's key outweighs every other in every head of the first layer:
whether that token is seen decides the result, so a far key that is lost changes the logits by as much as they vary at all.
"""
import json
import os

import numpy as np

import harness


def lightning(heads, dim, vdim, decay):
    assert len(decay) == heads
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def attention(heads, kv, dim, vdim, dims, base=10000.0, scale=None, softcap=6.0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "softcap": softcap,
         "rot": {"base": base, "dims": dims}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, limit, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def config(width, vocab, layers, mlps, scale=1.0, eps=1e-5):
    return {"architecture": "Zudovik", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": [dict(L, mlp=f) for L, f in zip(layers, mlps)]}


CONFIGS = {
    # every kind of layer, values of another size than the keys, keys and values read by a later layer and by one after it, a
    # layer without feed-forward, part of a head rotated
    "P": config(96, 300, [attention(4, 2, 16, 24, 8), lightning(3, 16, 24, [0.55, 0.9, 0.997]), attention(6, 3, 20, 12, 20, 500.0, 0.3, 4.0),
                          attention(6, 3, 20, 12, 20, 500.0, 0.25, 9.0, 2), attention(4, 2, 16, 24, 8, kv_from=0)],
                [dense(40), moe(6, 2, 3, 24, 0.8, (40, 1.3)), None, moe(5, 1, 2, 16, 1.5), dense(56)], scale=2.5, eps=3e-6),
    # one of everything: one head, one expert chosen, no identity experts, no expert for everybody, a decay of one
    "Q": config(64, 200, [lightning(1, 8, 32, [1.0]), attention(1, 1, 16, 16, 2, 30.0, 0.5, 2.0), attention(1, 1, 16, 16, 2, 30.0, 0.5, 3.0, 1)],
                [moe(2, 0, 1, 16, 1.0), None, moe(1, 1, 1, 8, 2.0, (8, 0.5))]),
    # sizes that the tensor-core kernels like; many experts; a value size that is not the keys' and is no power of two
    "R": config(128, 512, [lightning(4, 32, 64, [0.5, 0.8, 0.98, 0.9995]), attention(8, 2, 32, 32, 16, 20000.0, 0.2, 5.0),
                           lightning(2, 64, 32, [0.95, 0.999]), attention(4, 4, 48, 80, 48, 1000.0, 0.15, 8.0), attention(8, 2, 32, 32, 16, 20000.0, 0.2, 7.0, 1)],
                [dense(128), moe(16, 2, 4, 64, 1.0, (96, 1.5)), moe(8, 4, 3, 32, 0.7), dense(64), moe(4, 1, 2, 40, 1.2, (64, 0.9))], scale=1.5),
    # sizes that fit no tile: a width that is no multiple of 8, odd head counts and sizes, every expert chosen
    "S": config(100, 333, [attention(5, 5, 10, 14, 6, 77.0, 0.4, 3.0), lightning(5, 12, 10, [0.6, 0.7, 0.9, 0.97, 0.999]), attention(6, 2, 24, 40, 2, 777.0, 0.2, 7.0)],
                [moe(5, 2, 7, 22, 0.9, (30, 1.1)), dense(50), moe(9, 3, 3, 10, 1.4)], scale=0.7, eps=1e-6),
    "T": config(52, 97, [lightning(3, 7, 5, [0.75, 0.99, 0.0]), attention(3, 1, 7, 9, 6, 200.0, 0.5, 4.0), attention(10, 5, 6, 11, 4, 900.0, 0.4, 5.0),
                         attention(10, 5, 6, 11, 4, 900.0, 0.45, 5.0, 2)],
                [dense(22), None, moe(4, 4, 5, 6, 1.0, (14, 2.0)), None], scale=3.0),
    # heads as large as real models have them
    "U": config(256, 200, [attention(4, 2, 128, 128, 64, 10000.0, 0.09, 10.0), lightning(2, 128, 128, [0.9, 0.998]), attention(4, 2, 128, 128, 64, 10000.0, 0.09, 8.0, 0)],
                [moe(4, 1, 2, 64, 1.0, (64, 1.0)), dense(128), None]),
    # heads larger than the tensor-core kernels take, a value size beyond their tile
    "V": config(72, 120, [lightning(2, 160, 24, [0.8, 0.99]), attention(2, 1, 144, 136, 100, 5000.0, 0.08, 6.0), lightning(2, 24, 200, [0.97, 0.6]), attention(3, 1, 24, 200, 24)],
                [None, dense(24), None, None], scale=2.0),
    # single mechanisms
    "attention_only": config(64, 100, [attention(4, 2, 16, 24, 8, softcap=3.0)], [None]),
    "shared_keys_only": config(64, 100, [attention(4, 2, 16, 12, 16, 300.0), attention(4, 2, 16, 12, 16, 300.0, 0.4, 2.5, 0)], [None, None]),
    "lightning_only": config(64, 100, [lightning(3, 16, 24, [0.7, 0.95, 0.9995])], [None]),
    "dense_only": config(64, 100, [lightning(1, 8, 8, [0.5])], [dense(48)], scale=1.7),
    "experts_only": config(64, 100, [lightning(1, 8, 8, [0.5])], [moe(8, 3, 4, 16, 0.9, (24, 1.2))]),
    # a cap that lets one score stand out among hundreds; the second layer reads the same keys
    "far": config(64, 120, [attention(4, 2, 16, 16, 8, scale=0.4, softcap=25.0), attention(4, 2, 16, 16, 8, scale=0.4, softcap=20.0, kv_from=0)], [None, dense(32)]),
}
SEEDS = {name: 170 + i for i, name in enumerate(CONFIGS)}


def tensors_of(cfg, rng, clear_routing=False):
    """Every tensor of the design by name, float32.  clear_routing: the corrections are far apart, so that rounding cannot
    change a choice (what a comparison in bfloat16 needs)."""
    w = cfg["width"]
    out = {}

    def normal(shape, std=0.02, mean=0.0):
        return (rng.standard_normal(shape) * std + mean).astype(np.float32)

    size = 1.2                       # entries of the stream at the layer's input: every sublayer adds entries of about 1
    out["embed"] = normal((cfg["vocab"], w), size / cfg["embedding"]["scale"])
    out["head"] = normal((cfg["vocab"], w), 1.0 / np.sqrt(w))
    out["final.norm"] = normal((w,), 0.1, 1.0)
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        unit = 1.0 / (np.sqrt(w) * size)          # rows of this size make products of entries of about 1
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        out[p + "norm1"] = normal((w,), 0.1, 1.0)
        out[p + "mix.o"] = normal((w, H * dv), 1.0 / np.sqrt(H * dv))
        if L["type"] == "lightning":
            for n, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                out[p + "mix." + n] = normal((rows, w), unit)
            out[p + "mix.norm"] = normal((H * dv,), 0.2, 1.0)
        else:
            G = m["kv_heads"]
            # normed entries have a root mean square of one: scores of about 3 before the cap
            amount = (3.0 / (np.sqrt(d) * m["scale"])) ** 0.5
            out[p + "mix.q"], out[p + "mix.q.b"] = normal((H * d, w), unit), normal((H * d,), 0.3)
            out[p + "mix.q.norm"] = normal((H * d,), 0.3 * amount, amount)
            if m.get("kv_from") is None:
                out[p + "mix.k"], out[p + "mix.k.b"] = normal((G * d, w), unit), normal((G * d,), 0.3)
                out[p + "mix.k.norm"] = normal((G * d,), 0.3 * amount, amount)
                out[p + "mix.v"], out[p + "mix.v.b"] = normal((G * dv, w), unit), normal((G * dv,), 0.3)
            out[p + "mix.sink"] = normal((H,), 1.5, 1.0)
            out[p + "mix.g"] = normal((H, w), 1.5 * unit)
        size = np.sqrt(size * size + 1.0)
        mlp = L.get("mlp")
        if not mlp:
            continue
        unit = 1.0 / (np.sqrt(w) * size)
        out[p + "norm2"] = normal((w,), 0.1, 1.0)
        if mlp["kind"] == "dense":
            out[p + "mlp.up"] = normal((mlp["ff"], w), unit)
            out[p + "mlp.down"] = normal((w, mlp["ff"]), 1.0 / np.sqrt(mlp["ff"]))
        else:
            r = mlp["router"]
            E = r["experts"] + r["identity"]
            units = [("e%d." % e, mlp["expert"]["ff"]) for e in range(r["experts"])]
            if mlp.get("shared"):
                units.append(("shared.", mlp["shared"]["ff"]))
                out[p + "mlp.shared.sg"] = normal((1, w), 1.5 * unit)
            for n, f in units:
                out[p + "mlp." + n + "gate"], out[p + "mlp." + n + "up"] = normal((f, w), 1.2 * unit), normal((f, w), 1.2 * unit)
                out[p + "mlp." + n + "down"] = normal((w, f), 1.0 / np.sqrt(f))
            out[p + "mlp.router"] = normal((E, w), 1.2 * unit)
            if clear_routing:                     # further apart than any two scores
                out[p + "mlp.correction"] = (rng.permutation(E) * 1.2 - 0.6 * E).astype(np.float32)
            else:
                out[p + "mlp.correction"] = normal((E,), 0.1)
        size = np.sqrt(size * size + 1.0)
    return out


def standout(cfg, t, token, gain=12.0):
    """Changes the first layer (attention) of the tensors `t` in place: the last channel of every key head, which no rotation
    reaches, is large for `token` and small for every other token, and every query has a large fixed part there, so that the
    score against that token's key stands out; the token's value is made large too."""
    m = cfg["layers"][0]["mixer"]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    assert m["rot"]["dims"] < d
    x = t["embed"][token].astype(np.float64) * cfg["embedding"]["scale"]
    rng = np.random.default_rng(5)
    for g in range(G):
        t["l0.mix.k"][g * d + d - 1] = gain * x / (x @ x)
        t["l0.mix.k.b"][g * d + d - 1] = 0.0
    t["l0.mix.q.b"][d - 1::d] = 8.0
    for n in ("q", "k"):
        t["l0.mix.%s.norm" % n][d - 1::d] = 2.0
    t["l0.mix.v"] += (6.0 * np.outer(rng.standard_normal(G * dv), x) / (x @ x)).astype(np.float32)
    return t


def write_folder(path, cfg, tensors):
    from friday_inference_engine_b200.weights import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"),
                      [(n, "BF16", list(x.shape), harness.f32_to_bf16_bytes(x)) for n, x in tensors.items()])
    return path
