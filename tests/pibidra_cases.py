"""Small random models of the Pibidra design for the tests: configurations, weights that make every mechanism visible, and
a .safetensors writer."""
import json
import os
import struct

import numpy as np


def bf16_round(a):
    """float32 values rounded to bfloat16 (nearest even)."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    u = (u + 0x7fff + ((u >> 16) & 1)) & np.uint32(0xffff0000)
    return u.view(np.float32)


def attn(heads, kv_heads, dim, vdim, window, ff=None, bias_max=50, softcap=12.0, scale=None):
    return {"type": "attention",
            "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask={"size": window}, bias_max=bias_max,
                          softcap=softcap, scale=scale if scale is not None else dim ** -0.5),
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width, vocab, loop=None, eps=1e-5, emb_scale=0.7):
    c = {"architecture": "Pibidra", "embedding": {"scale": emb_scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


# heads, key/value heads, sizes, windows and loops that differ from one another, sizes that are no multiples of 8 or 16,
# a layer without feed-forward, one head, equal and unequal query and value sizes
CONFIGS = {
    "plain": config([attn(4, 2, 64, 64, 50, 128), attn(4, 2, 64, 64, 50, 128)], 128, 256),
    "mixed": config([attn(6, 2, 40, 24, 33, 100, 40, 9.0), attn(5, 1, 20, 12, 20, None, 17, 20.0, 0.3), attn(2, 2, 72, 136, 90, 48, 64, 5.0)],
                    90, 301, loop=(1, 2, 3), emb_scale=1.3),
    "looped": config([attn(1, 1, 32, 16, 65, 64), attn(8, 2, 16, 48, 64, 64, 100), attn(3, 3, 48, 48, 63, 80), attn(4, 1, 24, 32, 1, 32)],
                     104, 200, loop=(0, 3, 2), eps=1e-4),
    "once": config([attn(4, 4, 128, 80, 130, 160, 128, 30.0), attn(2, 1, 8, 8, 40, 16)], 64, 128, loop=(1, 2, 1)),
}


def table_rows(i):
    return (16, 12, 32, 7)[i % 4]


def weights(cfg, seed=0):
    """bf16-representable float32 tensors. Queries and keys share a common part, so that some keys stand out, and norm
    weights, biases, tables and gates are large enough to be seen in the logits."""
    g = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    rn = lambda *sh, s=1.0: bf16_round(g.standard_normal(sh) * s)
    t = {"embed": rn(V, D), "head": rn(V, D, s=D ** -0.5), "final.norm": rn(D, s=0.2)}
    if cfg.get("loop"):
        t["loop.step"] = rn(cfg["loop"]["times"], D, s=0.5)
    for i, l in enumerate(cfg["layers"]):
        p, m = "l%d." % i, l["mixer"]
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l["mlp"] else ()):
            t[p + n] = rn(D, s=0.3)
        common = g.standard_normal((dk, D))
        mat = lambda heads: bf16_round((np.concatenate([common + 0.7 * g.standard_normal((dk, D)) for _ in range(heads)])) * D ** -0.5)
        t[p + "mix.q"], t[p + "mix.k"] = mat(H), mat(G)
        t[p + "mix.v"] = rn(G * dv, D, s=D ** -0.5)
        t[p + "mix.q.b"], t[p + "mix.k.b"], t[p + "mix.v.b"] = rn(H * dk, s=0.3), rn(G * dk, s=0.3), rn(G * dv, s=0.3)
        t[p + "mix.q.norm"], t[p + "mix.k.norm"] = bf16_round(1.2 + 0.4 * g.standard_normal(H * dk)), bf16_round(1.2 + 0.4 * g.standard_normal(G * dk))
        t[p + "mix.rel"] = rn(table_rows(i), H, s=1.0)
        t[p + "mix.g"] = rn(H * dv, D, s=D ** -0.5)
        t[p + "mix.o"] = rn(D, H * dv, s=(H * dv) ** -0.5)
        if l["mlp"]:
            f = l["mlp"]["ff"]
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = rn(f, D, s=D ** -0.5), rn(f, D, s=D ** -0.5), rn(D, f, s=f ** -0.5)
    return t


def write_folder(folder, cfg, t):
    """config.json and model.safetensors (bf16)."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {"__metadata__": {"format": "pt"}}, [], 0
    for k, v in t.items():
        b = (np.ascontiguousarray(v, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        head[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    h = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))


def tokens(n, vocab, seed=0):
    """Random ids in which earlier stretches come back later (keys that match from far away)."""
    g = np.random.default_rng(seed)
    x = g.integers(0, vocab, n)
    for _ in range(max(1, n // 20)):
        a, b, w = g.integers(0, n, 3)
        w = 1 + w % 5
        m = min(w, n - max(a, b))
        x[b:b + m] = x[a:a + m]
    return [int(v) for v in x]


def rel_err(got, want):
    """Root mean square error over the vocabulary (means taken off) relative to the reference's spread, per row."""
    d = np.asarray(got, np.float64) - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / want.std()
