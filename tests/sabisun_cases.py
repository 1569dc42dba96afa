"""Small random models of the Sabisun design for the tests: configurations and weights that make every mechanism visible."""
import numpy as np

from pibidra_cases import bf16_round


def attn(heads, kv_heads, dim, vdim, window, keep, ff=None, scale=None, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask={"size": window, "keep_first": keep}, scale=scale if scale else 1.4 * dim ** -0.5)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def ssm(heads, vdim, state, groups, conv, norm_groups, ff=None):
    return {"type": "mamba2", "mixer": dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups),
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width, vocab, streams, mult=0.7, logit_scale=0.8, eps=1e-5):
    return {"architecture": "Sabisun", "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "residual_mult": mult, "streams": streams,
            "vocab": vocab, "width": width}


# head counts, sizes, windows, kept tokens (inside a page, over a page, none, more than the window), taps and groups that differ from one
# another, sizes that are no multiples of 8 or 16, parts of the norm that cross heads, layers without feed-forward
CONFIGS = {
    "plain": config([ssm(4, 32, 32, 2, 4, 2, 96), attn(4, 2, 32, 32, 50, 5, 96), ssm(4, 32, 32, 2, 4, 2, 96), attn(4, 2, 32, 32, 50, 5, 96, kv_from=1)],
                    96, 200, 3),
    "odd": config([ssm(6, 20, 12, 3, 2, 8, 60), attn(5, 1, 20, 12, 33, 70, None, 0.3), ssm(3, 40, 72, 1, 5, 1), attn(5, 1, 20, 12, 90, 0, 44, 0.2, kv_from=1),
                   attn(3, 3, 24, 40, 1, 3, 36), attn(5, 1, 20, 12, 33, 70, 50, 0.4, kv_from=1)], 90, 301, 4, 1.3, 1.7, 1e-4),
    "wide": config([attn(2, 1, 128, 80, 70, 64, 40, 0.05), ssm(2, 72, 136, 1, 1, 3, 40), attn(2, 2, 72, 136, 64, 15, 40, 0.06), attn(2, 1, 128, 80, 20, 30, 40, 0.04, kv_from=0)],
                   72, 128, 1, 1.0, 1.0),
    "states": config([ssm(8, 16, 64, 8, 3, 4, 64), ssm(2, 100, 24, 2, 4, 5)], 80, 160, 2, 0.5),
    "keys": config([attn(8, 2, 16, 16, 40, 12, 64), attn(8, 2, 16, 16, 200, 1, 64, kv_from=0)], 64, 150, 5, 0.9, 0.6),
}


def weights(cfg, seed=0):
    """bf16-representable float32 tensors. Queries and keys share a common part, so that some keys stand out; sinks take a good
    part of the weight; states decay at rates from a few to hundreds of tokens; the stream coefficients differ."""
    g = np.random.default_rng(seed)
    D, V, n = cfg["width"], cfg["vocab"], cfg["streams"]
    rn = lambda *sh, s=1.0: bf16_round(g.standard_normal(sh) * s)
    t = {"embed": rn(V, D), "final.norm": bf16_round(1 + 0.2 * g.standard_normal(D))}
    for i, l in enumerate(cfg["layers"]):
        p, m = "l%d." % i, l["mixer"]
        for q in (1, 2) if l["mlp"] else (1,):
            t[p + "norm%d" % q] = bf16_round(1 + 0.2 * g.standard_normal(D))
            t[p + "hc%d.in" % q] = bf16_round(g.uniform(0.2, 1.0, n))
            t[p + "hc%d.out" % q] = bf16_round(g.uniform(0.4, 1.4, n))
            t[p + "hc%d.mix" % q] = bf16_round(np.eye(n) * 0.85 + 0.12 * g.standard_normal((n, n)))
        if l["type"] == "attention":
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            common = np.random.default_rng(1000).standard_normal((dk, D))
            mat = lambda heads: bf16_round(np.concatenate([common + 0.7 * g.standard_normal((dk, D)) for _ in range(heads)]) * D ** -0.5)
            t[p + "mix.q"] = mat(H)
            if "kv_from" not in m:
                t[p + "mix.k"] = mat(G)
                t[p + "mix.v"] = rn(G * dv, D, s=1.5 * D ** -0.5)
            t[p + "mix.sink"] = bf16_round(m["scale"] * dk + g.uniform(1.5, 4.0, H))          # scores lie around scale * dim
            t[p + "mix.o"] = rn(D, H * dv, s=2 * (H * dv) ** -0.5)
        else:
            H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            inner, ch = H * P, H * P + 2 * G * N
            t[p + "mix.in"] = rn(inner + ch + H, D, s=D ** -0.5)
            t[p + "mix.conv"], t[p + "mix.conv.b"] = rn(ch, m["conv"], s=0.7), rn(ch, s=0.2)
            t[p + "mix.dt_bias"], t[p + "mix.A_log"] = bf16_round(g.uniform(-3.5, 0.5, H)), bf16_round(g.uniform(-4.0, 1.0, H))
            t[p + "mix.D"] = bf16_round(1 + 0.3 * g.standard_normal(H))
            t[p + "mix.norm"] = bf16_round(1 + 0.2 * g.standard_normal(inner))
            t[p + "mix.o"] = rn(D, inner, s=inner ** -0.5)
        if l["mlp"]:
            f = l["mlp"]["ff"]
            t[p + "mlp.up"], t[p + "mlp.down"] = rn(f, D, s=D ** -0.5), rn(D, f, s=f ** -0.5)
    return t
