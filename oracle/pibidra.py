"""Plain, slow restatement of the Pibidra decoder in float64 numpy, one function per mechanism.

Test infrastructure: nothing here is shared with the product (own config access, own loops over heads and
positions), and nothing here is fast. `forward` takes a parsed config and a dict of tensors (numpy, any float
type) and returns the logits of every position, optionally with the residual stream after every layer run.
"""
import math

import numpy as np

F = np.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm_zero_centred(x, w, eps):
    """Weight stored around zero: rms(x) * (1 + w)."""
    return rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def linear(w, x, b=None):
    y = x @ w.T
    return y if b is None else y + b


def bucket(n, rows, bias_max):
    """Row of the distance table for distance n: exact up to half the rows, logarithmic up to bias_max after it."""
    half = rows // 2
    if n < half:
        return n
    if half == 0 or bias_max <= half:
        return rows - 1
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(bias_max / half) * (rows - half)))


def distance_bias(table, bias_max, n):
    """table [rows, heads] -> the heads' biases at distance n."""
    return table[bucket(n, table.shape[0], bias_max)]


def softcapped(s, cap):
    return cap * np.tanh(s / cap)


def window_keys(i, size):
    """Positions that position i sees: itself and the size - 1 before it."""
    return range(max(0, i - size + 1), i + 1)


def sink_softmax(s):
    """exp(s_j) / (1 + sum exp(s_j)): a sink of score 0 without a value."""
    m = max(0.0, float(s.max()))
    e = np.exp(s - m)
    return e / (math.exp(-m) + e.sum())


def head_outputs(q, k, v, table, mx, sink=True):
    """q [S, H, dk], k [S, G, dk], v [S, G, dv] (normed already) -> [S, H, dv]. mx: window (mask.size), scale, softcap, bias_max."""
    S, H, _ = q.shape
    G, size = k.shape[1], mx["mask"]["size"]
    bias = np.stack([distance_bias(table, mx["bias_max"], n) for n in range(min(size, S))])           # [distance, H]
    o = np.zeros((S, H, v.shape[2]), F)
    for i in range(S):
        keys = np.array(window_keys(i, size))
        for hd in range(H):
            g = hd // (H // G)
            s = k[keys, g] @ q[i, hd] * mx["scale"]
            if mx["softcap"]:
                s = softcapped(s, mx["softcap"])
            s = s + bias[i - keys, hd]
            p = sink_softmax(s) if sink else np.exp(s - s.max()) / np.exp(s - s.max()).sum()
            o[i, hd] = p @ v[keys, g]
    return o


def attention(h, t, pre, mx, eps):
    """The mixer on h [S, width]; t: tensors, pre: 'l<i>.mix.'."""
    S = h.shape[0]
    H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = linear(t[pre + "q"], h, t[pre + "q.b"])
    k = linear(t[pre + "k"], h, t[pre + "k.b"])
    v = linear(t[pre + "v"], h, t[pre + "v.b"])
    q = norm_plain(q, t[pre + "q.norm"], eps).reshape(S, H, dk)      # the norm runs over all heads at once
    k = norm_plain(k, t[pre + "k.norm"], eps).reshape(S, G, dk)
    o = head_outputs(q, k, v.reshape(S, G, dv), t[pre + "rel"], mx).reshape(S, H * dv)
    return linear(t[pre + "o"], o * sigmoid(linear(t[pre + "g"], h)))


def feed_forward(h, t, pre):
    return linear(t[pre + "down"], gelu_tanh(linear(t[pre + "gate"], h)) * linear(t[pre + "up"], h))


def layer(x, t, i, spec, eps):
    p = "l%d." % i
    x = x + norm_zero_centred(attention(norm_zero_centred(x, t[p + "norm1"], eps), t, p + "mix.", spec["mixer"], eps), t[p + "norm1b"], eps)
    if spec["mlp"] is not None:
        x = x + norm_zero_centred(feed_forward(norm_zero_centred(x, t[p + "norm2"], eps), t, p + "mlp."), t[p + "norm2b"], eps)
    return x


def layer_runs(cfg):
    """[(layer, pass or None)] in the order they run; pass is given on the first layer of a pass."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        out += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return out + [(i, None) for i in range(lp["stop"], n)]


def forward(cfg, tensors, tokens, want_layers=False):
    t = {k: np.asarray(v, F) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    emb = t["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    x, trace = emb, []
    for i, p in layer_runs(cfg):
        if p is not None:
            if p > 0:
                x = x + emb
            x = x + t["loop.step"][p]
        x = layer(x, t, i, cfg["layers"][i], eps)
        trace.append(x)
    logits = linear(t["head"], norm_zero_centred(x, t["final.norm"], eps))
    return (logits, np.stack(trace)) if want_layers else logits
