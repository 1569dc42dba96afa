"""Plain, slow restatement of the Sabisun decoder in float64 numpy, one function per mechanism.

Test infrastructure: nothing here is shared with the product, and nothing here is fast. `forward` takes a parsed config and a
dict of tensors (numpy, any float type) and returns the logits of every position, optionally with the sum of the residual
streams after every layer. `act` is applied to every activation that may be kept in 16 bits (sublayer inputs, projections, keys and
values, convolution outputs, gated outputs): with a rounding function it tells how much rounding alone moves the results.
"""
import math

import numpy as np

F = np.float64


def exact(v):
    return v


def rms_norm(x, eps, w=1.0):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def silu(z):
    return z / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def linear(w, x):
    return x @ w.T


# ------------------------------------------------------------------------------------------ residual streams
def hyper_read(xs, w_in):
    """xs [streams, S, width] -> the sublayer's input before its norm."""
    return sum(w_in[s] * xs[s] for s in range(len(xs)))


def hyper_write(xs, mix, out, mult, y):
    """New streams: stream t = sum_s mix[from s, to t] * (old) stream s + mult * out[t] * y."""
    n = len(xs)
    return np.stack([sum(mix[s, t] * xs[s] for s in range(n)) + mult * out[t] * y for t in range(n)])


# ------------------------------------------------------------------------------------------ attention
def visible(i, mask):
    """Positions that position i sees: a window of mask.size, and the first mask.keep_first; everything up to i without a mask."""
    if not mask:
        return list(range(i + 1))
    return [j for j in range(i + 1) if i - j < mask["size"] or j < mask.get("keep_first", 0)]


def sink_softmax(s, sink):
    """exp(s_j) / (exp(sink) + sum exp(s_j)); sink None: an ordinary softmax."""
    m = s.max() if sink is None else max(float(sink), float(s.max()))
    e = np.exp(s - m)
    return e / (e.sum() + (0.0 if sink is None else math.exp(sink - m)))


def head_outputs(q, k, v, mask, scale, sinks):
    """q [S, H, dk], k [S, G, dk], v [S, G, dv], sinks [H] or None -> [S, H, dv]."""
    S, H, _ = q.shape
    G = k.shape[1]
    o = np.zeros((S, H, v.shape[2]), F)
    for i in range(S):
        keys = visible(i, mask)
        for h in range(H):
            g = h // (H // G)
            o[i, h] = sink_softmax(k[keys, g] @ q[i, h] * scale, None if sinks is None else sinks[h]) @ v[keys, g]
    return o


def keys_values(h, t, pre, mx, act=exact):
    S, G = h.shape[0], mx["kv_heads"]
    return act(linear(t[pre + "k"], h)).reshape(S, G, mx["dim"]), act(linear(t[pre + "v"], h)).reshape(S, G, mx["vdim"])


def attention(h, t, pre, mx, kv, act=exact):
    """The mixer on h [S, width] with the keys and values kv (its own or another layer's)."""
    S, H = h.shape[0], mx["heads"]
    q = act(linear(t[pre + "q"], h)).reshape(S, H, mx["dim"])
    o = head_outputs(q, kv[0], kv[1], mx.get("mask"), mx["scale"], t[pre + "sink"])
    return linear(t[pre + "o"], act(o.reshape(S, H * mx["vdim"])))


# ------------------------------------------------------------------------------------------ state-space mixer
def causal_conv(u, w, b):
    """u [S, channels], w [channels, taps] (last column: the current token) -> [S, channels]."""
    S, taps = u.shape[0], w.shape[1]
    y = np.zeros_like(u)
    for t in range(S):
        y[t] = b
        for k in range(taps):
            j = t - (taps - 1) + k
            if j >= 0:
                y[t] = y[t] + w[:, k] * u[j]
    return y


def ssm(x, B, C, dt, A_log, D, state=None):
    """x [S, heads, vdim], B and C [S, groups, N], dt [S, heads] (after softplus) -> y [S, heads, vdim], final state
    [heads, N, vdim]. S_t = exp(-exp(A_log) dt) S_{t-1} + dt B x^T;  y = S_t^T C + D x."""
    S, H, P = x.shape
    G, N = B.shape[1:]
    st = np.zeros((H, N, P), F) if state is None else np.array(state, F)
    y = np.zeros((S, H, P), F)
    for t in range(S):
        for h in range(H):
            g = h // (H // G)
            st[h] = math.exp(-math.exp(A_log[h]) * dt[t, h]) * st[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = st[h].T @ C[t, g] + D[h] * x[t, h]
    return y, st


def group_norm(y, w, groups, eps):
    """rms norm of y in `groups` equal parts, times w."""
    S, n = y.shape
    return rms_norm(y.reshape(S, groups, n // groups), eps).reshape(S, n) * w


def mamba2(h, t, pre, mx, eps, act=exact):
    p = act(linear(t[pre + "in"], h))
    w = [t[pre + n] for n in ("conv", "conv.b", "dt_bias", "A_log", "D", "norm")]
    return linear(t[pre + "o"], mamba2_inner(p, *w, mx, eps, act))


def mamba2_inner(p, conv, conv_b, dt_bias, A_log, D, gain, mx, eps, act=exact):
    """The mixer between its projections: p [S, z | x | B | C | dt] -> [S, inner]."""
    S = p.shape[0]
    H, P, N, G = mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * P
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = act(silu(causal_conv(xbc, conv, conv_b)))
    x, B, C = xbc[:, :inner], xbc[:, inner:inner + G * N], xbc[:, inner + G * N:]
    y, _ = ssm(x.reshape(S, H, P), B.reshape(S, G, N), C.reshape(S, G, N), softplus(dt + dt_bias), A_log, D)
    return act(group_norm(act(y.reshape(S, inner) * silu(z)), gain, mx["norm_groups"], eps))


# ------------------------------------------------------------------------------------------ the model
def feed_forward(h, t, pre, act=exact):
    return linear(t[pre + "down"], act(np.maximum(linear(t[pre + "up"], h), 0.0) ** 2))


def forward(cfg, tensors, tokens, want_layers=False, act=exact):
    t = {k: np.asarray(v, F) for k, v in tensors.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    xs = np.stack([t["embed"][np.asarray(tokens)]] * cfg["streams"])
    kv, trace = {}, []
    for i, spec in enumerate(cfg["layers"]):
        p, mx = "l%d." % i, spec["mixer"]
        h = act(rms_norm(hyper_read(xs, t[p + "hc1.in"]), eps, t[p + "norm1"]))
        if spec["type"] == "mamba2":
            y = mamba2(h, t, p + "mix.", mx, eps, act)
        else:
            src = mx.get("kv_from")
            kv[i] = kv[src] if src is not None else keys_values(h, t, p + "mix.", mx, act)
            y = attention(h, t, p + "mix.", mx, kv[i], act)
        xs = hyper_write(xs, t[p + "hc1.mix"], t[p + "hc1.out"], mult, y)
        if spec["mlp"] is not None:
            h = act(rms_norm(hyper_read(xs, t[p + "hc2.in"]), eps, t[p + "norm2"]))
            xs = hyper_write(xs, t[p + "hc2.mix"], t[p + "hc2.out"], mult, feed_forward(h, t, p + "mlp.", act))
        trace.append(xs.sum(0))
    logits = linear(t["embed"], act(rms_norm(xs.sum(0), eps, t["final.norm"]))) * cfg["logit_scale"]
    return (logits, np.stack(trace)) if want_layers else logits
