"""Host-side logic of the Sabisun family and self-checks of the plain restatement (no GPU)."""
import ctypes as C
import json

import numpy as np
import pytest

from oracle import sabisun as P
from pibidra_cases import tokens
from sabisun_cases import CONFIGS, weights


def test_restatement_mask():
    m = {"size": 3, "keep_first": 2}
    assert P.visible(1, m) == [0, 1] and P.visible(3, m) == [0, 1, 2, 3] and P.visible(9, m) == [0, 1, 7, 8, 9]
    assert P.visible(4, None) == [0, 1, 2, 3, 4] and P.visible(5, {"size": 1, "keep_first": 0}) == [5]
    assert P.visible(6, {"size": 2, "keep_first": 9}) == list(range(7))


def test_restatement_sink():
    s = np.array([0.3, -2.0, 5.0])
    assert np.allclose(P.sink_softmax(s, 1.5), np.exp(s) / (np.exp(1.5) + np.exp(s).sum()))
    assert np.allclose(P.sink_softmax(s, None).sum(), 1.0)
    assert P.sink_softmax(np.array([-400.0]), 300.0)[0] < 1e-100


def test_restatement_streams():
    x, y = np.arange(6.0).reshape(3, 1, 2), np.array([[10.0, 20.0]])
    mix = np.arange(9.0).reshape(3, 3)
    new = P.hyper_write(x, mix, np.array([1.0, 2.0, 3.0]), 0.5, y)
    assert np.allclose(new[1], 1 * x[0] + 4 * x[1] + 7 * x[2] + 0.5 * 2 * y)          # mix is indexed from, to
    assert np.allclose(P.hyper_read(x, np.array([1.0, -1.0, 2.0])), x[0] - x[1] + 2 * x[2])


def test_restatement_convolution_and_recurrence():
    g = np.random.default_rng(0)
    u, w, b = g.standard_normal((7, 3)), g.standard_normal((3, 4)), g.standard_normal(3)
    y = P.causal_conv(u, w, b)
    assert np.allclose(y[0], b + w[:, 3] * u[0]) and np.allclose(y[5], b + sum(w[:, k] * u[2 + k] for k in range(4)))
    # the recurrence in closed form
    x, B, Cm, dt = g.standard_normal((6, 4, 2)), g.standard_normal((6, 2, 3)), g.standard_normal((6, 2, 3)), g.uniform(0.1, 1, (6, 4))
    A, D = g.standard_normal(4), g.standard_normal(4)
    y, st = P.ssm(x, B, Cm, dt, A, D)
    a = np.cumsum(-np.exp(A) * dt, 0)
    for h in range(4):
        want = sum(np.exp(a[5, h] - a[s, h]) * dt[s, h] * (Cm[5, h // 2] @ B[s, h // 2]) * x[s, h] for s in range(6)) + D[h] * x[5, h]
        assert np.allclose(y[5, h], want)
    y1, st1 = P.ssm(x[:4], B[:4], Cm[:4], dt[:4], A, D)
    y2, st2 = P.ssm(x[4:], B[4:], Cm[4:], dt[4:], A, D, st1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(st2, st)


def test_restatement_norm_parts():
    got = P.group_norm(np.array([[3.0, 4.0, 1.0, 1.0]]), np.ones(4), 2, 0.0)
    assert np.allclose(got, [[3 / np.sqrt(12.5), 4 / np.sqrt(12.5), 1.0, 1.0]])


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_weights_make_mechanisms_visible(name):
    """One key more or less in a window or among the kept ones, the sinks, the streams' coefficients and the states' decays all
    move the logits of the small models by much more than the tests' bounds."""
    cfg = CONFIGS[name]
    t, tok = weights(cfg), tokens(120, cfg["vocab"])
    base = P.forward(cfg, t, tok)

    def moved(change_mask=None, **tensors):
        c = json.loads(json.dumps(cfg))
        for l in c["layers"]:
            if l["type"] == "attention" and change_mask:
                l["mixer"]["mask"][change_mask[0]] = max(0, l["mixer"]["mask"][change_mask[0]] + change_mask[1])
        return np.abs(P.forward(c, {**t, **tensors}, tok) - base).max() / base.std()

    if any(l["type"] == "attention" for l in cfg["layers"]):
        for key in ("keep_first", "size"):
            assert moved((key, 1)) > 0.01 and moved((key, -1)) > 0.01, key
    for k in t:
        if k.endswith("sink"):
            assert moved(**{k: t[k] - 20}) > 0.5
        if k.endswith(("A_log", "dt_bias", "mix.D", "conv.b")):
            assert moved(**{k: t[k] + 0.5}) > 0.02, k
        if ".hc" in k and cfg["streams"] > 1 and k != "l0.hc1.in":            # the streams start equal
            assert moved(**{k: t[k].T.copy() if t[k].ndim == 2 else t[k] * np.arange(1, cfg["streams"] + 1)}) > 0.01, k


def test_config_reader():
    from flexllm_b200 import _lib, models
    cfg = CONFIGS["odd"]
    c, l = models.sabisun_config(cfg, 2, 32, 100, _lib.BF16)
    assert (c.layers, c.width, c.vocab, c.streams, c.loop_times, c.max_batch, c.max_prefill, c.max_ctx) == (6, 90, 301, 4, 0, 2, 32, 100)
    assert abs(c.residual_mult - 1.3) < 1e-6 and abs(c.logit_scale - 1.7) < 1e-6 and c.embed_scale == 1.0
    assert (l[0].mixer, l[0].heads, l[0].vdim, l[0].state, l[0].groups, l[0].conv, l[0].norm_groups, l[0].ff) == (_lib.MIXER_SSM, 6, 20, 12, 3, 2, 8, 60)
    assert (l[1].mixer, l[1].heads, l[1].kv_heads, l[1].dim, l[1].vdim, l[1].window, l[1].keep_first, l[1].kv_from, l[1].ff) == (0, 5, 1, 20, 12, 33, 70, -1, 0)
    assert l[3].kv_from == 1 and l[3].keep_first == 0 and abs(l[3].scale - 0.2) < 1e-6
    for where, key, v in ((0, "type", "other"), (0, "mlp", {"kind": "other", "ff": 8})):
        bad = json.loads(json.dumps(cfg))
        bad["layers"][where][key] = v
        with pytest.raises(ValueError):
            models.sabisun_config(bad, 1, 8, 8, 0)


def test_registry():
    from flexllm_b200 import models
    assert models.entry({"architecture": "Sabisun"}).dtypes == ("bfloat16", "float32")
    with pytest.raises(models.UnsupportedDtype):
        models.create(CONFIGS["plain"], dtype="int8")


def test_configuration_is_checked_without_a_gpu():
    from flexllm_b200 import _lib, build, models
    build.build()
    lib = _lib.load()
    h = C.c_void_p()

    def status(i, **change):
        cfg = json.loads(json.dumps(CONFIGS["odd"]))
        cfg["layers"][i]["mixer"].update(change)
        c, keep = models.sabisun_config(cfg, 1, 8, 8, _lib.BF16)
        return lib.flexllm_model_create_decoder(C.byref(h), C.byref(c))
    assert status(0, groups=4) == _lib.EINVAL and status(0, norm_groups=7) == _lib.EINVAL and status(0, conv=0) == _lib.EINVAL
    assert status(1, kv_heads=2) == _lib.EINVAL and status(1, mask={"size": 0}) == _lib.EINVAL
    assert status(3, kv_from=3) == _lib.EINVAL and status(3, kv_from=0) == _lib.EINVAL and status(5, kv_from=3) == _lib.EINVAL
    assert status(3, dim=24) == _lib.EINVAL
    cfg = dict(CONFIGS["odd"], streams=9)
    c, keep = models.sabisun_config(cfg, 1, 8, 8, _lib.BF16)
    assert lib.flexllm_model_create_decoder(C.byref(h), C.byref(c)) == _lib.ENOTSUP
