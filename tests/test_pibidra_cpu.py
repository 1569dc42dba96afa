"""Host-side logic of the Pibidra family and of the trace replay, and self-checks of the plain restatement (no GPU)."""
import array
import io
import json
import os

import numpy as np
import pytest

from oracle import pibidra as P
from pibidra_cases import CONFIGS, tokens, weights


def test_restatement_buckets():
    assert [P.bucket(n, 16, 100) for n in range(8)] == list(range(8))
    assert P.bucket(8, 16, 100) == 8 and P.bucket(99, 16, 100) == 15 and P.bucket(10 ** 6, 16, 100) == 15
    # 8 * (100/8)^(1/8) = 10.97: 11 is the first distance of the next bucket
    assert P.bucket(10, 16, 100) == 8 and P.bucket(11, 16, 100) == 9


def test_restatement_window_and_sink():
    assert list(P.window_keys(5, 3)) == [3, 4, 5] and list(P.window_keys(1, 3)) == [0, 1] and list(P.window_keys(4, 1)) == [4]
    s = np.array([0.3, -2.0, 5.0])
    assert np.allclose(P.sink_softmax(s), np.exp(s) / (1 + np.exp(s).sum()))
    assert P.sink_softmax(np.array([-400.0]))[0] < 1e-100


def test_restatement_is_causal_and_windowed():
    cfg = CONFIGS["plain"]
    t = weights(cfg)
    a = tokens(120, cfg["vocab"])
    b = list(a)
    b[7] = (b[7] + 1) % cfg["vocab"]
    la, lb = P.forward(cfg, t, a), P.forward(cfg, t, b)
    reach = 2 * 49                                     # two layers of windows of 50
    diff = np.abs(la - lb).max(1)
    assert (diff[:7] == 0).all() and (diff[7:10] > 0).all() and (diff[7 + reach + 1:] == 0).all()


def test_restatement_loop_runs():
    assert P.layer_runs(CONFIGS["mixed"]) == [(0, None), (1, 0), (1, 1), (1, 2), (2, None)]
    assert [i for i, _ in P.layer_runs(CONFIGS["looped"])] == [0, 1, 2, 0, 1, 2, 3]
    once, t = CONFIGS["once"], weights(CONFIGS["once"])
    flat = {k: v for k, v in once.items() if k != "loop"}
    tok = tokens(20, once["vocab"])
    assert np.abs(P.forward(once, t, tok) - P.forward(flat, t, tok)).max() > 0.01       # one pass still adds its vector


def test_config_reader():
    from flexllm_b200 import _lib, models
    cfg = CONFIGS["mixed"]
    c, layers = models.pibidra_config(cfg, 2, 32, 100, _lib.BF16)
    assert (c.layers, c.width, c.vocab, c.loop_start, c.loop_stop, c.loop_times, c.max_batch, c.max_prefill, c.max_ctx) == (3, 90, 301, 1, 2, 3, 2, 32, 100)
    assert abs(c.embed_scale - 1.3) < 1e-6 and abs(c.eps - 1e-5) < 1e-11
    l = layers[1]
    assert (l.heads, l.kv_heads, l.dim, l.vdim, l.window, l.bias_max, l.ff) == (5, 1, 20, 12, 20, 17, 0)
    assert abs(l.scale - 0.3) < 1e-6 and l.softcap == 20.0
    c, _ = models.pibidra_config(CONFIGS["plain"], 1, 8, 8, _lib.F32)
    assert c.loop_times == 0
    bad = json.loads(json.dumps(cfg))
    bad["layers"][1]["type"] = "other"
    with pytest.raises(ValueError):
        models.pibidra_config(bad, 1, 8, 8, 0)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mlp"]["kind"] = "other"
    with pytest.raises(ValueError):
        models.pibidra_config(bad, 1, 8, 8, 0)


def test_registry():
    from flexllm_b200 import models
    assert {"Pibidra", "SpinQuantLlama"} <= set(models.REGISTRY)
    with pytest.raises(ValueError):
        models.create({"architecture": "nothing"})
    with pytest.raises(models.UnsupportedDtype):
        models.create(CONFIGS["plain"], dtype="int8")


def test_configuration_is_checked_without_a_gpu():
    import ctypes as C
    from flexllm_b200 import _lib, build, models
    build.build()
    lib = _lib.load()
    h = C.c_void_p()
    for change in (dict(kv_heads=3), dict(dim=0), dict(mask={"size": 0})):
        cfg = json.loads(json.dumps(CONFIGS["plain"]))
        cfg["layers"][0]["mixer"].update(change)
        c, keep = models.pibidra_config(cfg, 1, 8, 8, _lib.BF16)
        assert lib.flexllm_model_create_decoder(C.byref(h), C.byref(c)) == _lib.EINVAL
    cfg = json.loads(json.dumps(CONFIGS["mixed"]))
    cfg["loop"]["stop"] = 9
    c, keep = models.pibidra_config(cfg, 1, 8, 8, _lib.BF16)
    assert lib.flexllm_model_create_decoder(C.byref(h), C.byref(c)) == _lib.EINVAL


class FakeModel:
    vocab = 3

    def __init__(self):
        self.log = []

    def reset(self):
        self.log.append("reset")

    def step(self, batch, want=(), next_token=False):
        self.log.append((batch, list(want)))
        return array.array("f", [0.5] * (len(want) * self.vocab)), None

    def close(self):
        self.log.append("close")


def test_replay_keeps_one_request_live():
    from flexllm_b200.trace import Replay
    m = FakeModel()
    r = Replay(m)
    assert len(r.step([{"id": "a", "tokens": [1, 2], "want": [1]}], [])) == 3
    r.step([{"id": "a", "tokens": [0], "want": []}], ["a"])
    r.step([{"id": "b", "tokens": [2], "want": [0]}], ["b"])
    assert m.log == ["reset", ([[1, 2]], [1]), ([[0]], []), "reset", "reset", ([[2]], [0]), "reset"]
    r.step([{"id": "c", "tokens": [1], "want": []}], [])
    with pytest.raises(ValueError):
        r.step([{"id": "d", "tokens": [1], "want": []}], [])
    with pytest.raises(ValueError):
        r.step([{"id": "c", "tokens": [1]}, {"id": "d", "tokens": [1]}], [])


def test_replay_program(monkeypatch, tmp_path, capsys):
    from flexllm_b200 import build, models, trace
    monkeypatch.setattr(build, "build", lambda *a, **k: None)
    monkeypatch.setattr(models, "load", lambda *a, **k: FakeModel())
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 0], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [1], "want": []}], "end": ["a"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    assert trace.main(["--model", "m", "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "9"]) == 0
    assert capsys.readouterr().out == "done 0\ndone 1\n"
    assert np.fromfile(tmp_path / "0.f32", "<f4").size == 6 and not os.path.exists(tmp_path / "1.f32")

    def refuse(*a, **k):
        raise models.UnsupportedDtype("no")
    monkeypatch.setattr(models, "load", refuse)
    assert trace.main(["--model", "m", "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "9"]) == 3
