"""Model registry, configuration and host-side generation (ctypes only; no torch).

A model folder holds ``config.json``, whose ``architecture`` names an entry of ``REGISTRY``, and its weights. An entry
turns a configuration into a runner handle (``create``) and fills it (``load_weights``); everything after that -- steps,
generation, sampling, the cache -- is the library's runner, the same for every entry.
"""
import array
import ctypes as C
import json
import math
import os

from . import _lib
from .runtime import call, check, lib

DTYPES = {"bfloat16": _lib.BF16, "float32": _lib.F32}


class UnsupportedDtype(ValueError):
    """The architecture does not compute in the asked-for number format."""


def _i32(values):
    return (C.c_int32 * max(1, len(values)))(*values)


class HostModel:
    """A model of any family, driven through host buffers."""

    def __init__(self, handle, vocab):
        self._h, self.vocab = handle, vocab

    def close(self):
        if self._h:
            lib().flexllm_model_destroy(self._h)
            self._h = C.c_void_p()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    def limits(self):
        b, p, c = C.c_int(), C.c_int(), C.c_int()
        call("flexllm_model_limits", self._h, C.byref(b), C.byref(p), C.byref(c))
        return dict(max_batch=b.value, max_prefill=p.value, max_ctx=c.value)

    def reset(self):
        """Ends the live sequences; the next step starts new ones at position 0."""
        call("flexllm_model_reset", self._h, None)

    def step(self, batch, want=(), next_token=False):
        """The next tokens of the live sequences (lists of equal length, one per sequence). ``want``: indices into the
        flattened tokens. Returns (array('f') of len(want) * vocab logits, next tokens or None)."""
        B, n = len(batch), len(batch[0])
        flat = _i32([t for row in batch for t in row])
        lg = array.array("f", bytes(4 * len(want) * self.vocab))
        buf = (C.c_float * len(lg)).from_buffer(lg) if len(want) else None
        nx = (C.c_int32 * B)() if next_token else None
        call("flexllm_model_extend_host", self._h, flat, B, n, _i32(list(want)), len(want), buf, nx, None)
        return lg, list(nx) if next_token else None

    def generate(self, prompts, n_new, use_graph=True):
        """Prompts of equal length -> n_new tokens each."""
        B, n = len(prompts), len(prompts[0])
        if any(len(p) != n for p in prompts):
            raise ValueError("the prompts of a batch have one length")
        out = (C.c_int32 * (B * n_new))()
        call("flexllm_model_generate_host", self._h, _i32([t for p in prompts for t in p]), B, n, n_new, out, 1 if use_graph else 0, None)
        return [list(out[b * n_new:(b + 1) * n_new]) for b in range(B)]

    def set_sampling_host(self, lanes=0, top_k=0, rnd=(), n_new=1, B=1):
        """top_k 0: greedy. Else top-k sampling with uniform numbers rnd, n_new rows of B."""
        call("flexllm_model_set_sampling_host", self._h, lanes, top_k, (C.c_float * max(1, len(rnd)))(*rnd), n_new, B)


# --------------------------------------------------------------------------------------------- decoder family
ALL = 2 ** 31 - 1       # window of a layer without one


def create_decoder(cfg, c_config):
    h = C.c_void_p()
    call("flexllm_model_create_decoder", C.byref(h), C.byref(c_config))
    return HostModel(h, cfg["vocab"])


def load_safetensors(model, folder):
    call("flexllm_model_load_safetensors", model._h, os.path.join(folder, "model.safetensors").encode(), None)


# --------------------------------------------------------------------------------------------- Pibidra
def pibidra_config(cfg, max_batch, max_prefill, max_ctx, dtype):
    """config.json -> (C configuration, the layer array it points to)."""
    n = len(cfg["layers"])
    layers = (_lib.DecoderLayer * n)()
    for i, l in enumerate(cfg["layers"]):
        if l["type"] != "attention":
            raise ValueError("layer %d: unknown mixer %r" % (i, l["type"]))
        m, f = l["mixer"], l.get("mlp")
        if f is not None and f.get("kind", "dense") != "dense":
            raise ValueError("layer %d: unknown feed-forward %r" % (i, f["kind"]))
        mask = m.get("mask")
        layers[i] = _lib.DecoderLayer(m["heads"], m["kv_heads"], m["dim"], m["vdim"], mask["size"] if mask else ALL, m["bias_max"],
                                      m["scale"], m.get("softcap") or 0.0, f["ff"] if f else 0, _lib.MIXER_ATTENTION, _lib.ATTN_PIBIDRA,
                                      _lib.FF_GELU_GATE, 0, -1)
    loop = cfg.get("loop") or dict(start=0, stop=0, times=0)
    c = _lib.DecoderConfig(n, cfg["width"], cfg["vocab"], cfg["norm"]["eps"], cfg["embedding"]["scale"], loop["start"], loop["stop"],
                           loop["times"], max_batch, max_prefill, max_ctx, dtype, layers)
    return c, layers


class Pibidra:
    """Sandwich-normed decoder with windowed attention, distance bias, sink and looped layers; one .safetensors file."""
    name = "Pibidra"
    dtypes = ("bfloat16", "float32")

    @staticmethod
    def create(cfg, max_batch, max_prefill, max_ctx, dtype):
        c, keep = pibidra_config(cfg, max_batch, max_prefill, max_ctx, DTYPES[dtype])
        return create_decoder(cfg, c)

    @staticmethod
    def load_weights(model, folder, cfg):
        load_safetensors(model, folder)


# --------------------------------------------------------------------------------------------- Sabisun
def sabisun_config(cfg, max_batch, max_prefill, max_ctx, dtype):
    """config.json -> (C configuration, the layer array it points to)."""
    n = len(cfg["layers"])
    layers = (_lib.DecoderLayer * n)()
    for i, l in enumerate(cfg["layers"]):
        m, f = l["mixer"], l.get("mlp")
        if f is not None and f.get("kind", "dense") != "dense":
            raise ValueError("layer %d: unknown feed-forward %r" % (i, f["kind"]))
        d = layers[i]
        d.heads, d.vdim, d.kv_from = m["heads"], m["vdim"], -1
        d.ff, d.act = f["ff"] if f else 0, _lib.FF_RELU2
        if l["type"] == "attention":
            mask = m.get("mask")
            d.mixer, d.features = _lib.MIXER_ATTENTION, _lib.ATTN_HEAD_SINKS
            d.kv_heads, d.dim, d.scale = m["kv_heads"], m["dim"], m["scale"]
            d.window, d.keep_first = (mask["size"], mask.get("keep_first", 0)) if mask else (ALL, 0)
            if m.get("kv_from") is not None:
                d.kv_from = m["kv_from"]
        elif l["type"] == "mamba2":
            d.mixer = _lib.MIXER_SSM
            d.state, d.groups, d.conv, d.norm_groups = m["state"], m["groups"], m["conv"], m["norm_groups"]
        else:
            raise ValueError("layer %d: unknown mixer %r" % (i, l["type"]))
    c = _lib.DecoderConfig(n, cfg["width"], cfg["vocab"], cfg["norm"]["eps"], 1.0, 0, 0, 0, max_batch, max_prefill, max_ctx, dtype, layers,
                           cfg["streams"], cfg["residual_mult"], cfg["logit_scale"])
    return c, layers


class Sabisun:
    """State-space and windowed-attention layers between mixed residual streams (hyper-connections), squared-ReLU feed-forward,
    tied embeddings; one .safetensors file."""
    name = "Sabisun"
    dtypes = ("bfloat16", "float32")

    @staticmethod
    def create(cfg, max_batch, max_prefill, max_ctx, dtype):
        c, keep = sabisun_config(cfg, max_batch, max_prefill, max_ctx, DTYPES[dtype])
        return create_decoder(cfg, c)

    @staticmethod
    def load_weights(model, folder, cfg):
        load_safetensors(model, folder)


# --------------------------------------------------------------------------------------------- W8A8 Llama
class SpinQuantLlama:
    """The reference's W8A8 Llama: the parameter files of its demo beside a config.json with layers, hidden, heads_q,
    heads_kv, ffn, vocab."""
    name = "SpinQuantLlama"
    dtypes = ("int8",)

    @staticmethod
    def create(cfg, max_batch, max_prefill, max_ctx, dtype):
        f32 = lambda v: C.c_float(v).value
        c = _lib.ModelConfig(cfg["layers"], cfg["hidden"], cfg["heads_q"], cfg["heads_kv"], cfg["ffn"], cfg["vocab"], cfg.get("eps", 1e-5),
                             f32(math.sqrt(cfg["ffn"])), max_batch, max_prefill, max_ctx)
        h = C.c_void_p()
        call("flexllm_model_create", C.byref(h), C.byref(c))
        m = HostModel(h, cfg["vocab"])
        m.table_len = max_ctx + 1
        return m

    @staticmethod
    def load_weights(model, folder, cfg):
        D, F, HQ = cfg["hidden"], cfg["ffn"], cfg["heads_q"]
        KV, V, L = cfg["heads_kv"] * 64, cfg["vocab"], cfg["layers"]
        dims = dict(q=(D, D), k=(KV, D), v=(KV, D), o=(D, D), g=(F, D), u=(F, D), d=(D, F))
        buf = {"w" + k: (C.c_int8 * (n * m))() for k, (n, m) in dims.items()}
        buf.update({"s" + k: (C.c_float * n)() for k, (n, _) in dims.items()})
        buf.update(gamma0=(C.c_float * D)(), gamma1=(C.c_float * D)(), a_s=(C.c_float * HQ)())
        addr = lambda n: C.cast(buf[n], C.c_void_p) if n in buf else None
        files = _lib.CkptLayerBuffers(*[addr(n) for n, _ in _lib.CkptLayerBuffers._fields_])
        w = _lib.LayerWeights(*[addr(n) for n, _ in _lib.LayerWeights._fields_])
        for l in range(L):
            call("flexllm_ckpt_load_layer", folder.encode(), l, D, KV, F, HQ, C.byref(files))
            call("flexllm_model_load_layer", model._h, l, C.byref(w), None)
            check("flexllm_device_status", lib().flexllm_device_status())      # synchronises: the buffers are reused
        T = model.table_len
        lm_w, lm_s, gf = (C.c_int8 * (V * D))(), (C.c_float * V)(), (C.c_float * D)()
        cos_t, sin_t = (C.c_float * (T * 32))(), (C.c_float * (T * 32))()
        call("flexllm_ckpt_load_head", folder.encode(), L, D, V, T, lm_w, lm_s, None, gf, cos_t, sin_t, None)
        call("flexllm_model_load_head", model._h, lm_w, lm_s, gf, cos_t, sin_t, T, None)
        check("flexllm_device_status", lib().flexllm_device_status())


REGISTRY = {e.name: e for e in (SpinQuantLlama, Pibidra, Sabisun)}


def entry(cfg):
    name = cfg.get("architecture")
    if name not in REGISTRY:
        raise ValueError("unknown architecture %r (known: %s)" % (name, ", ".join(sorted(REGISTRY))))
    return REGISTRY[name]


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def create(cfg, max_batch=1, max_prefill=2048, max_ctx=4096, dtype=None):
    """A model of the configuration without weights."""
    e = entry(cfg)
    dtype = dtype or e.dtypes[0]
    if dtype not in e.dtypes:
        raise UnsupportedDtype("%s computes in %s, not in %s" % (e.name, " or ".join(e.dtypes), dtype))
    return e.create(cfg, max_batch, min(max_prefill, max_ctx), max_ctx, dtype)


def load(folder, max_batch=1, max_prefill=2048, max_ctx=4096, dtype=None):
    """The model of a folder, ready to run."""
    cfg = read_config(folder)
    m = create(cfg, max_batch, max_prefill, max_ctx, dtype)
    try:
        entry(cfg).load_weights(m, folder, cfg)
    except Exception:
        m.close()
        raise
    return m
