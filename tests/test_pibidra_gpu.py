"""Pibidra on the GPU against the plain float64 restatement (oracle/pibidra.py): every mechanism alone, then the model
through the runner's own entry points (whole prompts, portions, decoding, reuse, batches, generation, command line)."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import pibidra as P
from pibidra_cases import CONFIGS, bf16_round, rel_err, tokens, weights, write_folder

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# bounds of the root mean square error over the logits' spread; rounding alone gives about a tenth to a third of them
TOL = {"float32": 3e-5, "bfloat16": 0.06}


@pytest.fixture(scope="module")
def F():
    import flexllm_b200
    flexllm_b200.lib()
    return flexllm_b200


def up(n, a):
    return (n + a - 1) // a * a


def padded(a, ld, dtype=torch.float32):
    t = torch.zeros((a.shape[0], ld), dtype=dtype)
    t[:, :a.shape[1]] = torch.from_numpy(np.asarray(a, np.float32)).to(dtype)
    return t.cuda()


# ------------------------------------------------------------------------------------------------ linear layers
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("N,K", [(24, 40), (301, 90), (512, 256), (130, 1100), (1024, 2048)])
def test_linear(F, dtype, N, K):
    g = np.random.default_rng(N)
    w = bf16_round(g.standard_normal((N, K)) * K ** -0.5)
    b = g.standard_normal(N).astype(np.float32)
    wd, bd = padded(w, up(K, 8), torch.bfloat16), torch.from_numpy(b).cuda()
    for M in (1, 2, 3, 4, 5, 16, 17, 40, 64, 65, 130, 300):
        a = bf16_round(g.standard_normal((M, K)))
        want = P.linear(w.astype(np.float64), a.astype(np.float64), b)
        ad = padded(a, up(K, 8), dtype)
        got = F.linear_float(ad, wd, bd, K=K, out_f32=True).cpu().numpy()
        assert np.abs(got - want).max() < 2e-5 * np.abs(want).max(), (M, np.abs(got - want).max())
        got = F.linear_float(ad, wd, None, K=K).float().cpu().numpy()
        tol = 2e-5 if dtype == torch.float32 else 5e-3
        assert np.abs(got - (want - b)).max() < tol * np.abs(want).max(), M


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("ff,K", [(16, 64), (80, 90), (368, 512), (4096, 1024)])
def test_gated_gelu_linear(F, dtype, ff, K):
    g = np.random.default_rng(ff)
    gate, upw = (bf16_round(g.standard_normal((ff, K)) * 2 * K ** -0.5) for _ in range(2))
    w = np.stack([gate.reshape(-1, 16, K), upw.reshape(-1, 16, K)], 1).reshape(2 * ff, K)      # blocks of 16 gate, 16 up rows
    wd = padded(w, up(K, 8), torch.bfloat16)
    for M in (1, 3, 4, 7, 33, 64, 70, 200):
        a = bf16_round(g.standard_normal((M, K)))
        want = P.gelu_tanh(P.linear(gate.astype(np.float64), a)) * P.linear(upw.astype(np.float64), a)
        ad = padded(a, up(K, 8), dtype)
        got = F.linear_float(ad, wd, None, K=K, gelu_gate=True, out_f32=True).cpu().numpy()
        assert np.abs(got - want).max() < 3e-5 * np.abs(want).max(), (M, np.abs(got - want).max())
        got = F.linear_float(ad, wd, None, K=K, gelu_gate=True).float().cpu().numpy()
        assert np.abs(got - want).max() < 5e-3 * np.abs(want).max(), M


# ------------------------------------------------------------------------------------------------ norms
@pytest.mark.parametrize("D", [4, 90, 104, 512, 1000, 2048, 4090, 5120])
def test_sandwich_norm(F, D):
    g = np.random.default_rng(D)
    M, ld, eps = 5, up(D, 8), 1e-3
    x, y = g.standard_normal((M, D)) * 0.05, g.standard_normal((M, D)) * 3
    post, pre, vec = (1 + 0.3 * g.standard_normal((1, D)) for _ in range(3))
    xd = padded(x, ld)
    want_x = x + P.rms(y, eps) * post + vec
    h = F.sandwich_norm(xd, D, eps, padded(y, ld), padded(post, ld)[0], padded(vec, ld)[0], padded(pre, ld)[0])
    assert np.abs(xd.cpu().numpy()[:, :D] - want_x).max() < 3e-6 * np.abs(want_x).max()
    want_h = P.rms(want_x, eps) * pre
    assert np.abs(h.cpu().numpy()[:, :D] - want_h).max() < 4e-6 * np.abs(want_h).max()
    assert F.sandwich_norm(xd, D, eps, padded(y, ld), padded(post, ld)[0]) is None
    h16 = F.sandwich_norm(padded(x, ld), D, eps, gain_pre=padded(pre, ld)[0], dtype=torch.bfloat16)
    want_h = P.norm_plain(x, pre, eps)
    assert np.abs(h16.float().cpu().numpy()[:, :D] - want_h).max() < 4e-3 * np.abs(want_h).max()


# ------------------------------------------------------------------------------------------------ attention
class AttnCase:
    """One layer's attention on its own cache with a shuffled page table."""

    def __init__(self, F, H, G, dk, dv, window, S, B=1, dtype=torch.float32, softcap=15.0, sink=True, gate=True, rows=12, bias_max=60, seed=0,
                 scale=None, gain=1.5, table_scale=1.0):
        g = np.random.default_rng(seed)
        self.F, self.S, self.B, self.dtype = F, S, B, dtype
        scale = scale if scale is not None else dk ** -0.5
        self.H, self.G, self.dk, self.dv = H, G, dk, dv
        self.mx = dict(mask={"size": window}, scale=scale, softcap=softcap, bias_max=bias_max)
        self.sink, self.gate, self.eps = sink, gate, 1e-5
        self.q, self.k = (bf16_round(g.standard_normal((B, S, n * dk))) for n in (H, G))
        self.v, self.gt = bf16_round(g.standard_normal((B, S, G * dv))), bf16_round(g.standard_normal((B, S, H * dv)))
        self.qn, self.kn = (bf16_round(gain + 0.2 * g.standard_normal(n * dk)) for n in (H, G))
        self.table = bf16_round(table_scale * g.standard_normal((rows, H)))
        max_pages = (S + 63) // 64 + 1
        self.n_pages = B * max_pages + 3
        self.pt = torch.from_numpy(g.permutation(self.n_pages)[:B * max_pages].reshape(B, max_pages).astype(np.int32)).cuda()
        self.op = F.ops.WindowAttention(H, G, dk, dv, window, scale, softcap, torch.from_numpy(self.table), bias_max,
                                        torch.from_numpy(self.qn).cuda(), torch.from_numpy(self.kn).cuda(), self.pt, self.n_pages, S - 1,
                                        eps=self.eps, sink=sink, gate=gate, dtype=dtype)

    def point_at(self, i, j, head=0, b=0):
        """Makes position j's key and position i's query (of one head) stand out for each other; j's value is large."""
        g, dk = head // (self.H // self.G), self.dk
        u = bf16_round(np.sign(np.random.default_rng(i).standard_normal(dk)) * 4)
        self.q[b, i, head * dk:(head + 1) * dk] = u
        self.k[b, j, g * dk:(g + 1) * dk] = u
        self.v[b, j, g * self.dv:(g + 1) * self.dv] = 8 + np.arange(self.dv) % 4

    def want(self):
        out = np.zeros((self.B, self.S, self.H * self.dv))
        for b in range(self.B):
            q = P.norm_plain(self.q[b].astype(np.float64), self.qn, self.eps).reshape(self.S, self.H, self.dk)
            k = P.norm_plain(self.k[b].astype(np.float64), self.kn, self.eps).reshape(self.S, self.G, self.dk)
            o = P.head_outputs(q, k, self.v[b].astype(np.float64).reshape(self.S, self.G, self.dv), self.table.astype(np.float64), self.mx, self.sink)
            out[b] = o.reshape(self.S, -1) * (P.sigmoid(self.gt[b].astype(np.float64)) if self.gate else 1.0)
        return out

    def run(self, cuts):
        """Portions of the given lengths, all sequences side by side."""
        parts = [self.q, self.k, self.v] + ([self.gt] if self.gate else [])
        rows = np.concatenate([np.pad(p, ((0, 0), (0, 0), (0, up(p.shape[2], 8) - p.shape[2]))) for p in parts], 2)
        assert rows.shape[2] == self.op.row
        out, at = [], 0
        for n in cuts:
            proj = torch.from_numpy(np.ascontiguousarray(rows[:, at:at + n])).to(self.dtype).cuda().reshape(self.B * n, -1).contiguous()
            ctx = torch.full((self.B,), at, dtype=torch.int32, device="cuda")
            out.append(self.op(proj, ctx).float().cpu().numpy().reshape(self.B, n, -1))
            at += n
        assert at == self.S and self.F.lib().flexllm_device_status() == 0
        self.op.close()
        return np.concatenate(out, 1)


def cuts_of(S, kind):
    if kind == "whole":
        return [S]
    if kind == "tokens":
        return [1] * S
    out, sizes, i = [], [2, 3, 61, 1, 64, 65, 7, 2, 128, 1, 1, 33], 0
    while sum(out) < S:
        out.append(min(sizes[i % len(sizes)], S - sum(out)))
        i += 1
    return out


SHAPES = [  # H, G, dk, dv, window
    (4, 2, 64, 64, 50), (8, 1, 40, 24, 65), (6, 2, 72, 136, 130), (2, 2, 128, 128, 64), (16, 1, 32, 48, 63), (3, 3, 20, 12, 1),
    (5, 1, 16, 256, 200), (4, 4, 256, 64, 128), (2, 1, 264, 40, 90), (32, 1, 24, 16, 70), (2, 1, 64, 264, 31)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", SHAPES)
def test_attention_shapes_and_portions(F, shape, dtype):
    S = 210
    for kind in ("whole", "portions") + (("tokens",) if shape[0] <= 6 else ()):
        c = AttnCase(F, *shape, S, dtype=dtype)
        # keys just inside and just outside the window, at page borders, the first tokens, and near ones
        w = shape[4]
        for n, (i, j) in enumerate([(w - 1, 0), (w, 0), (w + 1, 1), (63 + w, 64), (128, 127), (128, 64), (64 + w, 64), (200, 200 - w), (205, 206 - w), (209, 209)]):
            if 0 <= j <= i < S:
                c.point_at(i, j, head=n % shape[0])
        want = c.want()
        err = np.abs(c.run(cuts_of(S, kind)) - want).max() / np.abs(want).max()
        assert err < (1e-5 if dtype == torch.float32 else 2e-2), (kind, err)


def test_window_edge_is_exact(F):
    """The key at distance window - 1 decides the output, the one at distance window does not enter at all."""
    w = 77
    for dtype in (torch.float32, torch.bfloat16):
        for kind in ("whole", "tokens", "portions"):
            outs = {}
            for j in (100, 99):                     # position 176 sees 100, not 99
                c = AttnCase(F, 2, 1, 32, 16, w, 180, dtype=dtype, seed=3)
                c.point_at(176, j)
                base = AttnCase(F, 2, 1, 32, 16, w, 180, dtype=dtype, seed=3)
                base.q[0, 176] = c.q[0, 176]
                outs[j] = c.run(cuts_of(180, kind))[0, 176] - base.run(cuts_of(180, kind))[0, 176]
            assert np.abs(outs[100]).max() > 1.0 and np.array_equal(outs[99], np.zeros_like(outs[99])), (dtype, kind)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("opts", [dict(softcap=0.0), dict(sink=False), dict(gate=False), dict(softcap=75.0, gain=3.0), dict(softcap=400.0, gain=4.0),
                                  dict(sink=False, softcap=90.0, gain=3.0), dict(softcap=2.0, gain=4.0), dict(scale=-0.2), dict(table_scale=6.0),
                                  dict(rows=1), dict(rows=7, bias_max=3), dict(rows=32, bias_max=128), dict(rows=16, bias_max=16)])
def test_attention_options(F, dtype, opts):
    for kind in ("whole", "portions", "tokens"):
        c = AttnCase(F, 4, 2, 48, 32, 90, 150, dtype=dtype, **opts)
        c.point_at(120, 40)
        want = c.want()
        err = np.abs(c.run(cuts_of(150, kind)) - want).max() / np.abs(want).max()
        assert err < (2e-5 if dtype == torch.float32 else 4e-2), (kind, err)


def test_sink_carries_weight(F):
    """With every score far below zero the sink takes the weight and the output vanishes; without it the values are averaged."""
    for dtype in (torch.float32, torch.bfloat16):
        for kind in ("whole", "tokens"):
            for sink in (True, False):
                c = AttnCase(F, 2, 1, 32, 16, 40, 70, dtype=dtype, sink=sink, gate=False, table_scale=0.0, seed=5)
                c.q[:] = np.tile(c.q[:, :1, :32], (1, 70, 2))
                c.k[:] = -c.q[:, :, :32]                                  # score = -softcap tanh(...) everywhere
                out = c.run(cuts_of(70, kind))
                want = c.want()
                assert np.abs(out - want).max() < 2e-2 * max(np.abs(want).max(), 1e-3), (dtype, kind, sink)
                assert (np.abs(out).max() < 1e-2) == sink


@pytest.mark.parametrize("rows,bias_max,window", [(16, 100, 200), (32, 128, 300), (12, 48, 100), (7, 50, 60), (2, 40, 90), (16, 8, 50), (1, 9, 20)])
def test_distance_table(F, rows, bias_max, window):
    """Every distance gets its bucket's bias, in every head; the entries around the window are masked."""
    from flexllm_b200 import _lib
    H, G = 6, 2
    s = _lib.AttnWindowShape(H, G, 16, 16, window, 1, 1, 0.25, 10.0, 1e-5)
    t = torch.arange(rows * H, dtype=torch.float32).reshape(rows, H).contiguous()
    n = F.lib().flexllm_attn_window_bias_floats(C.byref(s))
    out = torch.empty((n,), dtype=torch.float32, device="cuda")
    assert F.lib().flexllm_attn_window_bias(C.byref(s), t.data_ptr(), rows, bias_max, out.data_ptr(), None) == 0
    got = out.cpu().numpy().reshape(G, -1, H // G)
    pad = (got.shape[1] - window) // 2
    assert np.isneginf(got[:, :pad]).all() and np.isneginf(got[:, pad + window:]).all()
    half = rows // 2
    for d in range(window):
        # exact integer comparison: bucket b >= half needs (d / half)^(rows - half) >= (bias_max / half)^(b - half)
        if d < half:
            b = d
        elif half == 0 or bias_max <= half:
            b = rows - 1
        else:
            e = rows - half
            b = half
            while b < rows - 1 and d ** e * half ** (b + 1 - half) >= bias_max ** (b + 1 - half) * half ** e:
                b += 1
        assert np.array_equal(got[:, pad + d].reshape(-1), t[b].numpy()), (d, b)


def test_batches_and_reused_pages(F):
    """Sequences side by side equal each alone, and pages that held another sequence leave nothing behind."""
    for dtype in (torch.float32, torch.bfloat16):
        tol = 1e-5 if dtype == torch.float32 else 2e-2
        c = AttnCase(F, 4, 2, 32, 40, 70, 140, B=3, dtype=dtype, seed=9)
        want = c.want()
        assert np.abs(c.run(cuts_of(140, "portions")) - want).max() < tol * np.abs(want).max()
        c = AttnCase(F, 4, 2, 32, 40, 70, 140, B=2, dtype=dtype, seed=10)
        op, close = c.op, c.op.close
        op.close = lambda: None
        want = c.want()
        c.run([140])
        for cuts in ([140], cuts_of(140, "portions"), [100] + [1] * 40):       # the same pages again, old content in them
            assert np.abs(c.run(cuts) - want).max() < tol * np.abs(want).max()
        close()


def test_many_splits(F):
    """A long window with few sequences: the decode form splits the keys over CTAs and combines them."""
    for dtype in (torch.float32, torch.bfloat16):
        S = 1500
        c = AttnCase(F, 2, 1, 32, 16, 1400, S, dtype=dtype, seed=11, bias_max=900)
        for i, j in [(1490, 91), (1495, 95), (1496, 200), (1497, 1000), (1499, 101)]:
            c.point_at(i, j)
        want = c.want()
        err = np.abs(c.run([1480] + [1] * 20)[:, 1400:] - want[:, 1400:]).max() / np.abs(want).max()
        assert err < (1e-5 if dtype == torch.float32 else 2e-2), err


# ------------------------------------------------------------------------------------------------ the model
def make(F, cfg, t, dtype, max_batch=1, max_prefill=64, max_ctx=400):
    from flexllm_b200 import models
    m = F.ops.Model.adopt(models.create(cfg, max_batch, max_prefill, max_ctx, dtype))
    for k, v in t.items():
        m.load_tensor(k, torch.from_numpy(v).to(torch.bfloat16))
    return m


def run_cuts(m, tok, cuts):
    m.reset()
    out, at = [], 0
    for n in cuts:
        lg, _ = m.step([tok[at:at + n]], range(n))
        out.append(np.frombuffer(lg, np.float32).reshape(n, m.vocab))
        at += n
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_layers_and_logits(F, name, dtype):
    cfg = CONFIGS[name]
    t = weights(cfg, seed=1)
    tok = tokens(150, cfg["vocab"], seed=2)
    want, layers = P.forward(cfg, t, tok, want_layers=True)
    m = make(F, cfg, t, dtype, max_prefill=256)
    tr = torch.zeros(layers.shape, dtype=torch.float32, device="cuda")
    m.set_trace(tr)
    lg, nx = m.extend(torch.tensor([tok], dtype=torch.int32, device="cuda"), range(150), next_token=True)
    m.set_trace(None)
    got = tr.cpu().numpy()
    for i in range(len(layers)):
        e = np.sqrt(((got[i] - layers[i]) ** 2).mean()) / layers[i].std()
        assert e < (5e-6 if dtype == "float32" else 3e-2), (i, e)
    assert rel_err(lg.cpu().numpy(), want).max() < TOL[dtype]
    assert int(nx[0]) == int(lg[-1].argmax())
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_decoding_and_reuse(F, name, dtype):
    """The same logits however the tokens are cut, with chunks, rings that wrap, and slots used again."""
    cfg = CONFIGS[name]
    t = weights(cfg, seed=3)
    tok = tokens(330, cfg["vocab"], seed=4)
    want = P.forward(cfg, t, tok)
    m = make(F, cfg, t, dtype, max_prefill=64, max_ctx=700)
    for cuts in ([330], [200] + [1] * 130, cuts_of(330, "portions"), [2] * 165, [1] * 330, [330]):
        e = rel_err(run_cuts(m, tok, cuts), want)
        assert e.max() < TOL[dtype], (cuts[:4], int(e.argmax()), e.max())
        m.reset()
        m.step([tokens(97, cfg["vocab"], seed=len(cuts))])           # another request leaves its keys behind
    m.close()


def test_long_decoding(F):
    cfg = CONFIGS["looped"]
    t = weights(cfg, seed=5)
    tok = tokens(900, cfg["vocab"], seed=6)
    want = P.forward(cfg, t, tok)
    for dtype in ("float32", "bfloat16"):
        m = make(F, cfg, t, dtype, max_prefill=32, max_ctx=1000)
        e = rel_err(run_cuts(m, tok, [300] + [1] * 600), want)
        assert e.max() < TOL[dtype], (int(e.argmax()), e.max())
        m.close()


def greedy_gap(cfg, t, prompt, n):
    """Greedy continuation of the restatement, and the smallest gap between its two best logits."""
    seq, gap = list(prompt), np.inf
    for _ in range(n):
        lg = P.forward(cfg, t, seq)[-1]
        best = np.sort(lg)[-2:]
        gap = min(gap, best[1] - best[0])
        seq.append(int(lg.argmax()))
    return seq[len(prompt):], gap


def test_greedy_generation(F):
    """The runner's generation loop (prefill, captured decode steps): batches equal each prompt alone and the restatement."""
    cfg = CONFIGS["mixed"]
    t = weights(cfg, seed=7)
    prompts = [tokens(40, cfg["vocab"], seed=s) for s in (1, 2, 3, 4, 5)]
    refs = [greedy_gap(cfg, t, p, 12) for p in prompts]
    m = make(F, cfg, t, "float32", max_batch=5, max_prefill=16, max_ctx=60)
    for graph in (False, True, True):
        outs = m.generate(prompts, 12, use_graph=graph)
        for o, (want, gap) in zip(outs, refs):
            assert o == want or gap < 1e-3
    for p, (want, gap) in zip(prompts, refs):
        assert m.generate([p], 12)[0] == want or gap < 1e-3
    m.close()
    # bf16: the generated ids follow the model's own step logits
    m = make(F, cfg, t, "bfloat16", max_batch=5, max_prefill=64, max_ctx=60)
    out = m.generate(prompts, 12)
    m.reset()
    lg, _ = m.step([p + o for p, o in zip(prompts, out)], [b * 52 + 39 + i for b in range(5) for i in range(12)])
    lg = np.frombuffer(lg, np.float32).reshape(5, 12, -1)
    for b in range(5):
        for i in range(12):
            assert lg[b, i, out[b][i]] > lg[b, i].max() - 0.1 * lg.std()
    m.close()


@pytest.mark.parametrize("B", [1, 3, 8, 40, 64])
def test_batch_steps(F, B):
    """Side-by-side sequences (different kernels per row count) against each alone."""
    cfg = CONFIGS["plain"]
    t = weights(cfg, seed=8)
    toks = [tokens(30, cfg["vocab"], seed=100 + b) for b in range(B)]
    for dtype in ("float32", "bfloat16"):
        m = make(F, cfg, t, dtype, max_batch=B, max_prefill=16, max_ctx=64)
        got, at = [], 0
        for n in (20, 1, 2, 1, 1, 5):
            lg, _ = m.step([x[at:at + n] for x in toks], range(B * n))
            got.append(np.frombuffer(lg, np.float32).reshape(B, n, -1))
            at += n
        got = np.concatenate(got, 1)
        for b in {0, B // 2, B - 1}:
            assert rel_err(got[b], P.forward(cfg, t, toks[b])).max() < TOL[dtype]
        m.close()


def test_extend_after_generation(F):
    """Decoding leaves the cache as a step would: a later step of the same sequence goes on from it."""
    cfg = CONFIGS["once"]
    t = weights(cfg, seed=9)
    p = tokens(50, cfg["vocab"], seed=1)
    m = make(F, cfg, t, "float32", max_prefill=64, max_ctx=200)
    out = m.generate([p], 8)[0]
    seq = p + out[:7] + out[7:] + tokens(20, cfg["vocab"], seed=2)      # the last generated token has not been fed yet
    lg, _ = m.step([seq[57:]], range(len(seq) - 57))
    e = rel_err(np.frombuffer(lg, np.float32).reshape(-1, m.vocab), P.forward(cfg, t, seq)[57:])
    assert e.max() < TOL["float32"], e.max()
    m.close()


def test_sampling(F):
    cfg = CONFIGS["plain"]
    t = weights(cfg, seed=10)
    prompts = [tokens(33, cfg["vocab"], seed=s) for s in (1, 2)]
    m = make(F, cfg, t, "float32", max_batch=2, max_prefill=64, max_ctx=64)
    rnd = np.random.default_rng(0).random((10, 2)).astype(np.float32)
    m.set_sampling_host(8, 4, rnd.reshape(-1).tolist(), 10, 2)
    out = m.generate(prompts, 10)
    m.set_sampling_host()
    for b in range(2):
        lg = P.forward(cfg, t, prompts[b] + out[b])[32:42]
        for i in range(10):
            top = np.argsort(-lg[i])[:4]
            p = np.exp(lg[i][top] - lg[i][top[0]])
            p /= p.sum()
            pick = int(np.searchsorted(np.cumsum(p), rnd[i, b], side="right"))
            near = np.abs(np.cumsum(p) - rnd[i, b]).min() < 1e-3 or np.diff(-np.sort(-lg[i])[:5]).max() > -1e-3
            assert out[b][i] == top[min(pick, 3)] or near
    assert m.generate(prompts, 3) == m.generate(prompts, 3, use_graph=False)
    m.close()


def test_refusals(F):
    cfg = CONFIGS["plain"]
    m = make(F, cfg, {}, "bfloat16")
    with pytest.raises(F.FlexLLMError):
        m.step([[1, 2, 3]])                                   # no weights yet
    t = weights(cfg)
    with pytest.raises(F.FlexLLMError):
        m.load_tensor("head", torch.zeros((3, 4), dtype=torch.bfloat16))
    with pytest.raises(F.FlexLLMError):
        m.load_tensor("l9.norm1", torch.zeros((4,), dtype=torch.bfloat16))
    for k, v in t.items():
        m.load_tensor(k, torch.from_numpy(v).to(torch.bfloat16))
    with pytest.raises(F.FlexLLMError):
        m.step([[cfg["vocab"]]])                              # token out of range
    with pytest.raises(F.FlexLLMError):
        m.step([[1] * 401])                                   # past max_ctx
    m.step([[1] * 400])
    with pytest.raises(F.FlexLLMError):
        m.step([[1]])
    m.close()


# ------------------------------------------------------------------------------------------------ files, command line, replay
def test_folder_command_line_and_replay(F, tmp_path):
    cfg = CONFIGS["looped"]
    t = weights(cfg, seed=12)
    folder = str(tmp_path / "m")
    write_folder(folder, cfg, t)
    p = tokens(40, cfg["vocab"], seed=3)
    r = subprocess.run([sys.executable, "-m", "flexllm_b200", "generate", "--model", folder, "--prompt", ",".join(map(str, p)), "--n-new", "6",
                        "--dtype", "float32"], cwd=ROOT, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    want, gap = greedy_gap(cfg, t, p, 6)
    assert json.loads(r.stdout.splitlines()[-1]) == want or gap < 1e-3
    a, b = tokens(70, cfg["vocab"], seed=4), tokens(45, cfg["vocab"], seed=5)
    steps, n = [], 0
    for rid, tok, cuts in (("a", a, [30, 2, 1, 1, 36]), ("b", b, [45])):
        at = 0
        for c in cuts:
            at += c
            steps.append({"step": n, "entries": [{"id": rid, "tokens": tok[at - c:at], "want": [] if c == 2 else list(range(c))}],
                          "end": [rid] if at == len(tok) else []})
            n += 1
    for dtype in ("float32", "bfloat16"):
        out = str(tmp_path / dtype)
        os.makedirs(out)
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out, "--max-tokens", "70"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        assert r.stdout.split("\n")[:-1] == ["done %d" % i for i in range(n)]
        assert not os.path.exists(os.path.join(out, "1.f32"))
        got = {i: np.fromfile(os.path.join(out, "%d.f32" % i), np.float32).reshape(-1, cfg["vocab"]) for i in (0, 2, 3, 4, 5)}
        wa, wb = P.forward(cfg, t, a), P.forward(cfg, t, b)
        for i, w in ((0, wa[:30]), (2, wa[32:33]), (3, wa[33:34]), (4, wa[34:]), (5, wb)):
            d = got[i] - w
            e = np.sqrt(((d - d.mean(1, keepdims=True)) ** 2).mean(1)) / wa.std()
            assert e.max() < TOL[dtype], (dtype, i, e.max())


def test_llama_steps_equal_its_prefill(F):
    """The step call serves the W8A8 model too: portions of 128 give the prefill's tokens and logits bit for bit."""
    from flexllm_b200 import synthetic
    layers, hidden, hq, hkv, vocab, S = 2, 512, 8, 2, 1024, 384
    W = synthetic.numpy_weights(layers, hidden, hq, hkv, 8192, vocab, S + 4, seed=3)
    m = F.Model(layers, hidden, hq, hkv, 8192, vocab, max_batch=2, max_prefill=128, max_ctx=S + 4)
    synthetic.load_numpy_weights(m, W)
    tok = torch.from_numpy(np.random.default_rng(1).integers(0, vocab, (2, S)).astype(np.int32)).cuda()
    first = m.prefill(tok)
    ref = m.buffer(1, (2, vocab), torch.float32).clone()
    m.reset()
    for at, n in ((0, 128), (128, 256)):
        lg, nx = m.extend(tok[:, at:at + n].contiguous(), [n - 1, 2 * n - 1], next_token=True)
    assert torch.equal(nx, first) and torch.equal(lg, ref)
    m.begin(4)
    m.decode(3)
    torch.cuda.synchronize()
    m.close()


def test_registry_loads_the_w8a8_model_from_its_files(F, tmp_path):
    from flexllm_b200 import models, synthetic
    layers, hidden, hq, hkv, vocab, S = 1, 256, 4, 1, 256, 32
    W = synthetic.numpy_weights(layers, hidden, hq, hkv, 8192, vocab, S + 4, seed=5)
    folder = str(tmp_path / "llama")
    synthetic.write_reference_format(folder, W)
    json.dump(dict(architecture="SpinQuantLlama", layers=layers, hidden=hidden, heads_q=hq, heads_kv=hkv, ffn=8192, vocab=vocab),
              open(os.path.join(folder, "config.json"), "w"))
    tok = np.random.default_rng(1).integers(0, vocab, (1, S)).astype(np.int32)
    m = models.load(folder, max_batch=1, max_prefill=S, max_ctx=S + 4)
    got = m.generate(tok.tolist(), 4)
    m.close()
    ref = F.Model(layers, hidden, hq, hkv, 8192, vocab, max_batch=1, max_prefill=S, max_ctx=S + 4)
    synthetic.load_numpy_weights(ref, W)
    assert got == ref.generate_host(torch.from_numpy(tok), 4).tolist()
    ref.close()
