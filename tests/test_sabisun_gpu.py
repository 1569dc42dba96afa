"""Sabisun on the GPU against the plain float64 restatement (oracle/sabisun.py): every mechanism alone, then the model through the
runner's own entry points (whole prompts, portions, decoding, reuse, batches, generation, command line)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import sabisun as P
from pibidra_cases import bf16_round, rel_err, tokens, write_folder
from sabisun_cases import CONFIGS, config, attn, ssm, weights
from test_pibidra_gpu import cuts_of, make, padded, run_cuts, up

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 5e-5              # bound of the root mean square error over the logits' spread in 32 bits
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def F():
    import flexllm_b200
    flexllm_b200.lib()
    return flexllm_b200


def round16(v):
    return bf16_round(np.asarray(v, np.float32)).astype(np.float64)


class Reference:
    """Exact logits of a model, and how much rounding alone moves each position's."""

    def __init__(self, cfg, t, tok):
        self.want = P.forward(cfg, t, tok)
        self.rounding = rel_err(P.forward(cfg, t, tok, act=round16), self.want)

    def check(self, dtype, got, what="", rows=slice(None)):
        d = got - self.want[rows]
        e = np.sqrt(((d - d.mean(-1, keepdims=True)) ** 2).mean(-1)) / self.want.std()
        r = self.rounding[rows]
        limit = TOL if dtype == "float32" else np.maximum(0.04, 4 * r)
        assert (e < limit).all(), (dtype, what, int(e.argmax()), e.max(), r[e.argmax()])
        if dtype == "bfloat16" and len(e) > 20:
            assert np.median(e) < 1.5 * np.median(r), (what, np.median(e), np.median(r))


def cuda(a):
    return torch.from_numpy(np.ascontiguousarray(a, np.float32)).cuda()


# ------------------------------------------------------------------------------------------------ squared ReLU
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("N,K", [(24, 40), (301, 90), (1024, 512), (20000, 64)])
def test_squared_relu_linear(F, dtype, N, K):
    g = np.random.default_rng(N)
    w = bf16_round(g.standard_normal((N, K)) * K ** -0.5)
    wd = padded(w, up(K, 8), torch.bfloat16)
    for M in (1, 2, 3, 5, 16, 33, 64, 65, 200):
        a = bf16_round(g.standard_normal((M, K)))
        want = np.maximum(P.linear(w.astype(np.float64), a.astype(np.float64)), 0) ** 2
        got = F.linear_float(padded(a, up(K, 8), dtype), wd, None, K=K, relu2=True, out_f32=True).cpu().numpy()
        assert np.abs(got - want).max() < 3e-5 * want.max(), M


# ------------------------------------------------------------------------------------------------ residual streams
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8])
def test_streams(F, streams):
    g = np.random.default_rng(streams)
    for D in (4, 90, 520, 1500, 2050, 5000):
        M, ld, eps, n = 3, up(D, 8), 1e-3, streams
        x, y = g.standard_normal((n, M, D)) * 0.05, g.standard_normal((M, D))
        mix, out, read, gain = g.standard_normal((n, n)), g.standard_normal(n), g.standard_normal(n), 1 + 0.3 * g.standard_normal(D)
        xd = torch.zeros((M, n, ld), dtype=torch.float32)
        xd[:, :, :D] = torch.from_numpy(x.transpose(1, 0, 2).astype(np.float32))
        xd = xd.cuda()
        h = F.ops.hyper_norm(xd, D, eps, padded(y, ld), cuda(mix), cuda(out * 0.3), cuda(read), padded(gain[None], ld)[0])
        want = P.hyper_write(x, mix, out, 0.3, y)
        assert np.abs(xd.cpu().numpy()[:, :, :D].transpose(1, 0, 2) - want).max() < 3e-6 * np.abs(want).max()
        want_h = P.rms_norm(P.hyper_read(want, read), eps, gain)
        assert np.abs(h.cpu().numpy()[:, :D] - want_h).max() < 2e-5 * np.abs(want_h).max()
        before = xd.clone()
        h = F.ops.hyper_norm(xd, D, eps, read=cuda(read), gain=padded(gain[None], ld)[0], dtype=torch.bfloat16)
        assert torch.equal(before, xd) and np.abs(h.float().cpu().numpy()[:, :D] - want_h).max() < 5e-3 * np.abs(want_h).max()


# ------------------------------------------------------------------------------------------------ state-space mixer
class SsmCase:
    """The mixer between its projections on B sequences in a set of slots."""

    def __init__(self, F, H, Pd, N, G, taps, parts, S, B=1, dtype=torch.float32, seed=0, A_log=(-4.0, 1.0), dt_bias=(-3.5, 0.5)):
        g = np.random.default_rng(seed)
        self.F, self.B, self.S, self.dtype, self.dims, self.eps = F, B, S, dtype, (H, Pd, N, G, taps, parts), 1e-5
        self.z, self.x = (bf16_round(g.standard_normal((B, S, H, Pd))) for _ in range(2))
        self.Bm, self.C = (bf16_round(g.standard_normal((B, S, G, N))) for _ in range(2))
        self.dt = bf16_round(g.standard_normal((B, S, H)))
        ch = H * Pd + 2 * G * N
        self.cw, self.cb = bf16_round(g.standard_normal((ch, taps)) * 0.7), bf16_round(g.standard_normal(ch) * 0.2)
        self.dtb, self.A_log, self.D = g.uniform(*dt_bias, H), g.uniform(*A_log, H), 1 + 0.3 * g.standard_normal(H)
        self.gain = 1 + 0.2 * g.standard_normal(H * Pd)
        P8, N8 = up(Pd, 8), up(N, 8)
        pad = lambda a, n: np.pad(a, [(0, 0)] * (a.ndim - 1) + [(0, n - a.shape[-1])])
        chan = lambda a: np.concatenate([pad(a[..., :H * Pd].reshape(*a.shape[:-1], H, Pd), P8).reshape(*a.shape[:-1], -1),
                                         pad(a[..., H * Pd:].reshape(*a.shape[:-1], 2 * G, N), N8).reshape(*a.shape[:-1], -1)], -1)
        self.op = F.ops.StateSpaceMixer(H, Pd, N, G, taps, parts, cuda(chan(self.cw.T)), cuda(chan(self.cb)), cuda(self.dtb), cuda(-np.exp(self.A_log)),
                                        cuda(self.D), cuda(pad(self.gain.reshape(H, Pd), P8).reshape(-1)), B + 1, self.eps, dtype)
        self.op.state.fill_(7.0)                       # what other sequences left behind
        self.op.history.fill_(5.0)
        if self.op.state.shape[1] != H * Pd * N:       # the padding of state rows stays zero
            self.op.state.reshape(B + 1, H, Pd, -1)[..., N:] = 0
        self.pad = pad

    def rows(self):
        H, Pd, N, G, _, _ = self.dims
        P8, N8 = up(Pd, 8), up(N, 8)
        flat = lambda a, n: self.pad(a, n).reshape(self.B, self.S, -1)
        r = np.concatenate([flat(self.z, P8), flat(self.x, P8), flat(self.Bm, N8), flat(self.C, N8), self.pad(self.dt, up(H, 8))], -1)
        assert r.shape[2] == self.op.row
        return r

    def want(self, act=P.exact):
        H, Pd, N, G, taps, parts = self.dims
        mx = dict(heads=H, vdim=Pd, state=N, groups=G, norm_groups=parts)
        flat = lambda a, b: a[b].reshape(self.S, -1).astype(np.float64)
        return np.stack([P.mamba2_inner(np.concatenate([flat(a, b) for a in (self.z, self.x, self.Bm, self.C, self.dt)], 1), self.cw.astype(np.float64),
                                        self.cb, self.dtb, self.A_log, self.D, self.gain, mx, self.eps, act) for b in range(self.B)])

    def check(self, got, what):
        """fp32: close to the exact result; bf16: as close as rounding alone allows (rows in which terms cancel stand out)."""
        want = self.want()
        if self.dtype == torch.float32:
            assert rms_rel(got, want).max() < 1e-5, what
        else:
            e, r = rms_rel(got, want), rms_rel(self.want(round16), want)
            assert (e < np.maximum(1.5e-2, 4 * r)).all() and np.median(e) < 1.5 * np.median(r), (what, e.max(), r.max(), np.median(e), np.median(r))

    def run(self, cuts):
        H, Pd = self.dims[:2]
        rows, out, at = self.rows(), [], 0
        for n in cuts:
            proj = torch.from_numpy(np.ascontiguousarray(rows[:, at:at + n])).to(self.dtype).cuda().reshape(self.B * n, -1).contiguous()
            o = self.op(proj, torch.full((self.B,), at, dtype=torch.int32, device="cuda")).float().cpu().numpy().reshape(self.B, n, H, -1)
            assert (o[..., Pd:] == 0).all()
            out.append(o[..., :Pd].reshape(self.B, n, -1))
            at += n
        assert at == self.S and self.F.lib().flexllm_device_status() == 0
        return np.concatenate(out, 1)


SSM_SHAPES = [  # heads, value size, state, groups, taps, parts of the norm
    (4, 32, 32, 2, 4, 2), (6, 20, 12, 3, 2, 8), (3, 40, 72, 1, 5, 1), (2, 72, 136, 1, 1, 3), (2, 64, 128, 2, 3, 4), (2, 100, 256, 1, 4, 2),
    (8, 8, 16, 8, 9, 16), (1, 136, 64, 1, 4, 1), (5, 48, 40, 5, 4, 5)]


def rms_rel(got, want):
    """Per row."""
    return np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", SSM_SHAPES)
def test_state_space_shapes_and_portions(F, shape, dtype):
    S = 210
    for kind in ("whole", "portions", "tokens"):
        c = SsmCase(F, *shape, S, dtype=DT[dtype])
        c.check(c.run(cuts_of(S, kind)), kind)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_state_space_memory(F, dtype):
    """A large input long ago decides the output (slow decay): the state survives chunks, portions and single tokens in 32 bits."""
    S = 420
    for kind in ("whole", "portions", "tokens"):
        c = SsmCase(F, 2, 32, 32, 1, 3, 1, S, dtype=DT[dtype], A_log=(-6.0, -5.5), dt_bias=(-3.0, -2.5), seed=4)
        c.x[0, 5] = 12.0
        c.x[0, 20:] *= 0.05
        c.D[:] = 0.0
        c.op.w[4].zero_()
        want = c.want()
        near = SsmCase(F, 2, 32, 32, 1, 3, 1, S, dtype=DT[dtype], A_log=(-6.0, -5.5), dt_bias=(-3.0, -2.5), seed=4)
        near.x[0, 20:] *= 0.05
        near.D[:] = 0.0
        assert np.median(rms_rel(near.want()[:, 300:], want[:, 300:])) > 0.3
        c.check(c.run(cuts_of(S, kind)), kind)


def test_state_space_extremes(F):
    """Decays that vanish within a token and steps that softplus leaves as they are or drives to zero."""
    for dtype in ("float32", "bfloat16"):
        for opts in (dict(A_log=(3.0, 4.0), dt_bias=(2.0, 5.0)), dict(A_log=(-9.0, -8.0), dt_bias=(-12.0, -9.0)), dict(dt_bias=(25.0, 40.0), A_log=(-8.0, -7.0))):
            for kind in ("whole", "portions"):
                c = SsmCase(F, 4, 16, 24, 2, 4, 2, 150, dtype=DT[dtype], **opts)
                c.check(c.run(cuts_of(150, kind)), (dtype, opts, kind))


def test_state_space_batches_and_slots(F):
    for dtype in ("float32", "bfloat16"):
        c = SsmCase(F, 4, 24, 40, 2, 4, 3, 100, B=3, dtype=DT[dtype], seed=2)
        other = c.op.state[3].clone()
        for cuts in ([100], cuts_of(100, "portions"), [60] + [1] * 40):            # the same slots again, old content in them
            c.check(c.run(cuts), (dtype, cuts[:3]))
        assert torch.equal(c.op.state[3], other)                                  # a slot of nobody in the batch


# ------------------------------------------------------------------------------------------------ attention
class KeptCase:
    """One layer's attention with kept first positions and per-head sinks on its own cache with a shuffled page table."""

    def __init__(self, F, H, G, dk, dv, window, keep, S, B=1, dtype=torch.float32, seed=0, scale=None, sinks=True, shared=False):
        g = np.random.default_rng(seed)
        self.F, self.S, self.B, self.dtype, self.shared = F, S, B, dtype, shared
        self.H, self.G, self.dk, self.dv = H, G, dk, dv
        self.scale = scale if scale is not None else dk ** -0.5
        self.mask = {"size": window, "keep_first": keep}
        self.q, self.q2, self.k = (bf16_round(g.standard_normal((B, S, n * dk)) * 1.3) for n in (H, H, G))
        self.v = bf16_round(g.standard_normal((B, S, G * dv)))
        self.sinks = bf16_round(g.uniform(0.0, 4.0, H)) if sinks else None
        max_pages = (S + 63) // 64 + 1
        self.n_pages = B * max_pages + 3
        self.pt = torch.from_numpy(g.permutation(self.n_pages)[:B * max_pages].reshape(B, max_pages).astype(np.int32)).cuda()
        sd = cuda(self.sinks) if sinks else None
        op = lambda **k: F.ops.WindowAttention(H, G, dk, dv, window, self.scale, 0.0, None, 0, None, None, self.pt, self.n_pages, S - 1, sink=False,
                                               gate=False, dtype=dtype, keep_first=keep, sinks=sd, **k)
        self.op = op()
        self.op2 = op(kv_of=self.op) if shared else None

    def point_at(self, i, j, head=0, b=0, level=14.0):
        """Position i's query of one head and position j's key stand out for each other (score `level`); j's value is large."""
        g, dk = head // (self.H // self.G), self.dk
        u = np.sign(np.random.default_rng(i).standard_normal(dk))
        u = bf16_round(u * np.sqrt(level / (dk * abs(self.scale))))
        for q in (self.q, self.q2):
            q[b, i, head * dk:(head + 1) * dk] = u * np.sign(self.scale)
        self.k[b, j, g * dk:(g + 1) * dk] = u
        self.v[b, j, g * self.dv:(g + 1) * self.dv] = 8 + np.arange(self.dv) % 4

    def want(self, q=None):
        q = self.q if q is None else q
        f = lambda a, b, n, d: a[b].astype(np.float64).reshape(self.S, n, d)
        return np.stack([P.head_outputs(f(q, b, self.H, self.dk), f(self.k, b, self.G, self.dk), f(self.v, b, self.G, self.dv), self.mask, self.scale,
                                        self.sinks).reshape(self.S, -1) for b in range(self.B)])

    def run(self, cuts, close=True):
        pad = lambda a: np.pad(a, ((0, 0), (0, 0), (0, up(a.shape[2], 8) - a.shape[2])))
        rows, rows2 = np.concatenate([pad(a) for a in (self.q, self.k, self.v)], 2), pad(self.q2)
        assert rows.shape[2] == self.op.row
        out, out2, at = [], [], 0
        for n in cuts:
            ctx = torch.full((self.B,), at, dtype=torch.int32, device="cuda")
            dev = lambda r: torch.from_numpy(np.ascontiguousarray(r[:, at:at + n])).to(self.dtype).cuda().reshape(self.B * n, -1).contiguous()
            out.append(self.op(dev(rows), ctx).float().cpu().numpy().reshape(self.B, n, -1))
            if self.shared:
                out2.append(self.op2(dev(rows2), ctx).float().cpu().numpy().reshape(self.B, n, -1))
            at += n
        assert at == self.S and self.F.lib().flexllm_device_status() == 0
        if close:
            self.op.close()
        return (np.concatenate(out, 1), np.concatenate(out2, 1)) if self.shared else np.concatenate(out, 1)


KEPT_SHAPES = [  # H, G, dk, dv, window, keep
    (4, 2, 64, 64, 50, 4), (8, 1, 40, 24, 65, 64), (6, 2, 72, 136, 30, 65), (2, 2, 128, 128, 64, 1), (16, 1, 32, 48, 63, 10), (3, 3, 20, 12, 1, 7),
    (5, 1, 16, 256, 100, 130), (4, 4, 256, 64, 40, 0), (2, 1, 264, 40, 90, 5), (32, 1, 24, 16, 70, 6), (2, 1, 64, 264, 31, 66), (4, 2, 32, 32, 500, 3)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", KEPT_SHAPES)
def test_kept_window_shapes_and_portions(F, shape, dtype):
    S, w, kp = 300, shape[4], shape[5]
    for kind in ("whole", "portions") + (("tokens",) if shape[0] <= 6 else ()):
        c = KeptCase(F, *shape, S, dtype=dtype)
        pairs = [(w - 1, 0), (w, 0), (w + kp, kp), (w + kp, max(0, kp - 1)), (128, 127), (128, 64), (290, kp), (291, max(0, kp - 1)), (292, 0), (250, 251 - w),
                 (251, 251 - w), (299, 299), (200, 64), (201, 63)]
        for n, (i, j) in enumerate(pairs):
            if 0 <= j <= i < S:
                c.point_at(i, j, head=n % shape[0])
        want = c.want()
        err = np.abs(c.run(cuts_of(S, kind)) - want).max() / np.abs(want).max()
        assert err < (1e-5 if dtype == torch.float32 else 2e-2), (kind, err)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_window_and_kept_edges_are_exact(F, dtype):
    """Last key in the window, first one outside it, last kept position, first one that is not kept."""
    w, kp, S = 77, 67, 260
    for kind in ("whole", "tokens", "portions"):
        outs = {}
        for i, j in ((250, 174), (250, 173), (251, 66), (251, 67), (252, 0)):
            c, base = (KeptCase(F, 2, 1, 32, 16, w, kp, S, dtype=dtype, seed=3) for _ in range(2))
            c.point_at(i, j)
            base.q[0, i] = c.q[0, i]
            outs[i, j] = c.run(cuts_of(S, kind))[0, i] - base.run(cuts_of(S, kind))[0, i]
        for pair, seen in (((250, 174), True), ((250, 173), False), ((251, 66), True), ((251, 67), False), ((252, 0), True)):
            assert np.abs(outs[pair]).max() > 1.0 if seen else np.array_equal(outs[pair], np.zeros_like(outs[pair])), (kind, pair)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_learned_sinks(F, dtype):
    """Sinks far above and far below the scores, different per head; without sinks the weights add up to one."""
    for kind in ("whole", "tokens", "portions"):
        for sinks in ([30.0, -30.0, 2.0, 5.0], [-200.0, 200.0, 0.0, 80.0], None):
            c = KeptCase(F, 4, 2, 32, 24, 40, 3, 130, dtype=dtype, sinks=sinks is not None, seed=6)
            if sinks:
                c.sinks = np.float32(sinks)
                c.op.sinks.copy_(cuda(sinks))
            want = c.want()
            err = np.abs(c.run(cuts_of(130, kind)) - want).max() / np.abs(want).max()
            assert err < (1e-5 if dtype == torch.float32 else 2e-2), (kind, sinks, err)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_rising_and_extreme_scores(F, dtype):
    """The running maximum grows by a lot from page to page, or lies far from zero on either side; a negative scale."""
    for kind in ("whole", "portions", "tokens"):
        for case in ("rising", "falling", "low", "negative"):
            c = KeptCase(F, 4, 2, 32, 48, 400, 2, 280, dtype=dtype, seed=7, scale=-0.2 if case == "negative" else 0.5, sinks=case != "low")
            if case in ("rising", "falling"):
                c.q[:, :, 0::32] = 4.0
                ramp = np.arange(280) * (0.25 if case == "rising" else -0.25)
                c.k[:, :, 0::32] = bf16_round(ramp)[None, :, None]
            if case == "low":
                c.q[:, :, 0::32], c.k[:, :, 0::32] = 16.0, -16.0
            want = c.want()
            err = np.abs(c.run(cuts_of(280, kind)) - want).max() / np.abs(want).max()
            assert err < (2e-5 if dtype == torch.float32 else 2e-2), (kind, case, err)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_shared_keys_and_values(F, dtype):
    for kind in ("whole", "portions", "tokens"):
        c = KeptCase(F, 4, 2, 40, 32, 50, 9, 200, dtype=dtype, seed=8, shared=True)
        c.point_at(150, 8)
        for got, q in zip(c.run(cuts_of(200, kind)), (c.q, c.q2)):
            want = c.want(q)
            assert np.abs(got - want).max() < (1e-5 if dtype == torch.float32 else 2e-2) * np.abs(want).max(), kind


def test_kept_window_splits_and_batches(F):
    """Long windows, whose keys the decode form splits over CTAs; sequences side by side; pages used again."""
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        S = 1500
        c = KeptCase(F, 2, 1, 32, 16, 1300, 70, S, dtype=dtype, seed=11)
        for i, j in [(1490, 191), (1495, 195), (1496, 69), (1497, 70), (1498, 0), (1499, 1000)]:
            c.point_at(i, j)
        want = c.want()
        err = np.abs(c.run([1480] + [1] * 20)[:, 1400:] - want[:, 1400:]).max() / np.abs(want).max()
        assert err < tol, err
        c = KeptCase(F, 4, 2, 32, 40, 70, 5, 140, B=3, dtype=dtype, seed=9)
        want = c.want()
        for cuts in ([140], cuts_of(140, "portions"), [100] + [1] * 40):
            assert np.abs(c.run(cuts, close=False) - want).max() < tol * np.abs(want).max()
        c.op.close()


# ------------------------------------------------------------------------------------------------ the model
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
        assert e < (1e-5 if dtype == "float32" else 3e-2), (i, e)
    Reference(cfg, t, tok).check(dtype, lg.cpu().numpy())
    assert int(nx[0]) == int(lg[-1].argmax())
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_decoding_and_reuse(F, name, dtype):
    """The same logits however the tokens are cut, with chunks, rings that wrap, kept pages, and slots used again."""
    cfg = CONFIGS[name]
    t = weights(cfg, seed=3)
    tok = tokens(330, cfg["vocab"], seed=4)
    ref = Reference(cfg, t, tok)
    m = make(F, cfg, t, dtype, max_prefill=64, max_ctx=1200)
    for cuts in ([330], [200] + [1] * 130, cuts_of(330, "portions"), [2] * 165, [1] * 330, [330]):
        ref.check(dtype, run_cuts(m, tok, cuts), cuts[:4])
        m.reset()
        m.step([tokens(97, cfg["vocab"], seed=len(cuts))])           # another request leaves its keys and states behind
    m.close()


def test_long_decoding(F):
    cfg = CONFIGS["plain"]
    t = weights(cfg, seed=5)
    tok = tokens(900, cfg["vocab"], seed=6)
    ref = Reference(cfg, t, tok)
    for dtype in ("float32", "bfloat16"):
        m = make(F, cfg, t, dtype, max_prefill=32, max_ctx=1000)
        ref.check(dtype, run_cuts(m, tok, [300] + [1] * 600))
        m.close()


def test_many_state_heads_and_no_window(F):
    """A layer without a mask sees everything; a wider model, whose products take other kernels."""
    full = attn(4, 4, 32, 32, 1, 0, 256)
    full["mixer"]["mask"] = None
    cfg = config([ssm(16, 32, 64, 4, 4, 8, 256), full, ssm(16, 32, 64, 4, 4, 1, 256)], 256, 1000, 2)
    t = weights(cfg, seed=15)
    tok = tokens(300, cfg["vocab"], seed=16)
    ref = Reference(cfg, t, tok)
    for dtype in ("float32", "bfloat16"):
        m = make(F, cfg, t, dtype, max_prefill=256, max_ctx=300)
        for cuts in ([300], [170] + [1] * 30 + [100]):
            ref.check(dtype, run_cuts(m, tok, cuts), cuts[:2])
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
    cfg = CONFIGS["odd"]
    t = weights(cfg, seed=7)
    prompts = [tokens(40, cfg["vocab"], seed=s) for s in (1, 2, 3, 4, 5)]
    refs = [greedy_gap(cfg, t, p, 10) for p in prompts]
    m = make(F, cfg, t, "float32", max_batch=5, max_prefill=16, max_ctx=60)
    for graph in (False, True, True):
        outs = m.generate(prompts, 10, use_graph=graph)
        for o, (want, gap) in zip(outs, refs):
            assert o == want or gap < 1e-3
    for p, (want, gap) in zip(prompts, refs):
        assert m.generate([p], 10)[0] == want or gap < 1e-3
    m.close()
    # bf16: the generated ids follow the model's own step logits
    m = make(F, cfg, t, "bfloat16", max_batch=5, max_prefill=64, max_ctx=60)
    out = m.generate(prompts, 10)
    m.reset()
    lg, _ = m.step([p + o for p, o in zip(prompts, out)], [b * 50 + 39 + i for b in range(5) for i in range(10)])
    lg = np.frombuffer(lg, np.float32).reshape(5, 10, -1)
    for b in range(5):
        for i in range(10):
            assert lg[b, i, out[b][i]] > lg[b, i].max() - 0.1 * lg.std()
    m.close()


def test_generation_after_a_longer_request(F):
    """The slots and pages of a finished generation serve the next one."""
    cfg = CONFIGS["plain"]
    t = weights(cfg, seed=17)
    m = make(F, cfg, t, "float32", max_batch=2, max_prefill=32, max_ctx=400)
    m.generate([tokens(300, cfg["vocab"], seed=1), tokens(300, cfg["vocab"], seed=2)], 20)
    for n in (7, 90):
        p = tokens(n, cfg["vocab"], seed=n)
        want, gap = greedy_gap(cfg, t, p, 8)
        assert m.generate([p], 8)[0] == want or gap < 1e-3
    m.close()


@pytest.mark.parametrize("B", [1, 3, 8, 40, 64])
def test_batch_steps(F, B):
    """Side-by-side sequences (different kernels per row count) against each alone."""
    cfg = CONFIGS["plain"]
    t = weights(cfg, seed=8)
    toks = [tokens(50, cfg["vocab"], seed=100 + b) for b in range(B)]
    for dtype in ("float32", "bfloat16"):
        m = make(F, cfg, t, dtype, max_batch=B, max_prefill=32, max_ctx=64)
        got, at = [], 0
        for n in (20, 1, 2, 1, 1, 5, 20):
            lg, _ = m.step([x[at:at + n] for x in toks], range(B * n))
            got.append(np.frombuffer(lg, np.float32).reshape(B, n, -1))
            at += n
        got = np.concatenate(got, 1)
        for b in {0, B // 2, B - 1}:
            Reference(cfg, t, toks[b]).check(dtype, got[b], b)
        m.close()


def test_extend_after_generation(F):
    """Decoding leaves cache and states as a step would: a later step of the same sequence goes on from them."""
    cfg = CONFIGS["states"]
    t = weights(cfg, seed=9)
    p = tokens(50, cfg["vocab"], seed=1)
    m = make(F, cfg, t, "float32", max_prefill=64, max_ctx=200)
    out = m.generate([p], 8)[0]
    seq = p + out + tokens(20, cfg["vocab"], seed=2)                    # the last generated token has not been fed yet
    lg, _ = m.step([seq[57:]], range(len(seq) - 57))
    Reference(cfg, t, seq).check("float32", np.frombuffer(lg, np.float32).reshape(-1, m.vocab), rows=slice(57, None))
    m.close()


def test_sampling(F):
    cfg = CONFIGS["plain"]
    t = weights(cfg, seed=10)
    prompts = [tokens(33, cfg["vocab"], seed=s) for s in (1, 2)]
    m = make(F, cfg, t, "float32", max_batch=2, max_prefill=64, max_ctx=64)
    rnd = np.random.default_rng(0).random((10, 2)).astype(np.float32)
    m.set_sampling_host(8, 4, rnd.reshape(-1).tolist(), 10, 2)
    out = m.generate(prompts, 10)
    assert out == m.generate(prompts, 10, use_graph=False)
    m.set_sampling_host()
    for b in range(2):
        lg = P.forward(cfg, t, prompts[b] + out[b])[32:42]
        for i in range(10):
            assert out[b][i] in np.argsort(-lg[i])[:5]
    m.close()


# ------------------------------------------------------------------------------------------------ files, command line, replay
def test_folder_command_line_and_replay(F, tmp_path):
    cfg = CONFIGS["odd"]
    t = weights(cfg, seed=12)
    folder = str(tmp_path / "m")
    write_folder(folder, cfg, t)
    p = tokens(40, cfg["vocab"], seed=3)
    r = subprocess.run([sys.executable, "-m", "flexllm_b200", "generate", "--model", folder, "--prompt", ",".join(map(str, p)), "--n-new", "6",
                        "--dtype", "float32"], cwd=ROOT, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    want, gap = greedy_gap(cfg, t, p, 6)
    assert json.loads(r.stdout.splitlines()[-1]) == want or gap < 1e-3
    a, b = tokens(120, cfg["vocab"], seed=4), tokens(45, cfg["vocab"], seed=5)
    steps, n = [], 0
    for rid, tok, cuts in (("a", a, [80, 2, 1, 1, 36]), ("b", b, [45])):
        at = 0
        for c in cuts:
            at += c
            steps.append({"step": n, "entries": [{"id": rid, "tokens": tok[at - c:at], "want": [] if c == 2 else list(range(c))}],
                          "end": [rid] if at == len(tok) else []})
            n += 1
    for dtype in ("float32", "bfloat16"):
        out = str(tmp_path / dtype)
        os.makedirs(out)
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out, "--max-tokens", "120"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        got = {i: np.fromfile(os.path.join(out, "%d.f32" % i), np.float32).reshape(-1, cfg["vocab"]) for i in (0, 2, 3, 4, 5)}
        ra, rb = Reference(cfg, t, a), Reference(cfg, t, b)
        for i, ref, rows in ((0, ra, slice(0, 80)), (2, ra, slice(82, 83)), (3, ra, slice(83, 84)), (4, ra, slice(84, None)), (5, rb, slice(None))):
            ref.check(dtype, got[i], i, rows)
