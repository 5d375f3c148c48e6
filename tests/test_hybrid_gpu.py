"""Hybrid designs on the GPU against the plain float64 oracle: every mechanism through the C ABI, then whole models through
the scheduler, the generator and the command-line programs."""
import ctypes as C
import json
import os
import subprocess

import numpy as np
import pytest

from _hybrid import CONFIGS, O, attention, bf16_bits, bf16_round, config, delta, logits_error, make_weights, write_model
from _support import ROOT, load_package, max_abs_rel

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def pkg():
    p = load_package()
    p.build()
    p.ffi.require_device()
    return p


@pytest.fixture(scope="module")
def g(pkg):
    return pkg.ffi


def dev(g, a):
    return g.DeviceBuffer.from_numpy(np.asarray(a))


def sync(g):
    g.check(g.cuda().greta_cuda_device_synchronize(), "synchronize")
    code = C.c_int()
    g.check(g.cuda().greta_cuda_linear_gemm_status(C.byref(code)))
    assert code.value == 0


def pad_cols(a, ld):
    return np.pad(a, ((0, 0), (0, ld - a.shape[1])))


# ------------------------------------------------------------------ dense linears
def run_linear(g, W, x, fmt, segs, gemm, ln=None, resid=None):
    """segs: (rows, act, bias or None, out_fmt).  -> list of outputs [M][rows] (float32)"""
    lib = g.cuda()
    N, K = W.shape
    M = x.shape[0]
    ldw = (K + 63) // 64 * 64
    wd = dev(g, bf16_bits(pad_cols(W, ldw)) if fmt == g.FMT_BF16 else pad_cols(W, ldw).astype(np.float32))
    lin = g.Linear(fmt, wd.ptr, N, K, ldw, len(segs))
    outs, keep, row = [], [wd], 0
    for i, (rows, act, bias, out_fmt) in enumerate(segs):
        ld, col0, pair = 2 * rows + 5, 3, rows + 1
        o = g.DeviceBuffer(M * ld * 4, zero=True)
        if resid is not None:
            o.upload(np.ascontiguousarray(pad_cols(np.pad(resid, ((0, 0), (col0, 0))), ld), np.float32))
        b = None if bias is None else dev(g, bias.astype(np.float32))
        lin.seg[i] = g.OutSegment(row, rows, act, out_fmt, int(resid is not None), None if b is None else b.ptr, o.ptr, ld, col0, pair)
        outs.append((o, rows, ld, col0, pair, out_fmt))
        keep.append(b)
        row += rows
    if gemm:
        ldx = ldw
        xd = dev(g, bf16_bits(pad_cols(x, ldx)) if fmt == g.FMT_BF16 else pad_cols(x, ldx).astype(np.float32))
        g.check(lib.greta_cuda_linear_gemm(None, C.byref(lin), xd.ptr, ldx, M), "linear_gemm")
    else:
        xd = dev(g, pad_cols(x, K + 3).astype(np.float32))
        lw, lb = (dev(g, v.astype(np.float32)) for v in ln[:2]) if ln else (None, None)
        g.check(lib.greta_cuda_linear_gemv(None, C.byref(lin), xd.ptr, K + 3, lw.ptr if ln else None, lb.ptr if ln else None, ln[2] if ln else 0.0, M),
                "linear_gemv")
        keep += [lw, lb]
    sync(g)
    res = []
    for o, rows, ld, col0, pair, out_fmt in outs:
        if out_fmt == g.OUT_F32:
            res.append(o.download(np.float32, M * ld).reshape(M, ld)[:, col0:col0 + rows])
        else:
            h = (o.download(np.uint16, M * ld).astype(np.uint32) << 16).view(np.float32).reshape(M, ld)
            v = h[:, col0:col0 + rows].copy()
            if out_fmt == g.OUT_BF16_PAIR:
                v += h[:, col0 + pair:col0 + pair + rows]
            res.append(v)
    return res


ACTS = {0: lambda z: z, 1: O.gelu_erf, 2: O.sigmoid, 3: np.tanh, 4: lambda z: np.exp(-np.exp(-0.5) * O.sigmoid(z))}


@pytest.mark.parametrize("gemm", [False, True])
@pytest.mark.parametrize("fmt", ["bf16", "f32"])
def test_linear_segments_activations_and_formats(g, gemm, fmt):
    rng = np.random.default_rng(5)
    f = g.FMT_BF16 if fmt == "bf16" else g.FMT_F32
    for N_parts, K, M in (((70, 33, 1, 130, 61), 200, 5), ((5, 300, 2, 11, 9), 1000, 8), ((129, 127, 128, 64, 33), 72, 3 if not gemm else 45),
                          ((2, 3, 4, 5, 6), 37, 1 if not gemm else 300)):
        N = sum(N_parts)
        W, x = bf16_round(rng.normal(0, 1 / np.sqrt(K), (N, K))), bf16_round(rng.normal(0, 2, (M, K)))
        segs = [(n, a, rng.normal(size=n) if a != 1 else None, (g.OUT_F32, g.OUT_BF16, g.OUT_F32, g.OUT_BF16_PAIR, g.OUT_F32)[a])
                for a, n in enumerate(N_parts)]
        got = run_linear(g, W, x, f, segs, gemm)
        z, row = x.astype(np.float64) @ W.T.astype(np.float64), 0
        for (n, a, bias, out_fmt), y in zip(segs, got):
            want = ACTS[a](z[:, row:row + n] + (0 if bias is None else bias.astype(np.float32)))
            tol = 4e-3 if out_fmt == g.OUT_BF16 else 3e-5 if out_fmt == g.OUT_BF16_PAIR else 3e-6
            assert np.abs(y - want).max() <= tol * max(1.0, np.abs(want).max()), (N_parts, M, a)
            row += n


@pytest.mark.parametrize("M", [9, 33, 64, 100, 257])
def test_linear_gemm_tiles_and_residual(g, M):
    """Every token-tile width, several tiles per CTA, K that is no multiple of a stage, sums added to what is there."""
    rng = np.random.default_rng(M)
    for N, K in ((20000, 100), (4000, 264), (300, 520), (200, 2100), (700, 1100)):
        W, x = bf16_round(rng.normal(0, 1 / np.sqrt(K), (N, K))), bf16_round(rng.normal(size=(M, K)))
        resid = rng.normal(size=(M, N)).astype(np.float32)
        got = run_linear(g, W, x, g.FMT_BF16, [(N, 0, None, g.OUT_F32)], True, resid=resid)[0]
        want = resid + x.astype(np.float32) @ W.T
        assert np.abs(got - want).max() < 1e-4


@pytest.mark.parametrize("M", [1, 2, 3, 8])
@pytest.mark.parametrize("fmt", ["bf16", "f32"])
def test_linear_gemv_norm_and_long_rows(g, M, fmt):
    rng = np.random.default_rng(M)
    f = g.FMT_BF16 if fmt == "bf16" else g.FMT_F32
    for N, K in ((600, 300), (2500, 70), (9700, 136), (40, 17000)):     # every row grouping; rows longer than a chunk
        W = bf16_round(rng.normal(0, 1 / np.sqrt(K), (N, K)))
        x, lw, lb = rng.normal(3, 2, (M, K)).astype(np.float32), rng.normal(1, 0.3, K).astype(np.float32), rng.normal(size=K).astype(np.float32)
        got = run_linear(g, W, x, f, [(N, 0, None, g.OUT_F32)], False, ln=(lw, lb, 1e-3))[0]
        want = O.layer_norm(x.astype(np.float64), lw, lb, 1e-3) @ W.T.astype(np.float64)
        assert max_abs_rel(got, want) < 1e-5


def test_layer_norm_and_embedding(g):
    rng = np.random.default_rng(2)
    lib = g.cuda()
    M, D, V, P = 7, 300, 50, 20
    x, w, b = rng.normal(5, 3, (M, D)).astype(np.float32), rng.normal(1, 1, D).astype(np.float32), rng.normal(size=D).astype(np.float32)
    xd, wd, bd = dev(g, x), dev(g, w), dev(g, b)
    want = O.layer_norm(x.astype(np.float64), w, b, 1e-2)
    o = g.DeviceBuffer(M * 320 * 4, zero=True)
    g.check(lib.greta_cuda_layer_norm(None, xd.ptr, wd.ptr, bd.ptr, 1e-2, o.ptr, g.OUT_F32, M, D, 320))
    sync(g)
    got = o.download(np.float32, M * 320).reshape(M, 320)
    assert max_abs_rel(got[:, :D], want) < 2e-6 and not got[:, D:].any()
    table, pos = rng.normal(size=(V, D)).astype(np.float32), rng.normal(size=(P, D)).astype(np.float32)
    toks = np.array([0, 49, 3, 3, 50, -1, 7], np.int32)
    td, pd, kd = dev(g, table), dev(g, pos), dev(g, toks)
    dp = dev(g, np.array([5, 0, 19, 20, 1, 2, 3], np.uint32))
    for d_pos, where in ((None, np.arange(M) + 15), (dp.ptr, np.array([5, 0, 19, 20, 1, 2, 3]))):
        g.check(lib.greta_cuda_embedding_positions(None, kd.ptr, td.ptr, pd.ptr, g.FMT_F32, o.ptr, M, D, V, P, d_pos, 15))
        sync(g)
        want = np.array([(table[t] if 0 <= t < V else 0) + (pos[p] if p < P else np.zeros(D, np.float32)) for t, p in zip(toks, where)])
        assert np.array_equal(o.download(np.float32, M * D).reshape(M, D), want.astype(np.float32))


# ------------------------------------------------------------------ attention
class Attn:
    """One layer's windowed attention on the device: caches of `slots` sequences, projections given per call."""

    def __init__(self, g, H, G, dim, vdim, taps, window, keep, max_seq, chunk, scale, softcap, p, conv, cache, slots=1, eps=1e-5):
        self.g, self.lib = g, g.cuda()
        self.H, self.G, self.dim, self.vdim = H, G, dim, vdim
        self.Ccols = (H + G) * dim + G * vdim
        ring = min(max_seq - keep, window - 1 + chunk) if window else max_seq - keep
        eb = 2 if cache == "f16" else 4
        up8 = lambda d: (d + 7) // 8 * 8
        rows = slots * G * (keep + ring)
        # garbage from "earlier sequences": everything a correct kernel reads has been written before
        junk = lambda n: dev(g, np.random.default_rng(9).normal(0, 30, n).astype(np.float16 if cache == "f16" else np.float32))
        self.bufs = [junk(rows * up8(dim)), junk(rows * up8(vdim)), dev(g, np.full(slots * max(taps, 1) * self.Ccols, 7, np.float32))]
        self.bufs += [dev(g, np.asarray(v, np.float32)) for v in (p["temp"], p["r1"], p["r2"], p["sink"])]
        self.bufs.append(dev(g, np.asarray(conv, np.float32)) if taps else None)
        b = self.bufs
        self.a = g.WindowAttn(H, G, dim, vdim, taps, window, keep, ring, scale, softcap, eps, b[3].ptr, b[4].ptr, b[5].ptr, b[6].ptr,
                              b[7].ptr if taps else None, None, self.Ccols + 3, g.FMT_F16 if cache == "f16" else g.FMT_F32, b[0].ptr, b[1].ptr, b[2].ptr)

    def _proj(self, raw):
        d = dev(self.g, pad_cols(np.asarray(raw, np.float32), self.Ccols + 3))
        self.a.proj = d.ptr
        return d

    def portion(self, raw, pos0, slot=0, mma=False):
        g, M = self.g, len(raw)
        d = self._proj(raw)
        rows = g.Rows(M, slot, pos0, None)
        q = g.DeviceBuffer(M * self.H * ((self.dim + 7) // 8 * 8) * 4)
        ld = self.H * self.vdim + 5
        o = g.DeviceBuffer(M * ld * 4, zero=True)
        g.check(self.lib.greta_cuda_window_attn_prepare(None, C.byref(self.a), C.byref(rows), q.ptr), "prepare")
        if mma:
            g.check(self.lib.greta_cuda_window_attn_prefill(None, C.byref(self.a), C.byref(rows), q.ptr, o.ptr, g.OUT_F32, ld), "prefill")
        else:
            g.check(self.lib.greta_cuda_window_attn(None, C.byref(self.a), C.byref(rows), q.ptr, o.ptr, g.OUT_F32, ld, pos0 + M), "rows")
        sync(g)
        del d
        return o.download(np.float32, M * ld).reshape(M, ld)[:, :ld - 5].reshape(M, self.H, self.vdim)

    def decode(self, raw, positions, max_len):
        """Row m is the next token of slot m."""
        g, M = self.g, len(raw)
        d, dp = self._proj(raw), dev(self.g, np.asarray(positions, np.uint32))
        rows = g.Rows(M, 0, 0, dp.ptr)
        ld = self.H * self.vdim
        o = g.DeviceBuffer(M * ld * 4)
        g.check(self.lib.greta_cuda_window_attn(None, C.byref(self.a), C.byref(rows), None, o.ptr, g.OUT_F32, ld, max_len), "decode")
        sync(g)
        del d
        return o.download(np.float32, M * ld).reshape(M, self.H, self.vdim)


def attn_oracle(raw, H, G, dim, vdim, conv, window, keep, scale, softcap, p, eps=1e-5):
    T = len(raw)
    u = O.causal_conv(raw.astype(np.float64), conv.astype(np.float64)) if conv is not None else raw.astype(np.float64)
    q = O.rms_unit(u[:, :H * dim].reshape(T, H, dim), eps)
    k = O.rms_unit(u[:, H * dim:(H + G) * dim].reshape(T, G, dim), eps)
    return O.attend(q, k, u[:, (H + G) * dim:].reshape(T, G, vdim), p, window if window else T + 1, keep, scale, softcap)


def head_params(rng, H):
    return {"temp": (0.5 + rng.random(H)).astype(np.float32), "r1": (0.1 + 0.5 * rng.random(H)).astype(np.float32),
            "r2": (0.05 + rng.random(H)).astype(np.float32), "sink": rng.normal(0, 1, H).astype(np.float32)}


ATTN_CASES = [  # H, G, dim, vdim, taps, window, keep
    (4, 2, 32, 48, 3, 37, 5), (3, 3, 20, 9, 4, 1, 3), (10, 1, 64, 64, 2, 64, 0), (2, 2, 136, 256, 1, 100, 70), (8, 4, 64, 40, 0, 33, 200), (6, 2, 72, 128, 5, 0, 0)]


@pytest.mark.parametrize("case", range(len(ATTN_CASES)))
@pytest.mark.parametrize("cache", ["f32", "f16"])
def test_attention_portions_and_decoding(g, case, cache):
    """Portions down to two tokens, the tensor-core kernel, then decoding through the cache, all against the oracle."""
    H, G, dim, vdim, taps, window, keep = ATTN_CASES[case]
    rng = np.random.default_rng(case)
    T, p = 230, head_params(rng, H)
    conv = rng.normal(0, 0.8, ((H + G) * dim + G * vdim, taps)).astype(np.float32) if taps else None
    raw = rng.normal(size=(T, (H + G) * dim + G * vdim)).astype(np.float32)
    want = attn_oracle(raw, H, G, dim, vdim, conv, window, keep, 0.4, 6.0, p)
    tol = 1e-5 if cache == "f32" else 3e-3
    for cuts in ([200], [64, 2, 3, 60, 17, 54], [2] * 3 + [100, 94]):
        at = Attn(g, H, G, dim, vdim, taps, window, keep, 256, max(cuts), 0.4, 6.0, p, conv, cache)
        pos, got = 0, []
        for n in cuts:
            got.append(at.portion(raw[pos:pos + n], pos, mma=cache == "f16" and n >= 16))
            pos += n
        for t in range(pos, T):
            got.append(at.decode(raw[t:t + 1], [t], 256))
        assert max_abs_rel(np.concatenate(got), want) < tol, cuts


@pytest.mark.parametrize("form", ["rows", "mma", "decode"])
def test_attention_edges_stand_out(g, form):
    """One key is lined up with one query so that its weight is near one if and only if it is seen: just inside and just
    outside the window, the last kept and the first not kept, keys at a tile's border and on the wrap of the ring."""
    H, G, dim, vdim, window, keep, T = 2, 1, 32, 16, 50, 6, 180
    rng = np.random.default_rng(11)
    p = {"temp": np.ones(H, np.float32), "r1": np.full(H, 0.05, np.float32), "r2": np.full(H, 0.3, np.float32), "sink": np.array([-1.0, 2.0], np.float32)}
    for i, j in [(179, 130), (179, 129), (179, 5), (179, 6), (179, 0), (179, 179), (120, 71), (120, 70), (63, 64 - 50), (64, 64 - 50), (64, 15), (170, 128),
                 (170, 127), (60, 5), (60, 6), (60, 10), (60, 11)]:
        raw = 0.2 * rng.normal(size=(T, (H + G) * dim + G * vdim)).astype(np.float32)
        raw[:, H * dim:(H + G) * dim] = rng.normal(size=(T, dim))
        for h in range(H):                                  # every other query looks elsewhere
            raw[i, h * dim:(h + 1) * dim] = raw[j, H * dim:(H + G) * dim]
        raw[j, (H + G) * dim:] = 5.0
        want = attn_oracle(raw, H, G, dim, vdim, None, window, keep, 0.5, 20.0, p)
        seen = O.visible(i, j, window, keep)
        assert (want[i, 0].mean() > 4.5) == seen            # the case does what it says
        at = Attn(g, H, G, dim, vdim, 0, window, keep, 256, 90, 0.5, 20.0, p, None, "f16" if form == "mma" else "f32")
        if form == "decode":
            at.portion(raw[:60], 0)
            got = np.concatenate([want[:60]] + [at.decode(raw[t:t + 1], [t], 256) for t in range(60, i + 1)])
        else:
            got = np.concatenate([at.portion(raw[a:b], a, mma=form == "mma") for a, b in ((0, 90), (90, 180))])
        assert np.abs(got[i] - want[i]).max() < (2e-5 if form != "mma" else 1e-2), (i, j)


def test_attention_sink_and_optional_parts(g):
    """The sink alone can take the weight; softcap, temperature, bias and sink may be absent."""
    H, G, dim, vdim, T = 3, 3, 24, 24, 40
    rng = np.random.default_rng(4)
    raw = rng.normal(size=(T, 3 * H * dim)).astype(np.float32)
    none = {"temp": np.ones(H), "r1": np.zeros(H), "r2": np.zeros(H), "sink": np.full(H, -1e30)}
    strong = dict(none, sink=np.array([3.0, 30.0, -5.0], np.float32))
    for p, drop in ((strong, ("temp", "r1", "r2")), (none, ("temp", "r1", "r2", "sink"))):
        for cap in (3.0, 0.0):
            want = attn_oracle(raw, H, G, dim, vdim, None, 12, 2, 0.3, cap if cap else 1e9, p)
            for cache in ("f32", "f16"):
                at = Attn(g, H, G, dim, vdim, 0, 12, 2, 64, T, 0.3, cap, {k: np.asarray(v, np.float32) for k, v in p.items()}, None, cache)
                for n in drop:
                    setattr(at.a, n, None)
                got = at.portion(raw, 0, mma=cache == "f16")
                assert np.abs(got - want).max() < (1e-5 if cache == "f32" else 4e-3)


def test_attention_batch_of_unequal_sequences_and_reused_slots(g):
    H, G, dim, vdim, taps, window, keep = 4, 2, 40, 24, 3, 20, 4
    rng = np.random.default_rng(8)
    p, cols = head_params(rng, H), (H + G) * dim + G * vdim
    conv = rng.normal(0, 0.8, (cols, taps)).astype(np.float32)
    for cache, tol in (("f32", 1e-5), ("f16", 3e-3)):
        at = Attn(g, H, G, dim, vdim, taps, window, keep, 128, 64, 0.4, 6.0, p, conv, cache, slots=3)
        for turn in range(2):                                # the second turn meets what the first left in the slots
            lens = [(50, 3, 17), (2, 64, 9)][turn]
            raws = [rng.normal(size=(n + 30, cols)).astype(np.float32) for n in lens]
            wants = [attn_oracle(r, H, G, dim, vdim, conv, window, keep, 0.4, 6.0, p) for r in raws]
            for s, n in enumerate(lens):
                assert max_abs_rel(at.portion(raws[s][:n], 0, slot=s), wants[s][:n]) < tol
            for t in range(30):
                pos = [n + t for n in lens]
                got = at.decode(np.stack([r[i] for r, i in zip(raws, pos)]), pos, 128)
                assert max_abs_rel(got, np.stack([w[i] for w, i in zip(wants, pos)])) < tol


# ------------------------------------------------------------------ delta rule
class Delta:
    def __init__(self, g, H, d, rank, w2, w0, norm, slots=1, eps=1e-5):
        self.g, self.lib, self.H, self.d = g, g.cuda(), H, d
        n = self.lib.greta_cuda_delta_state_bytes(H, d) // 4
        self.keep = [dev(g, np.full(slots * n, 1e3, np.float32))] + [dev(g, np.asarray(v, np.float32)) for v in (w2, w0, norm)]
        self.n, self.rank, self.eps = n, rank, eps

    def desc(self, cols, t=None, decay=None):
        g, HD = self.g, self.H * self.d
        proj = dev(g, np.concatenate([cols[c].reshape(-1, HD) for c in ("r", "k", "v", "a", "gate")] + [np.zeros((len(cols["r"]), 3))], 1).astype(np.float32))
        ld = 5 * HD + 3
        at = lambda i: proj.ptr + 4 * i * HD
        td = dev(g, np.asarray(t, np.float32)) if t is not None else None
        dd = dev(g, np.asarray(decay, np.float32).reshape(-1, HD)) if decay is not None else None
        b = self.keep
        s = g.DeltaRule(self.H, self.d, self.rank, ld, self.eps, at(0), at(1), at(2), at(3), at(4), dd.ptr if dd else None, HD, td.ptr if td else None,
                        self.rank, b[1].ptr, b[2].ptr, b[3].ptr, b[0].ptr)
        return s, (proj, td, dd)

    def portion(self, cols, decay, pos0, slot=0):
        g, M, HD = self.g, len(cols["r"]), self.H * self.d
        s, hold = self.desc(cols, decay=decay)
        rows = g.Rows(M, slot, pos0, None)
        ob, o = g.DeviceBuffer(M * HD * 4), g.DeviceBuffer(M * (HD + 7) * 4)
        g.check(self.lib.greta_cuda_delta_scan(None, C.byref(s), C.byref(rows), ob.ptr), "scan")
        g.check(self.lib.greta_cuda_delta_output(None, C.byref(s), ob.ptr, M, o.ptr, g.OUT_F32, HD + 7), "output")
        sync(g)
        del hold
        return o.download(np.float32, M * (HD + 7)).reshape(M, HD + 7)[:, :HD]

    def step(self, cols, t, positions):
        g, M, HD = self.g, len(cols["r"]), self.H * self.d
        s, hold = self.desc(cols, t=t)
        dp = dev(g, np.asarray(positions, np.uint32))
        rows = g.Rows(M, 0, 0, dp.ptr)
        o = g.DeviceBuffer(M * HD * 4)
        g.check(self.lib.greta_cuda_delta_step(None, C.byref(s), C.byref(rows), o.ptr, g.OUT_F32, HD), "step")
        sync(g)
        del hold
        return o.download(np.float32, M * HD).reshape(M, HD)


def delta_inputs(rng, T, H, d, rank):
    cols = {c: rng.normal(size=(T, H, d)).astype(np.float32) for c in ("r", "k", "v")}
    cols["a"], cols["gate"] = (O.sigmoid(rng.normal(size=(2, T, H, d)))).astype(np.float32)
    return cols, np.tanh(rng.normal(size=(T, rank))).astype(np.float32)


def delta_want(cols, t, w2, w0, norm, eps=1e-5):
    T, H, d = cols["r"].shape
    f = {k: v.astype(np.float64) for k, v in cols.items()}
    dec = np.exp(-np.exp(-0.5) * O.sigmoid(t.astype(np.float64) @ w2.T + w0)).reshape(T, H, d)
    o, _ = O.delta_scan(f["r"], f["k"], f["v"], dec, f["a"])
    return O.rms_unit(o, eps).reshape(T, H * d) * norm * f["gate"].reshape(T, H * d), dec


@pytest.mark.parametrize("H,d,rank", [(3, 40, 7), (2, 64, 33), (1, 7, 1), (2, 96, 16), (1, 130, 5), (2, 256, 40), (5, 32, 3)])
def test_delta_rule_portions_and_decoding(g, H, d, rank):
    rng = np.random.default_rng(d)
    w2, w0, norm = rng.normal(0, 1, (H * d, rank)).astype(np.float32), rng.normal(-3, 2, H * d).astype(np.float32), rng.normal(1, 0.3, H * d).astype(np.float32)
    T = 90
    cols, t = delta_inputs(rng, T, H, d, rank)
    cols["k"][5] = 0                                         # the 1e-6 of the unit key
    cols["k"][6] *= 1e-4
    want, dec = delta_want(cols, t, w2, w0, norm)
    sub = lambda a, b: {k: v[a:b] for k, v in cols.items()}
    for cuts in ([70], [2, 16, 2, 17, 33], [64, 6]):
        m = Delta(g, H, d, rank, w2, w0, norm)
        pos, got = 0, []
        for n in cuts:
            got.append(m.portion(sub(pos, pos + n), dec[pos:pos + n], pos))
            pos += n
        for i in range(pos, T):
            got.append(m.step(sub(i, i + 1), t[i:i + 1], [i]))
        assert max_abs_rel(np.concatenate(got), want) < 3e-5, cuts


def test_delta_rule_batch_and_reused_slots(g):
    H, d, rank = 2, 48, 6
    rng = np.random.default_rng(3)
    w2, w0, norm = rng.normal(0, 1, (H * d, rank)).astype(np.float32), rng.normal(-2, 1, H * d).astype(np.float32), np.ones(H * d, np.float32)
    m = Delta(g, H, d, rank, w2, w0, norm, slots=3)
    for lens in ((30, 2, 11), (3, 20, 0)):                   # a slot that starts with a decoded token, slots used again
        data = [delta_inputs(rng, n + 12, H, d, rank) for n in lens]
        wants = [delta_want(c, t, w2, w0, norm) for c, t in data]
        for s, n in enumerate(lens):
            if n:
                got = m.portion({k: v[:n] for k, v in data[s][0].items()}, wants[s][1][:n], 0, slot=s)
                assert max_abs_rel(got, wants[s][0][:n]) < 3e-5
        for i in range(12):
            pos = [n + i for n in lens]
            got = m.step({k: np.stack([data[s][0][k][pos[s]] for s in range(3)]) for k in data[0][0]}, np.stack([data[s][1][pos[s]] for s in range(3)]), pos)
            assert max_abs_rel(got, np.stack([wants[s][0][pos[s]] for s in range(3)])) < 3e-5


def test_delta_rule_remembers_far_back(g):
    """Slow decay and no removal: a single write at position 0 is read back hundreds of tokens later, in one portion or many."""
    H, d, T = 1, 32, 400
    rng = np.random.default_rng(6)
    cols = {c: np.zeros((T, H, d), np.float32) for c in ("r", "k", "v", "a", "gate")}
    cols["gate"] += 1
    cols["k"][0, 0, 3] = cols["r"][:, 0, 3] = 1
    cols["v"][0] = rng.normal(size=d)
    dec = np.full((T, H, d), 0.9999, np.float32)
    want = O.rms_unit(cols["v"][0, 0].astype(np.float64) * 0.9999 ** 399, 1e-9)
    for cuts in ([400], [16] * 25, [399, 1]):
        m = Delta(g, H, d, 1, np.zeros((d, 1)), np.zeros(d), np.ones(d), eps=1e-9)
        pos = 0
        for n in cuts:
            out = m.portion({k: v[pos:pos + n] for k, v in cols.items()}, dec[pos:pos + n], pos)
            pos += n
        assert max_abs_rel(out[-1], want) < 1e-4


# ------------------------------------------------------------------ whole models
FMTS = {"f32": (0, 2e-5), "bf16": (2, 3e-2)}


@pytest.fixture(scope="module")
def models(pkg, tmp_path_factory):
    out = {}
    for name, (cfg, rank) in CONFIGS.items():
        w = make_weights(cfg, rank, 17)
        folder = write_model(str(tmp_path_factory.mktemp(name)), cfg, w, pkg)
        toks = np.random.default_rng(1).integers(0, cfg["vocab"], 150)
        out[name] = (cfg, w, folder, toks, O.forward(cfg, w, toks))
    return out


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_model_whole_portions_and_token_by_token(pkg, models, name, dtype):
    cfg, _, folder, toks, want = models[name]
    fmt, tol = FMTS[dtype]
    T = len(toks)
    m = pkg.model.Model.open(folder, fmt, max_seq=160, prefill_chunk=100)
    whole = m.forward_logits(toks, 0, np.arange(T))                      # two portions of at most 100
    assert logits_error(whole, want) < tol
    assert np.abs(m.forward(toks, 0) - whole[-1]).max() < tol * np.abs(whole[-1]).max()
    one = np.concatenate([m.forward_logits(toks[t:t + 1], t, [0]) for t in range(T)])
    assert logits_error(one, want) < tol
    for cuts in ([2] * 5 + [64, 3, 9, 30, 34], [33, 8, 7, 102], [149, 1]):
        pos, got = 0, []
        for n in cuts:
            got.append(m.forward_logits(toks[pos:pos + n], pos, np.arange(n)))
            pos += n
        assert logits_error(np.concatenate(got), want) < tol, cuts
    m.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_model_layers_one_by_one(pkg, models, dtype, tmp_path):
    """The residual stream after each layer: models cut after 1, 2, ... layers."""
    cfg, w, _, toks, _ = models["mixed"]
    fmt, tol = FMTS[dtype]
    ref = []
    O.forward(cfg, w, toks[:40], ref)
    for n in range(1, len(cfg["layers"]) + 1):
        folder = write_model(str(tmp_path / str(n)), dict(cfg, layers=cfg["layers"][:n]), w, pkg)
        m = pkg.model.Model.open(folder, fmt, max_seq=64)
        m.forward(toks[:40], 0)
        got = np.stack([m.hidden(r) for r in range(40)])
        assert max_abs_rel(got, ref[n - 1]) < (1e-5 if dtype == "f32" else 2e-2), n
        m.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_slots_are_used_again(pkg, models, dtype):
    cfg, w, folder, toks, _ = models["mixed"]
    fmt, tol = FMTS[dtype]
    m = pkg.model.Model.open(folder, fmt, batch=2, max_seq=160)
    rng = np.random.default_rng(5)
    for slot, n in ((0, 120), (1, 40), (0, 1), (1, 100), (0, 33), (0, 2)):
        seq = rng.integers(0, cfg["vocab"], n)
        m.set_sequence(slot)
        got = m.forward_logits(seq, 0, np.arange(n))
        assert logits_error(got, O.forward(cfg, w, seq)) < tol, (slot, n)


def greedy(pkg, models, name, dtype, prompts, n_new):
    """Greedy ids through Generator, checked against the logits the oracle gives for the ids produced (ties within rounding allowed)."""
    cfg, w, folder, _, _ = models[name]
    fmt, tol = FMTS[dtype]
    m = pkg.model.Model.open(folder, fmt, batch=len(prompts), max_seq=200)
    out = m.generate_batch(prompts, n_new) if len(prompts) > 1 else [m.generate(prompts[0], n_new)[0]]
    m.close()
    for p, ids in zip(prompts, out):
        seq = np.concatenate([p, ids])
        z = O.forward(cfg, w, seq[:-1])[len(p) - 1:]
        spread = np.sqrt((z * z).mean())
        for i, row in enumerate(z):
            assert row.max() - row[ids[i]] <= 4 * tol * spread, (name, i)
    return out


@pytest.mark.parametrize("name,dtype", [("mixed", "f32"), ("mixed", "bf16"), ("odd", "bf16"), ("wide_heads", "bf16")])
def test_greedy_generation_single_sequence(pkg, models, name, dtype):
    toks = models[name][3]
    out = greedy(pkg, models, name, dtype, [toks[:50]], 60)               # decodes past every window
    if dtype == "f32":
        ids, gap = O.generate(models[name][0], models[name][1], toks[:50], 12)
        assert gap < 1e-3 or list(out[0][:12]) == ids


@pytest.mark.parametrize("dtype,batch", [("f32", 3), ("bf16", 5), ("bf16", 12)])
def test_greedy_generation_of_a_batch_of_unequal_prompts(pkg, models, dtype, batch):
    toks = models["mixed"][3]
    lens = [3, 70, 1, 41, 64, 2, 90, 17, 33, 5, 16, 100][:batch]
    prompts = [np.roll(toks, 7 * i)[:n].astype(np.int32) for i, n in enumerate(lens)]
    together = greedy(pkg, models, "mixed", dtype, prompts, 25)
    if dtype == "f32":                                                    # and each alone
        for p, ids in zip(prompts, together):
            assert list(greedy(pkg, models, "mixed", dtype, [p], 25)[0]) == list(ids)


def test_limits_are_errors_not_faults(pkg, models):
    cfg, _, folder, toks, _ = models["mixed"]
    with pytest.raises(pkg.ffi.GretaError, match="learned positions"):
        pkg.model.Model.open(folder, max_seq=cfg["max_positions"] + 1)
    m = pkg.model.Model.open(folder, max_seq=64)
    with pytest.raises(pkg.ffi.GretaError, match="exceeds"):
        m.forward(toks[:65], 0)
    with pytest.raises(pkg.ffi.GretaError, match="ascend"):
        m.forward_logits(toks[:5], 0, [3, 3])
    m.generate(toks[:60], 5)                                              # ends exactly at the last position
    with pytest.raises(pkg.ffi.GretaError, match="exceeds"):
        m.generate(toks[:60], 6)
    m.close()


def test_synthetic_weights_and_missing_tensors(pkg, models, tmp_path):
    cfg, w, _, toks, _ = models["mixed"]
    m = pkg.model.Model.from_config(cfg, max_seq=100)
    m.load_synthetic(3)
    a, b = m.forward(toks[:50], 0), m.forward(toks[:50], 0)
    assert np.isfinite(a).all() and np.array_equal(a, b) and a.std() > 0.1
    m.close()
    short = {n: v for n, v in w.items() if n != "l1.mix.r1" and n != "l2.mlp.down"}
    with pytest.raises(pkg.ffi.GretaError, match="l2.mlp.down"):
        pkg.model.Model.open(write_model(str(tmp_path / "short"), cfg, short, pkg))
    wrong = dict(w, head=w["head"][:, :-1])
    with pytest.raises(pkg.ffi.GretaError, match="unexpected shape of head"):
        pkg.model.Model.open(write_model(str(tmp_path / "wrong"), cfg, wrong, pkg))


# ------------------------------------------------------------------ command line
def test_trace_run_replays_steps(pkg, models, tmp_path):
    cfg, w, folder, toks, want = models["mixed"]
    V = cfg["vocab"]
    lines, expect, pos = [], {}, 0
    for n, (k, places) in enumerate([(40, [39, 0, 7]), (2, []), (9, [8]), (1, [0]), (1, [0])]):
        lines.append({"step": n, "entries": [{"id": "a", "tokens": toks[pos:pos + k].tolist(), "want": places}], "end": ["a"] if n == 4 else []})
        if places:
            expect[n] = want[[pos + p for p in places]]
        pos += k
    other = toks[::-1][:30]
    lines.append({"step": 9, "entries": [{"id": "b", "tokens": other.tolist(), "want": [29]}], "end": ["b"]})
    expect[9] = O.forward(cfg, w, other)[29:30]
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 3e-2)):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                           input="\n".join(map(json.dumps, lines)) + "\n", capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {l['step']}" for l in lines]
        assert sorted(os.listdir(out)) == sorted(f"{n}.f32" for n in expect)
        for n, z in expect.items():
            assert logits_error(np.fromfile(out / f"{n}.f32", "<f4").reshape(-1, V), z) < tol, (dtype, n)
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--out", str(tmp_path), "--dtype", "float32"],
                       input='{"step": 0, "entries": [{"id": "a", "tokens": [%d], "want": [0]}]}\n' % V, capture_output=True, text=True, timeout=300)
    assert r.returncode != 0 and "vocabulary" in r.stderr


def test_greta_infer_generates(pkg, models):
    folder, toks = models["odd"][2], models["odd"][3]
    exe = os.path.join(ROOT, "bin", "greta_infer")
    prompt = ",".join(map(str, toks[:20]))
    m = pkg.model.Model.open(folder, pkg.ffi.FMT_F32, max_seq=64)
    ids = m.generate(toks[:20], 10)[0]
    m.close()
    r = subprocess.run([exe, "--model", folder, "--dtype", "float32", "--tokens", f"{prompt};{prompt}", "--max-tokens", "10", "--max-seq", "64"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split() == [",".join(map(str, ids))] * 2
