"""Latent attention / gated delta rule design on the GPU against the plain float64 oracle: every mechanism through the C ABI,
then whole models through the scheduler, the generator and the command-line programs."""
import ctypes as C
import json
import os
import subprocess

import numpy as np
import pytest

from _latent import CONFIGS, L, bf16_bits, bf16_round, logits_error, make_weights, write_model
from _support import ROOT, load_package, max_abs_rel
from test_hybrid_gpu import dev, pad_cols, sync

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


def up(n, to):
    return (n + to - 1) // to * to


# ------------------------------------------------------------------ dense operators
def test_rms_norm_rows_and_scaled_embedding(g):
    rng = np.random.default_rng(2)
    lib = g.cuda()
    for M, D, ldx, ld in ((7, 300, 304, 320), (3, 77, 80, 77), (5, 9000, 9000, 9000)):
        x, w = rng.normal(5, 3, (M, D)).astype(np.float32), rng.normal(1, 1, D).astype(np.float32)
        x[0] *= 1e-4                                         # the epsilon matters
        xd, wd, o = dev(g, pad_cols(x, ldx)), dev(g, w), g.DeviceBuffer(M * ld * 4, zero=True)
        want = L.rms_norm(x.astype(np.float64), w, 1e-2)
        for fmt, kind, tol in ((g.OUT_F32, np.float32, 2e-6), (g.OUT_F16, np.float16, 1e-3)):
            g.check(lib.greta_cuda_rms_norm(None, xd.ptr, ldx, wd.ptr, 1e-2, o.ptr, fmt, M, D, ld))
            sync(g)
            got = o.download(kind, M * ld).reshape(M, ld).astype(np.float64)
            assert max_abs_rel(got[:, :D], want) < tol
            assert fmt != g.OUT_F32 or not got[:, D:].any()
    V, D, ld = 50, 90, 128
    table, toks = rng.normal(size=(V, ld)).astype(np.float32), np.array([0, 49, 3, 50, -1, 7], np.int32)
    want = np.array([2.5 * table[t, :D] if 0 <= t < V else np.zeros(D, np.float32) for t in toks]).astype(np.float32)
    for fmt, bits in ((g.FMT_F32, table), (g.FMT_BF16, bf16_bits(table))):
        td, kd, o = dev(g, bits), dev(g, toks), g.DeviceBuffer(6 * D * 4)
        g.check(lib.greta_cuda_embedding_scaled(None, kd.ptr, td.ptr, fmt, ld, 2.5, o.ptr, 6, D, V))
        sync(g)
        assert np.allclose(o.download(np.float32, 6 * D).reshape(6, D), want, rtol=0 if fmt == g.FMT_F32 else 4e-3, atol=0)


@pytest.mark.parametrize("M", [1, 3, 8])
@pytest.mark.parametrize("fmt", ["bf16", "f32"])
def test_gemv_behind_a_root_mean_square_norm(g, M, fmt):
    rng = np.random.default_rng(M)
    f = g.FMT_BF16 if fmt == "bf16" else g.FMT_F32
    lib = g.cuda()
    for N, K in ((600, 300), (9700, 136), (40, 17000), (33, 50)):
        W, x = bf16_round(rng.normal(0, 1 / np.sqrt(K), (N, K))), rng.normal(1, 2, (M, K)).astype(np.float32)
        lw, ldw = rng.normal(1, 0.3, K).astype(np.float32), up(K, 64)
        wd, xd, nd, o = dev(g, bf16_bits(pad_cols(W, ldw)) if fmt == "bf16" else pad_cols(W, ldw)), dev(g, pad_cols(x, K + 4)), dev(g, lw), g.DeviceBuffer(M * N * 4)
        lin = g.Linear(f, wd.ptr, N, K, ldw, 1)
        lin.seg[0] = g.OutSegment(0, N, g.ACT_NONE, g.OUT_F32, 0, None, o.ptr, N, 0, 0)
        g.check(lib.greta_cuda_linear_gemv(None, C.byref(lin), xd.ptr, K + 4, nd.ptr, None, 1e-3, M))
        sync(g)
        want = L.rms_norm(x.astype(np.float64), lw, 1e-3) @ W.T.astype(np.float64)
        assert max_abs_rel(o.download(np.float32, M * N).reshape(M, N), want) < 1e-5


@pytest.mark.parametrize("gemm", [False, True])
@pytest.mark.parametrize("fmt", ["bf16", "f32"])
def test_linear_squared_relu_and_decay(g, gemm, fmt):
    rng = np.random.default_rng(5)
    f, lib = (g.FMT_BF16 if fmt == "bf16" else g.FMT_F32), g.cuda()
    for n1, n2, K, M in ((70, 133, 200, 5), (129, 64, 72, 100 if gemm else 2), (5, 3, 37, 300 if gemm else 1)):
        N, ldw = n1 + n2, up(K, 64)
        W, x = bf16_round(rng.normal(0, 3 / np.sqrt(K), (N, K))), bf16_round(rng.normal(0, 2, (M, K)))
        bias, rate = rng.normal(-2, 4, n2).astype(np.float32), np.exp(rng.normal(-2, 2, n2)).astype(np.float32)
        wd = dev(g, bf16_bits(pad_cols(W, ldw)) if fmt == "bf16" else pad_cols(W, ldw))
        xd = dev(g, bf16_bits(pad_cols(x, ldw)) if gemm and fmt == "bf16" else pad_cols(x, ldw))
        o, bd, rd = g.DeviceBuffer(M * N * 4), dev(g, bias), dev(g, rate)
        lin = g.Linear(f, wd.ptr, N, K, ldw, 2)
        lin.seg[0] = g.OutSegment(0, n1, g.ACT_RELU2, g.OUT_F32, 0, None, o.ptr, N, 0, 0)
        lin.seg[1] = g.OutSegment(n1, n2, g.ACT_SOFTPLUS_DECAY, g.OUT_F32, 0, bd.ptr, o.ptr, N, n1, 0, rd.ptr)
        if gemm:
            g.check(lib.greta_cuda_linear_gemm(None, C.byref(lin), xd.ptr, ldw, M))
        else:
            g.check(lib.greta_cuda_linear_gemv(None, C.byref(lin), xd.ptr, ldw, None, None, 0.0, M))
        sync(g)
        z = x.astype(np.float64) @ W.T.astype(np.float64)
        got = o.download(np.float32, M * N).reshape(M, N)
        assert max_abs_rel(got[:, :n1], np.maximum(z[:, :n1], 0) ** 2) < 5e-6
        assert np.abs(got[:, n1:] - np.exp(-rate.astype(np.float64) * L.softplus(z[:, n1:] + bias))).max() < 5e-6


@pytest.mark.parametrize("M", [3, 40, 300])
def test_linear_gemm_with_fp16_operands(g, M):
    rng = np.random.default_rng(M)
    for N, K in ((700, 100), (130, 520)):
        W, x, ldw, ldx = rng.normal(0, 1 / np.sqrt(K), (N, K)).astype(np.float16), rng.normal(size=(M, K)).astype(np.float16), up(K, 64), up(K, 8) + 16
        junk = np.full((M, ldx), 7, np.float16)              # columns past K are not read
        junk[:, :K] = x
        wd, xd, o = dev(g, pad_cols(W, ldw)), dev(g, junk), g.DeviceBuffer(M * N * 2)
        lin = g.Linear(g.FMT_F16, wd.ptr, N, K, ldw, 1)
        lin.seg[0] = g.OutSegment(0, N, g.ACT_NONE, g.OUT_F16, 0, None, o.ptr, N, 0, 0)
        g.check(g.cuda().greta_cuda_linear_gemm(None, C.byref(lin), xd.ptr, ldx, M))
        sync(g)
        assert max_abs_rel(o.download(np.float16, M * N).reshape(M, N).astype(np.float64), x.astype(np.float64) @ W.T.astype(np.float64)) < 1e-3


# ------------------------------------------------------------------ latent attention
class Latent:
    """One layer's latent attention on the device: caches of `slots` sequences full of garbage, inputs given per call."""

    def __init__(self, g, p, cap, cache, slots=1):
        self.g, self.lib, self.p, self.cap, self.cache = g, g.cuda(), p, cap, cache
        H, d, r, vd, R = (p[k] for k in ("H", "dim", "rot", "vdim", "rank"))
        half = cache == "f16"
        kind = np.float16 if half else np.float32
        d8, v8, ldw = up(d, 8), up(vd, 8), up(R, 64)
        w = np.zeros((H * (d8 + v8), ldw), kind)
        w[:H * d8].reshape(H, d8, ldw)[:, :d, :R] = p["uk"].reshape(H, d, R)
        w[H * d8:].reshape(H, v8, ldw)[:, :vd, :R] = p["uv"].reshape(H, vd, R)
        row = self.lib.greta_cuda_latent_row(R, r)
        ang = np.arange(cap)[:, None] * p["freq"]
        table = np.stack([np.cos(ang), np.sin(ang)], -1) * p["amp"]
        self.w = dev(g, w)
        self.bufs = [dev(g, table.astype(np.float32)), dev(g, np.asarray(p["sink"], np.float32)) if p["sink"] is not None else None,
                     dev(g, np.asarray(p["norm"], np.float32)), dev(g, np.random.default_rng(9).normal(0, 30, slots * cap * row).astype(kind))]
        b = self.bufs
        self.row, self.kv_rows, self.Hd, self.Hv = row, H * (d8 + v8), H * d8, H * v8
        self.a = g.LatentAttn(H, d, r, vd, R, 2 * len(p["freq"]), int(p["inter"]), cap, cap, p["scale"], p["eps"], b[0].ptr, b[1].ptr if b[1] else None, b[2].ptr,
                              None, 0, None, 0, None, 0, g.FMT_F16 if half else g.FMT_F32, self.w.ptr, ldw, b[3].ptr)

    def _inputs(self, x):
        """x: dict of q [M, H, dim + rot], down [M, rank + rot], gate [M, H vdim] or None, all in one projected row."""
        parts = [x["q"].reshape(len(x["q"]), -1), x["down"]] + ([x["gate"]] if x["gate"] is not None else [])
        starts = np.cumsum([0] + [p.shape[1] + 3 for p in parts])
        flat = np.concatenate([np.pad(p, ((0, 0), (0, 3))) for p in parts], 1).astype(np.float32)
        d = dev(self.g, flat)
        self.a.ld_q = self.a.ld_down = self.a.ld_gate = flat.shape[1]
        self.a.q, self.a.down = d.ptr, d.ptr + 4 * int(starts[1])
        self.a.gate = d.ptr + 4 * int(starts[2]) if x["gate"] is not None else None
        return d

    def _absorbed(self, rows, M, max_len):
        g, p = self.g, self.p
        ld = p["H"] * p["vdim"] + 5
        o, scratch = g.DeviceBuffer(M * ld * 4, zero=True), g.DeviceBuffer(self.lib.greta_cuda_latent_scratch_bytes(C.byref(self.a), M, max_len))
        scratch.fill(0xC3)
        g.check(self.lib.greta_cuda_latent_absorbed(None, C.byref(self.a), C.byref(rows), scratch.ptr, o.ptr, g.OUT_F32, ld, max_len), "absorbed")
        sync(g)
        return o.download(np.float32, M * ld).reshape(M, ld)[:, :ld - 5]

    def portion(self, x, pos0, slot=0, expanded=False):
        g, M, p = self.g, len(x["q"]), self.p
        d, rows = self._inputs(x), g.Rows(M, slot, pos0, None)
        if not expanded:
            return self._absorbed(rows, M, pos0 + M)
        n = pos0 + M
        k, v = g.DeviceBuffer(n * self.Hd * 2), g.DeviceBuffer(n * self.Hv * 2)
        ld = p["H"] * p["vdim"] + 5
        o = g.DeviceBuffer(M * ld * 4, zero=True)
        q = g.DeviceBuffer(M * self.lib.greta_cuda_latent_query_row(p["H"], p["dim"], p["rot"]) * 2)
        g.check(self.lib.greta_cuda_latent_prepare(None, C.byref(self.a), C.byref(rows), q.ptr), "prepare")
        lin = g.Linear(g.FMT_F16, self.w.ptr, self.kv_rows, p["rank"], self.a.ld_w, 2)
        lin.seg[0] = g.OutSegment(0, self.Hd, 0, g.OUT_F16, 0, None, k.ptr, self.Hd, 0, 0)
        lin.seg[1] = g.OutSegment(self.Hd, self.Hv, 0, g.OUT_F16, 0, None, v.ptr, self.Hv, 0, 0)
        g.check(self.lib.greta_cuda_linear_gemm(None, C.byref(lin), self.bufs[3].ptr + slot * self.cap * self.row * 2, self.row, n), "keys and values")
        g.check(self.lib.greta_cuda_latent_prefill(None, C.byref(self.a), C.byref(rows), q.ptr, k.ptr, v.ptr, o.ptr, g.OUT_F32, ld), "prefill")
        sync(g)
        del d
        return o.download(np.float32, M * ld).reshape(M, ld)[:, :ld - 5]

    def decode(self, x, positions, max_len):
        """Row m is the next token of slot m."""
        d, dp = self._inputs(x), dev(self.g, np.asarray(positions, np.uint32))
        out = self._absorbed(self.g.Rows(len(x["q"]), 0, 0, dp.ptr), len(x["q"]), max_len)
        del d
        return out


def latent_params(rng, H, dim, rot, vdim, rank, inter=False, sink=True, rot_dims=None, yarn=None, scale=None):
    freq, amp = L.frequencies(rot if rot_dims is None else rot_dims, 200.0, yarn)
    half = lambda a: a.astype(np.float16).astype(np.float64)
    return {"H": H, "dim": dim, "rot": rot, "vdim": vdim, "rank": rank, "inter": inter, "freq": freq, "amp": amp, "eps": 1e-5,
            "scale": float(np.float32(scale if scale else 1.3 * (dim + rot) ** -0.5)), "uk": half(rng.normal(0, rank ** -0.5, (H * dim, rank))),
            "uv": half(rng.normal(0, rank ** -0.5, (H * vdim, rank))), "norm": (1 + 0.2 * rng.normal(size=rank)).astype(np.float32),
            "sink": rng.normal(0, 1.5, H).astype(np.float32) if sink else None}


def latent_inputs(rng, p, T, gate=True):
    f = lambda *s: rng.normal(size=s).astype(np.float32)
    return {"q": 1.5 * f(T, p["H"], p["dim"] + p["rot"]), "down": f(T, p["rank"] + p["rot"]),
            "gate": L.sigmoid(f(T, p["H"] * p["vdim"])).astype(np.float32) if gate else None}


def latent_want(p, x):
    T, H, d, R = len(x["q"]), p["H"], p["dim"], p["rank"]
    q, down = x["q"].astype(np.float64), x["down"].astype(np.float64)
    c = L.rms_norm(down[:, :R], p["norm"].astype(np.float64), p["eps"])
    qr = L.rotate(q[:, :, d:], np.arange(T), p["freq"], p["amp"], p["inter"])
    kr = L.rotate(down[:, None, R:], np.arange(T), p["freq"], p["amp"], p["inter"])[:, 0]
    o = L.attend(q[:, :, :d], qr, (c @ p["uk"].T).reshape(T, H, d), kr, (c @ p["uv"].T).reshape(T, H, p["vdim"]), p["scale"], p["sink"])
    return o.reshape(T, -1) * (1.0 if x["gate"] is None else x["gate"])


def rows_of(x, a, b):
    return {k: v if v is None else v[a:b] for k, v in x.items()}


YARN = {"factor": 6.0, "original": 50, "fast": 4.0, "slow": 1.0}
LATENT_CASES = [dict(H=4, dim=32, rot=16, vdim=48, rank=64), dict(H=3, dim=20, rot=6, vdim=9, rank=33, inter=True, sink=False),
                dict(H=17, dim=64, rot=32, vdim=64, rank=200, yarn=YARN), dict(H=1, dim=7, rot=2, vdim=1, rank=5, inter=True),
                dict(H=36, dim=24, rot=40, vdim=130, rank=512, rot_dims=24), dict(H=2, dim=250, rot=128, vdim=256, rank=1000, inter=True, rot_dims=100),
                dict(H=5, dim=192, rot=64, vdim=72, rank=300, sink=False, rot_dims=2)]


@pytest.mark.parametrize("case", range(len(LATENT_CASES)))
@pytest.mark.parametrize("cache", ["f32", "f16"])
def test_latent_attention_portions_and_decoding(g, case, cache):
    """Whole, in portions down to two tokens (absorbed and expanded), then decoded through the cache, all against the oracle."""
    rng = np.random.default_rng(case)
    p = latent_params(rng, **LATENT_CASES[case])
    T = 220
    x = latent_inputs(rng, p, T, gate=case % 2 == 0)
    want = latent_want(p, x)
    tol = 2e-5 if cache == "f32" else 4e-3
    for cuts in ([200], [64, 2, 3, 60, 17, 54], [2] * 3 + [100, 94]):
        at = Latent(g, p, 240, cache)
        pos, got = 0, []
        for n in cuts:
            got.append(at.portion(rows_of(x, pos, pos + n), pos, expanded=cache == "f16" and n >= 16))
            pos += n
        for t in range(pos, T):
            got.append(at.decode(rows_of(x, t, t + 1), [t], 240))
        assert max_abs_rel(np.concatenate(got), want) < tol, cuts


@pytest.mark.parametrize("form", ["absorbed f32", "absorbed f16", "expanded"])
def test_latent_attention_far_keys_stand_out(g, form):
    """One key is lined up with one query so that its weight is near one: the first positions, tile and split borders, the token
    itself, the one before it, in portions and in decoding; lined up through the latent or through the rotated part."""
    rng = np.random.default_rng(11)
    T, cache = 200, "f32" if form.endswith("f32") else "f16"
    for inter, rotated in ((False, False), (True, True), (False, True)):
        p = latent_params(rng, 2, 32, 16, 24, 48, inter=inter, scale=0.5)
        for i, j in [(199, 0), (199, 1), (199, 63), (199, 64), (199, 65), (199, 127), (199, 128), (199, 191), (199, 192), (199, 198), (199, 199), (128, 0), (127, 64),
                     (64, 63), (64, 64), (63, 0)]:
            x = latent_inputs(rng, p, T, gate=False)
            x["q"] *= 0.2
            x["down"][:, p["rank"]:] *= 0.3
            want_c = L.rms_norm(x["down"][j, :p["rank"]].astype(np.float64), p["norm"].astype(np.float64), p["eps"])
            for h in range(2):
                if rotated:                                  # q turned to position j's direction as seen from i
                    x["down"][j, p["rank"]:] = 4.0 * np.sign(x["down"][j, p["rank"]:])
                    kr = L.rotate(x["down"][j:j + 1, None, p["rank"]:].astype(np.float64), [j], p["freq"], 1.0, inter)
                    x["q"][i, h, 32:] = 2.0 * L.rotate(kr, [i], -p["freq"], 1.0, inter)[0, 0]
                else:
                    x["q"][i, h, :32] = 2.0 * (p["uk"].reshape(2, 32, -1)[h] @ want_c)
            want = latent_want(p, x)
            v = (want_c @ p["uv"].T)
            share = (want[i] @ v) / (v @ v)
            assert share > 0.8, (i, j, share)                # the case does what it says
            at = Latent(g, p, 256, cache)
            if form == "expanded":
                got = np.concatenate([at.portion(rows_of(x, a, b), a, expanded=True) for a, b in ((0, 90), (90, 200))])
            else:
                got = np.concatenate([at.portion(rows_of(x, 0, i), 0, expanded=cache == "f16"), at.decode(rows_of(x, i, i + 1), [i], 256)])
            assert np.abs(got[i] - want[i]).max() < (1e-4 if cache == "f32" else 2e-2), (i, j)


def test_latent_attention_sink_counts_once(g):
    """The sink alone can take the weight, at the first position as at the last, also when it far exceeds every score."""
    rng = np.random.default_rng(4)
    p = latent_params(rng, 3, 24, 8, 24, 40)
    for sink in ([3.0, 30.0, -5.0], [0.0, 0.0, -80.0]):
        p["sink"] = np.array(sink, np.float32)
        x = latent_inputs(rng, p, 70)
        want = latent_want(p, x)
        for cache, expanded in (("f32", False), ("f16", False), ("f16", True)):
            at = Latent(g, p, 80, cache)
            got = at.portion(rows_of(x, 0, 69), 0, expanded=expanded)
            got = np.concatenate([got, at.decode(rows_of(x, 69, 70), [69], 80)])
            assert np.abs(got - want).max() < (1e-5 if cache == "f32" else 3e-3)


@pytest.mark.parametrize("cache", ["f32", "f16"])
def test_latent_attention_batch_of_unequal_sequences_and_reused_slots(g, cache):
    rng = np.random.default_rng(8)
    p = latent_params(rng, 20, 24, 8, 32, 56)
    tol, lens_of = (2e-5, 4e-3)[cache == "f16"], [(50, 3, 17, 140, 1, 64, 65, 2, 100, 7, 33, 128), (2, 64, 9, 1, 127, 5, 90, 63, 20, 111, 3, 40)]
    at = Latent(g, p, 160, cache, slots=12)                  # twelve rows: pairs of head groups share a CTA in the fp16 form
    for lens in lens_of:                                     # the second turn meets what the first left in the slots
        xs = [latent_inputs(rng, p, n + 8) for n in lens]
        wants = [latent_want(p, x) for x in xs]
        for s, n in enumerate(lens):
            assert max_abs_rel(at.portion(rows_of(xs[s], 0, n), 0, slot=s, expanded=cache == "f16" and n >= 16), wants[s][:n]) < tol
        for t in range(8):
            pos = [n + t for n in lens]
            x = {k: np.stack([x[k][i] for x, i in zip(xs, pos)]) for k in xs[0]}
            assert max_abs_rel(at.decode(x, pos, 160), np.stack([w[i] for w, i in zip(wants, pos)])) < tol


def test_latent_attention_long_context_in_many_splits(g):
    """One row over thousands of keys; every split has its own standing key in turn."""
    rng = np.random.default_rng(3)
    p = latent_params(rng, 2, 16, 8, 16, 32, scale=0.6)
    T = 4000
    x = latent_inputs(rng, p, T, gate=False)
    x["q"] *= 0.1
    c = L.rms_norm(x["down"][:, :32].astype(np.float64), p["norm"].astype(np.float64), p["eps"])
    kr = L.rotate(x["down"][:, None, 32:].astype(np.float64), np.arange(T), p["freq"], p["amp"], False)[:, 0]
    for cache in ("f16", "f32"):
        at = Latent(g, p, T, cache)
        at.portion(rows_of(x, 0, T - 1), 0, expanded=cache == "f16")
        for j in (0, 127, 128, 1999, 2000, 3967, 3968, T - 2):
            last = rows_of(x, T - 1, T)
            last = dict(last, q=last["q"].copy())
            for h in range(2):
                last["q"][0, h, :16] = 3.0 * (p["uk"].reshape(2, 16, -1)[h] @ c[j])
            q = last["q"][0].astype(np.float64)
            qr = L.rotate(q[None, :, 16:], [T - 1], p["freq"], p["amp"], False)[0]
            for h in range(2):
                s = ((c @ p["uk"].reshape(2, 16, -1)[h].T) @ q[h, :16] + kr @ qr[h]) * p["scale"]
                e = np.exp(s - s.max())
                want = (e @ c @ p["uv"].reshape(2, 16, -1)[h].T) / (e.sum() + np.exp(p["sink"][h] - s.max()))
                got = at.decode(last, [T - 1], T)[0, h * 16:(h + 1) * 16]
                assert np.abs(got - want).max() < (2e-5 if cache == "f32" else 5e-3), (j, h)


# ------------------------------------------------------------------ gated delta rule
class Gated:
    def __init__(self, g, p, slots=1):
        self.g, self.lib, self.p = g, g.cuda(), p
        H, G, d, vd, taps = (p[k] for k in ("H", "G", "dim", "vdim", "taps"))
        self.C = 2 * G * d + H * vd
        n = self.lib.greta_cuda_gated_delta_state_bytes(H, d, vd) // 4
        f32 = lambda a: dev(g, np.asarray(a, np.float32))
        self.b = {"state": f32(np.full(slots * n, 1e3)), "history": f32(np.full(slots * taps * self.C, 1e3)), "conv": f32(p["conv"]), "norm": f32(p["norm"]),
                  "a2": f32(p["a2"]), "g2": f32(p["g2"]), "rate": f32(np.repeat(np.exp(p["A_log"]), d)), "dt": f32(p["dt_bias"])}

    def desc(self, x):
        g, p, b = self.g, self.p, self.b
        H, d, vd, ra, rg = (p[k] for k in ("H", "dim", "vdim", "ra", "rg"))
        M, ld = len(x["proj"]), self.C + H + 2
        f32 = lambda a: dev(g, np.ascontiguousarray(a, np.float32))
        proj = f32(pad_cols(np.concatenate([x["proj"], x["beta"]], 1), ld))
        low = f32(np.concatenate([x["t"], np.full((M, 1), 9.0), x["t2"]], 1))
        ldu = up(self.C, 4)
        u, dec, gate = g.DeviceBuffer(M * ldu * 4), f32(x["decay"].reshape(M, -1)), f32(x["gate"].reshape(M, -1))
        s = g.GatedDelta(H, p["G"], d, vd, p["taps"], ra, rg, p["eps"], proj.ptr, ld, b["conv"].ptr, b["history"].ptr, proj.ptr + 4 * self.C, ld, b["norm"].ptr,
                         b["state"].ptr, low.ptr, ra + 1 + rg, ra + 1, b["a2"].ptr, b["g2"].ptr, b["rate"].ptr, b["dt"].ptr, u.ptr, ldu, dec.ptr, gate.ptr, H * d, H * vd)
        return s, (proj, low, u, dec, gate)

    def portion(self, x, pos0, slot=0):
        g, M, HV = self.g, len(x["proj"]), self.p["H"] * self.p["vdim"]
        s, hold = self.desc(x)
        rows = g.Rows(M, slot, pos0, None)
        ob, o = g.DeviceBuffer(M * HV * 4), g.DeviceBuffer(M * (HV + 7) * 4)
        g.check(self.lib.greta_cuda_gated_delta_prepare(None, C.byref(s), C.byref(rows)), "prepare")
        g.check(self.lib.greta_cuda_gated_delta_scan(None, C.byref(s), C.byref(rows), ob.ptr), "scan")
        g.check(self.lib.greta_cuda_gated_delta_output(None, C.byref(s), ob.ptr, M, o.ptr, g.OUT_F32, HV + 7), "output")
        sync(g)
        del hold
        return o.download(np.float32, M * (HV + 7)).reshape(M, HV + 7)[:, :HV]

    def step(self, x, positions):
        g, M, HV = self.g, len(x["proj"]), self.p["H"] * self.p["vdim"]
        s, hold = self.desc(x)
        dp, o = dev(g, np.asarray(positions, np.uint32)), g.DeviceBuffer(M * HV * 4)
        g.check(self.lib.greta_cuda_gated_delta_step(None, C.byref(s), C.byref(g.Rows(M, 0, 0, dp.ptr)), o.ptr, g.OUT_F32, HV), "step")
        sync(g)
        del hold
        return o.download(np.float32, M * HV).reshape(M, HV)


def gated_params(rng, H, G, dim, vdim, taps, ra, rg):
    f = lambda *s: rng.normal(size=s).astype(np.float32)
    return {"H": H, "G": G, "dim": dim, "vdim": vdim, "taps": taps, "ra": ra, "rg": rg, "eps": 1e-5, "conv": 0.7 * f(2 * G * dim + H * vdim, taps),
            "norm": 1 + 0.2 * f(vdim), "a2": 1.5 * f(H * dim, ra) / ra ** 0.5, "g2": 1.5 * f(H * vdim, rg) / rg ** 0.5, "A_log": f(H) - 1, "dt_bias": f(H * dim) - 2}


def gated_inputs(rng, p, T):
    f = lambda *s: rng.normal(size=s).astype(np.float32)
    x = {"proj": f(T, 2 * p["G"] * p["dim"] + p["H"] * p["vdim"]), "beta": L.sigmoid(2 * f(T, p["H"])).astype(np.float32), "t": f(T, p["ra"]), "t2": f(T, p["rg"])}
    z = (x["t"].astype(np.float64) @ p["a2"].T.astype(np.float64)).reshape(T, p["H"], p["dim"])
    x["decay"] = L.channel_decay(z, p["A_log"].astype(np.float64), p["dt_bias"].astype(np.float64))
    x["gate"] = L.sigmoid(x["t2"].astype(np.float64) @ p["g2"].T.astype(np.float64))
    return x


def gated_want(p, x):
    T, H, G, d, vd = len(x["proj"]), p["H"], p["G"], p["dim"], p["vdim"]
    u = L.silu(L.causal_conv(x["proj"].astype(np.float64), p["conv"].astype(np.float64)))
    q, k = L.unit(u[:, :G * d].reshape(T, G, d)) * d ** -0.5, L.unit(u[:, G * d:2 * G * d].reshape(T, G, d))
    o, _ = L.gated_scan(q, k, u[:, 2 * G * d:].reshape(T, H, vd), x["decay"], x["beta"].astype(np.float64))
    return L.rms_norm(o, p["norm"].astype(np.float64), p["eps"]).reshape(T, H * vd) * x["gate"]


GATED_CASES = [(6, 2, 40, 56, 3, 7, 12), (2, 2, 64, 64, 4, 33, 16), (1, 1, 7, 9, 2, 1, 1), (4, 1, 96, 128, 1, 16, 20), (2, 1, 130, 200, 6, 5, 8), (2, 2, 256, 34, 4, 40, 3),
               (3, 3, 32, 256, 5, 8, 8)]


@pytest.mark.parametrize("case", range(len(GATED_CASES)))
def test_gated_delta_portions_and_decoding(g, case):
    rng = np.random.default_rng(case)
    p = gated_params(rng, *GATED_CASES[case])
    T = 90
    x = gated_inputs(rng, p, T)
    x["proj"][20:26] *= 1e-3                                 # the 1e-6 of the unit vectors, the eps of the norm
    want = gated_want(p, x)
    for cuts in ([70], [2, 16, 2, 17, 33], [64, 6], [3, 2, 2]):
        m = Gated(g, p)
        pos, got = 0, []
        for n in cuts:
            got.append(m.portion(rows_of(x, pos, pos + n), pos))
            pos += n
        for i in range(pos, T):
            got.append(m.step(rows_of(x, i, i + 1), [i]))
        assert max_abs_rel(np.concatenate(got), want) < 5e-5, cuts


def test_gated_delta_batch_and_reused_slots(g):
    rng = np.random.default_rng(3)
    p = gated_params(rng, 4, 2, 48, 24, 4, 6, 5)
    m = Gated(g, p, slots=3)
    for lens in ((30, 2, 11), (3, 20, 0)):                   # a slot that starts with a decoded token, slots used again
        xs = [gated_inputs(rng, p, n + 12) for n in lens]
        wants = [gated_want(p, x) for x in xs]
        for s, n in enumerate(lens):
            if n:
                assert max_abs_rel(m.portion(rows_of(xs[s], 0, n), 0, slot=s), wants[s][:n]) < 5e-5
        for i in range(12):
            pos = [n + i for n in lens]
            x = {k: np.stack([xs[s][k][pos[s]] for s in range(3)]) for k in xs[0]}
            assert max_abs_rel(m.step(x, pos), np.stack([wants[s][pos[s]] for s in range(3)])) < 5e-5


def test_gated_delta_remembers_far_back(g):
    """Slow decay, one write at position 0 and none after it: read back hundreds of tokens later, in one portion or many."""
    rng = np.random.default_rng(6)
    p = gated_params(rng, 2, 1, 32, 40, 2, 1, 1)
    p["conv"][:, 0], p["conv"][:, 1], p["eps"], T = 0, 1, 1e-12, 400
    x = gated_inputs(rng, p, T)
    x["proj"][:, :64] = rng.normal(size=64)                  # the same query and key throughout
    x["beta"][1:] = 0
    x["decay"][:] = np.exp(-np.exp(p["A_log"].astype(np.float64))[:, None] * 1e-4)
    want = gated_want(p, x)
    for cuts in ([400], [16] * 25, [399, 1], [2, 398]):
        m, pos = Gated(g, p), 0
        for n in cuts:
            out = m.portion(rows_of(x, pos, pos + n), pos)
            pos += n
        assert max_abs_rel(out[-1], want[-1]) < 1e-4


# ------------------------------------------------------------------ whole models
FMTS = {"f32": (0, 3e-5), "bf16": (2, 3e-2)}


@pytest.fixture(scope="module")
def models(pkg, tmp_path_factory):
    out = {}
    for name, (cfg, ra, rg) in CONFIGS.items():
        w = make_weights(cfg, ra, rg, 17)
        folder = write_model(str(tmp_path_factory.mktemp(name)), cfg, w, pkg)
        toks = np.random.default_rng(1).integers(0, cfg["vocab"], 150)
        out[name] = (cfg, w, folder, toks, L.forward(cfg, w, toks))
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
    for cuts in ([2] * 5 + [64, 3, 9, 30, 34], [33, 8, 7, 102], [149, 1], [15, 16, 17, 102]):
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
    fmt, _ = FMTS[dtype]
    ref = []
    L.forward(cfg, w, toks[:40], ref)
    for n in range(1, len(cfg["layers"]) + 1):
        folder = write_model(str(tmp_path / str(n)), dict(cfg, layers=cfg["layers"][:n]), w, pkg)
        m = pkg.model.Model.open(folder, fmt, max_seq=64)
        m.forward(toks[:40], 0)
        got = np.stack([m.hidden(r) for r in range(40)])
        assert max_abs_rel(got, ref[n - 1]) < (2e-5 if dtype == "f32" else 2e-2), n
        m.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_slots_are_used_again(pkg, models, dtype):
    cfg, w, folder, _, _ = models["mixed"]
    fmt, tol = FMTS[dtype]
    m = pkg.model.Model.open(folder, fmt, batch=2, max_seq=160)
    rng = np.random.default_rng(5)
    for slot, n in ((0, 120), (1, 40), (0, 1), (1, 100), (0, 33), (0, 2)):
        seq = rng.integers(0, cfg["vocab"], n)
        m.set_sequence(slot)
        got = m.forward_logits(seq, 0, np.arange(n))
        assert logits_error(got, L.forward(cfg, w, seq)) < tol, (slot, n)
    m.close()


def greedy(pkg, models, name, dtype, prompts, n_new):
    """Greedy ids through Generator, checked against the logits the oracle gives for the ids produced (ties within rounding allowed)."""
    cfg, w, folder, _, _ = models[name]
    fmt, tol = FMTS[dtype]
    m = pkg.model.Model.open(folder, fmt, batch=len(prompts), max_seq=200)
    out = m.generate_batch(prompts, n_new) if len(prompts) > 1 else [m.generate(prompts[0], n_new)[0]]
    m.close()
    for p, ids in zip(prompts, out):
        seq = np.concatenate([p, ids])
        z = L.forward(cfg, w, seq[:-1])[len(p) - 1:]
        spread = np.sqrt((z * z).mean())
        for i, row in enumerate(z):
            assert row.max() - row[ids[i]] <= 4 * tol * spread, (name, i)
    return out


@pytest.mark.parametrize("name,dtype", [("mixed", "f32"), ("mixed", "bf16"), ("odd", "bf16"), ("wide", "bf16")])
def test_greedy_generation_single_sequence(pkg, models, name, dtype):
    toks = models[name][3]
    out = greedy(pkg, models, name, dtype, [toks[:50]], 100)              # decodes past several tiles of keys
    if dtype == "f32":
        ids, gap = L.generate(models[name][0], models[name][1], toks[:50], 12)
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


def test_limits_defaults_and_missing_tensors(pkg, models, tmp_path):
    cfg, w, folder, toks, _ = models["odd"]
    m = pkg.model.Model.open(folder)
    assert m.cfg["max_seq"] == 8192                                       # nothing in the design bounds it
    m.close()
    m = pkg.model.Model.open(folder, max_seq=64)
    with pytest.raises(pkg.ffi.GretaError, match="exceeds"):
        m.forward(toks[:65], 0)
    m.generate(toks[:60], 5)                                              # ends exactly at the last position
    with pytest.raises(pkg.ffi.GretaError, match="exceeds"):
        m.generate(toks[:60], 6)
    m.close()
    m = pkg.model.Model.from_config(models["mixed"][0], max_seq=100)
    m.load_synthetic(3)
    a, b = m.forward(toks[:50], 0), m.forward(toks[:50], 0)
    assert np.isfinite(a).all() and np.array_equal(a, b) and a.std() > 0.1
    m.close()
    for gone in ("l0.mix.uk", "l1.mix.a1", "l3.mix.sink", "l2.norm2", "final.norm", "l3.mix.dq"):
        short = {n: v for n, v in w.items() if n != gone}
        with pytest.raises(pkg.ffi.GretaError, match=gone):
            pkg.model.Model.open(write_model(str(tmp_path / gone), cfg, short, pkg))
    with pytest.raises(pkg.ffi.GretaError, match="unexpected shape of l0.mix.dkv"):
        pkg.model.Model.open(write_model(str(tmp_path / "wrong"), cfg, dict(w, **{"l0.mix.dkv": w["l0.mix.dkv"][:-1]}), pkg))


# ------------------------------------------------------------------ command line
def test_trace_run_replays_steps(pkg, models, tmp_path):
    cfg, w, folder, toks, want = models["mixed"]
    V = cfg["vocab"]
    lines, expect, pos = [], {}, 0
    for n, (k, places) in enumerate([(40, [39, 0, 7]), (2, []), (9, [8]), (1, [0]), (1, [0]), (30, [0, 29])]):
        lines.append({"step": n, "entries": [{"id": "a", "tokens": toks[pos:pos + k].tolist(), "want": places}], "end": ["a"] if n == 5 else []})
        if places:
            expect[n] = want[[pos + p for p in places]]
        pos += k
    other = toks[::-1][:30]
    lines.append({"step": 9, "entries": [{"id": "b", "tokens": other.tolist(), "want": [29]}], "end": ["b"]})
    expect[9] = L.forward(cfg, w, other)[29:30]
    for dtype, tol in (("float32", 3e-5), ("bfloat16", 3e-2)):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "83"],
                           input="\n".join(map(json.dumps, lines)) + "\n", capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {l['step']}" for l in lines]
        for n, z in expect.items():
            assert logits_error(np.fromfile(out / f"{n}.f32", "<f4").reshape(-1, V), z) < tol, (dtype, n)


def test_greta_infer_generates(pkg, models):
    folder, toks = models["odd"][2], models["odd"][3]
    prompt = ",".join(map(str, toks[:20]))
    m = pkg.model.Model.open(folder, pkg.ffi.FMT_F32, max_seq=64)
    ids = m.generate(toks[:20], 10)[0]
    m.close()
    r = subprocess.run([os.path.join(ROOT, "bin", "greta_infer"), "--model", folder, "--dtype", "float32", "--tokens", f"{prompt};{prompt}", "--max-tokens", "10"],
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split() == [",".join(map(str, ids))] * 2
