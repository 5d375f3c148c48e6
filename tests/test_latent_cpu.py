"""Latent attention / gated delta rule design without a GPU: configuration, rotation tables, argument checks, the oracle by itself."""
import ctypes as C
import json
import math

import numpy as np
import pytest

from _latent import CONFIGS, L, config, gated, latent, latent_2, logits_error, make_weights
from _support import load_package


@pytest.fixture(scope="module")
def pkg():
    p = load_package()
    p.build()
    return p


def check(pkg, cfg):
    h = pkg.ffi.host()
    rc = h.greta_host_check_config(json.dumps(cfg).encode())
    return None if rc == 0 else h.greta_host_last_error().decode()


def test_registry_and_configuration(pkg):
    assert "Tetilorn" in pkg.model.architectures()
    for cfg, _, _ in CONFIGS.values():
        assert check(pkg, cfg) is None
    base = CONFIGS["mixed"][0]

    def broken(edit):
        cfg = json.loads(json.dumps(base))
        edit(cfg)
        return check(pkg, cfg)

    layer = lambda c, i: c["layers"][i]["mixer"]
    assert "unknown layer type" in broken(lambda c: c["layers"][0].update(type="attention"))
    assert "unknown kind" in broken(lambda c: c["layers"][0]["mlp"].update(kind="gated"))
    assert "multiple of kv_heads" in broken(lambda c: layer(c, 0).update(kv_heads=4))
    assert "conv" in broken(lambda c: layer(c, 0).update(conv=0))
    assert "kv_rank" in broken(lambda c: layer(c, 1).pop("kv_rank"))
    assert "q_rank" in broken(lambda c: layer(c, 1).pop("q_rank"))
    assert "scale" in broken(lambda c: layer(c, 3).pop("scale"))
    assert "rot" in broken(lambda c: layer(c, 1).pop("rot"))
    assert "even" in broken(lambda c: layer(c, 1)["rot"].update(dims=5))
    assert "exceeds rot_dim" in broken(lambda c: layer(c, 1)["rot"].update(dims=14))
    assert "original" in broken(lambda c: layer(c, 1)["rot"]["scaling"].pop("original"))
    assert "factor" in broken(lambda c: layer(c, 1)["rot"]["scaling"].update(factor=-1))
    assert "embedding.scale" in broken(lambda c: c.pop("embedding"))
    assert "width" in broken(lambda c: c.pop("width"))
    assert "eps" in broken(lambda c: c.update(norm={}))


@pytest.mark.parametrize("dims,base,yarn", [(8, 1e4, None), (2, 7.0, None), (64, 1e4, (40.0, 4096, 32.0, 1.0)), (32, 500.0, (4.0, 64, 16.0, 1.0)),
                                            (6, 40.0, (32.0, 8, 3.0, 2.5)), (10, 1e6, (8.0, 100000, 1.0, 1.0)), (16, 100.0, (2.0, 4, 1e-3, 1e-4))])
def test_rotation_frequencies(pkg, dims, base, yarn):
    """Against the oracle, and the oracle against the formula pair by pair (also where both borders of the ramp fall together)."""
    scaling = dict(zip(("factor", "original", "fast", "slow"), yarn)) if yarn else None
    f, amp = L.frequencies(dims, base, scaling)
    for i in range(dims // 2):
        plain = base ** (-2.0 * i / dims)
        if yarn:
            border = [dims * math.log(yarn[1] / (2 * math.pi * t)) / (2 * math.log(base)) for t in yarn[2:]]
            lo, hi = max(math.floor(border[0]), 0), min(math.ceil(border[1]), dims - 1)
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            assert math.isclose(f[i], plain * (1 - r) + plain / yarn[0] * r, rel_tol=1e-12)
        else:
            assert math.isclose(f[i], plain, rel_tol=1e-12)
    assert math.isclose(amp, 0.1 * math.log(yarn[0]) + 1 if yarn else 1.0)
    out, a = (C.c_double * (dims // 2))(), C.c_double()
    y = (C.c_double * 4)(*yarn) if yarn else None
    assert pkg.ffi.host().greta_host_rotary(dims, base, y, out, C.byref(a)) == 0
    assert np.allclose(np.array(out), f, rtol=1e-13) and math.isclose(a.value, amp)
    assert pkg.ffi.host().greta_host_rotary(3, base, None, out, C.byref(a)) != 0


def test_argument_checks_of_the_operators(pkg):
    f, lib = pkg.ffi, pkg.ffi.cuda()
    buf = (C.c_float * 4096)()
    p = (C.addressof(buf) + 15) // 16 * 16
    rows = f.Rows(4, 0, 0, None)
    a = f.LatentAttn(4, 16, 8, 16, 32, 8, 0, 10, 10, 0.3, 1e-6, p, None, p, p, 96, p, 40, None, 0, f.FMT_F16, p, 64, p)
    assert lib.greta_cuda_latent_prepare(None, C.byref(a), C.byref(f.Rows(4, 0, 7, None)), p) == 4                  # positions past the cache
    for change in (dict(dim=257), dict(vdim=0), dict(rank=1025), dict(rot_dim=129), dict(rot_dims=7), dict(rot_dims=10), dict(rotation=None),
                   dict(fmt=f.FMT_BF16), dict(cache=None), dict(cache=p + 4), dict(down=None), dict(latent_norm=None)):
        a2 = f.LatentAttn.from_buffer_copy(a)
        for k, v in change.items():
            setattr(a2, k, v)
        assert lib.greta_cuda_latent_prepare(None, C.byref(a2), C.byref(rows), p) == 4, change
        assert lib.greta_cuda_latent_absorbed(None, C.byref(a2), C.byref(rows), p, p, 0, 64, 10) == 4, change
        assert lib.greta_cuda_latent_prefill(None, C.byref(a2), C.byref(rows), p, p, p, p, 0, 64) == 4, change
    for change in (dict(ld_w=63), dict(ld_w=0), dict(w_kv=None), dict(q=None)):
        a2 = f.LatentAttn.from_buffer_copy(a)
        for k, v in change.items():
            setattr(a2, k, v)
        assert lib.greta_cuda_latent_absorbed(None, C.byref(a2), C.byref(rows), p, p, 0, 64, 10) == 4, change
    a.fmt = f.FMT_F32
    assert lib.greta_cuda_latent_prefill(None, C.byref(a), C.byref(rows), p, p, p, p, 0, 64) == 4
    assert lib.greta_cuda_latent_row(33, 8) == 48 + 16 and lib.greta_cuda_latent_query_row(3, 65, 8) == 3 * (128 + 64)
    d = f.GatedDelta(4, 2, 16, 24, 3, 8, 8, 1e-6, p, 200, p, p, p, 4, p, p)
    for change in (dict(kv_heads=3), dict(dim=300), dict(vdim=257), dict(taps=0), dict(history=None), dict(state=None), dict(state=p + 4)):
        d2 = f.GatedDelta.from_buffer_copy(d)
        for k, v in change.items():
            setattr(d2, k, v)
        assert lib.greta_cuda_gated_delta_prepare(None, C.byref(d2), C.byref(rows)) == 4, change
    assert lib.greta_cuda_gated_delta_scan(None, C.byref(d), C.byref(rows), p) == 4                            # no decay, no inputs
    assert lib.greta_cuda_gated_delta_step(None, C.byref(d), C.byref(rows), p, 0, 96) == 4                     # rows of a portion
    assert lib.greta_cuda_gated_delta_state_bytes(3, 40, 24) == 3 * 24 * 64 * 4
    lin = f.Linear(f.FMT_BF16, p, 8, 64, 64, 1)
    lin.seg[0] = f.OutSegment(0, 8, f.ACT_SOFTPLUS_DECAY, 0, 0, None, p, 8, 0, 0)
    assert lib.greta_cuda_linear_gemm(None, C.byref(lin), p, 64, 16) == 4                                      # no rates
    lin.seg[0].act, lin.fmt = 0, f.FMT_F16
    assert lib.greta_cuda_linear_gemv(None, C.byref(lin), p, 64, None, None, 0.0, 1) == 4                      # fp16 weights: the GEMM only


def test_oracle_rotation_depends_on_distance_only():
    rng = np.random.default_rng(0)
    freq, amp = L.frequencies(8, 30.0)
    q, k = rng.normal(size=(2, 1, 1, 11))
    for inter in (False, True):
        dots = [(L.rotate(q, [p + 5], freq, amp, inter) * L.rotate(k, [p], freq, amp, inter))[0, 0, :8].sum() for p in (0, 3, 100)]
        assert np.allclose(dots, dots[0])
        assert np.array_equal(L.rotate(q, [9], freq, amp, inter)[..., 8:], q[..., 8:])                         # past the rotated channels
    turned = L.rotate(np.array([[[1.0, 0.0, 0.0, 0.0]]]), [1], np.array([math.pi / 2, 0.0]), 1.0, True)
    assert np.allclose(turned, [[[0, 1, 0, 0]]])
    turned = L.rotate(np.array([[[1.0, 0.0, 0.0, 0.0]]]), [1], np.array([math.pi / 2, 0.0]), 1.0, False)
    assert np.allclose(turned, [[[0, 0, 1, 0]]])


def test_oracle_gated_scan_matches_the_matrix_form():
    rng = np.random.default_rng(1)
    T, H, G, d, vd = 9, 4, 2, 6, 5
    q, k = rng.normal(size=(2, T, G, d))
    v, g, beta = rng.normal(size=(T, H, vd)), rng.random((T, H, d)), rng.random((T, H))
    o, S = L.gated_scan(q, k, v, g, beta)
    for h in range(H):
        M = np.zeros((d, vd))
        for t in range(T):
            kk = k[t, h // 2]
            M = (np.eye(d) - beta[t, h] * np.outer(kk, kk)) @ np.diag(g[t, h]) @ M + beta[t, h] * np.outer(kk, v[t, h])
            assert np.allclose(M.T @ q[t, h // 2], o[t, h])
        assert np.allclose(M, S[h])


def test_oracle_sink_takes_its_share():
    q, k = np.zeros((2, 1, 2, 1)), np.zeros((2, 2, 1))
    v = np.ones((2, 2, 3))
    out = L.attend(q[0].repeat(2, 0), np.zeros((2, 2, 4)), k, np.zeros((2, 4)), v, 1.0, np.array([0.0, math.log(3.0)]))
    assert np.allclose(out[:, 0, 0], [1 / 2, 2 / 3]) and np.allclose(out[:, 1, 0], [1 / 4, 2 / 5])


def test_oracle_is_causal_and_reads_every_tensor():
    cfg = config(32, 40, [gated(4, 2, 8, 6, 3, 12), latent(4, 8, 4, 6, 12, 10, 0.5, 20), latent_2(2, 6, 2, 8, 9, 0.6, 0)], 1.3)
    w = make_weights(cfg, 5, 7, 3)
    rng = np.random.default_rng(0)
    toks = rng.integers(0, 40, 20)
    base = L.forward(cfg, w, toks)
    other = toks.copy()
    other[15] = (other[15] + 1) % 40
    moved = L.forward(cfg, w, other)
    assert np.array_equal(base[:15], moved[:15]) and not np.allclose(base[15:], moved[15:])
    for name in w:
        if name == "embed":
            continue
        changed = dict(w)
        changed[name] = w[name] + 0.25 * rng.normal(size=w[name].shape)
        assert logits_error(L.forward(cfg, changed, toks), base) > 1e-4, name
