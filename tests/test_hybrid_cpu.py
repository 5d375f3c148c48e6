"""Hybrid designs without a GPU: registry and configuration, file reading, argument checks, and the oracle against itself."""
import ctypes as C
import json

import numpy as np
import pytest

from _hybrid import CONFIGS, O, attention, config, delta, logits_error, make_weights
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
    assert "Bidonex" in pkg.model.architectures()
    for cfg, _ in CONFIGS.values():
        assert check(pkg, cfg) is None
    base = CONFIGS["mixed"][0]

    def broken(edit):
        cfg = json.loads(json.dumps(base))
        edit(cfg)
        return check(pkg, cfg)

    assert "not registered" in broken(lambda c: c.update(architecture="Other"))
    assert "unknown layer type" in broken(lambda c: c["layers"][0].update(type="linear"))
    assert "unknown kind" in broken(lambda c: c["layers"][0]["mlp"].update(kind="moe"))
    assert "multiple of kv_heads" in broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=4))
    assert "width" in broken(lambda c: c.pop("width"))
    assert "eps" in broken(lambda c: c.update(norm={}))
    assert "size" in broken(lambda c: c["layers"][1]["mixer"].update(mask={"keep_first": 3}))
    assert "whole number" in broken(lambda c: c["layers"][1]["mixer"].update(conv=2.5))
    h = pkg.ffi.host()
    for text in ("", "{", '{"architecture": "Bidonex"', '{"a": [1,]}', '{"a": 1} x', '"\\u12"'):
        assert h.greta_host_check_config(text.encode()) != 0
    # escapes, nesting and unknown members are no obstacle
    cfg = dict(base, note={"text": 'a "quoted" \\ line\nwith é \U0001F600', "list": [None, True, -1.5e3, {}]})
    assert check(pkg, cfg) is None


def test_argument_checks_of_the_operators(pkg):
    f, lib = pkg.ffi, pkg.ffi.cuda()
    buf = (C.c_float * 256)()
    p = (C.addressof(buf) + 15) // 16 * 16
    lin = f.Linear(f.FMT_BF16, p, 8, 64, 64, 1)
    lin.seg[0] = f.OutSegment(0, 8, 0, 0, 0, None, p, 8, 0, 0)
    bad = [dict(fmt=f.FMT_Q4_0), dict(ldw=65), dict(K=128), dict(w=p + 4), dict(n_segments=0), dict(n_segments=2), dict(N=9), dict(w=None)]
    for change in bad:
        l2 = f.Linear.from_buffer_copy(lin)
        for k, v in change.items():
            setattr(l2, k, v)
        assert lib.greta_cuda_linear_gemv(None, C.byref(l2), p, 64, None, None, 0.0, 1) == 4, change
        assert lib.greta_cuda_linear_gemm(None, C.byref(l2), p, 64, 16) == 4, change
    assert lib.greta_cuda_linear_gemv(None, C.byref(lin), p, 64, None, None, 0.0, 9) == 4
    rows = f.Rows(4, 0, 0, None)
    a = f.WindowAttn(4, 2, 32, 32, 0, 8, 2, 10, 1.0, 5.0, 1e-6, None, None, None, None, None, p, 256, f.FMT_F16, p, p, None)
    assert lib.greta_cuda_window_attn_prepare(None, C.byref(a), C.byref(f.Rows(4, 0, 100, None)), p) == 4    # ring of 10 < 8 - 1 + 4
    for change in (dict(kv_heads=3), dict(dim=257), dict(ring=0), dict(cache_fmt=9), dict(conv=p), dict(r1=p), dict(k_cache=None)):
        a2 = f.WindowAttn.from_buffer_copy(a)
        for k, v in change.items():
            setattr(a2, k, v)
        assert lib.greta_cuda_window_attn(None, C.byref(a2), C.byref(rows), p, p, 0, 64, 100) == 4, change
    d = f.DeltaRule(2, 300, 4, 64, 1e-6)
    assert lib.greta_cuda_delta_scan(None, C.byref(d), C.byref(rows), p) == 4
    assert lib.greta_cuda_delta_state_bytes(3, 40) == 3 * 40 * 64 * 4


def test_oracle_masks_and_convolution_by_hand():
    assert [j for j in range(10) if O.visible(7, j, 3, 2)] == [0, 1, 5, 6, 7]
    assert [j for j in range(10) if O.visible(1, j, 1, 4)] == [0, 1]
    u = np.arange(1.0, 7.0).reshape(6, 1)
    assert np.allclose(O.causal_conv(u, np.array([[100.0, 10.0, 1.0]]))[:, 0], [1, 12, 123, 234, 345, 456])


def test_oracle_scan_matches_the_matrix_form():
    rng = np.random.default_rng(1)
    T, H, d = 9, 2, 6
    r, k, v = rng.normal(size=(3, T, H, d))
    w, a = rng.random((2, T, H, d))
    o, S = O.delta_scan(r, k, v, w, a)
    for h in range(H):
        M = np.zeros((d, d))
        for t in range(T):
            u = k[t, h] / np.sqrt((k[t, h] ** 2).sum() + 1e-6)
            M = (np.diag(w[t, h]) - np.outer(a[t, h] * u, u)) @ M + np.outer(k[t, h], v[t, h])
            assert np.allclose(M.T @ r[t, h], o[t, h])
        assert np.allclose(M, S[h])


def test_oracle_is_causal_and_reads_every_mechanism():
    """A later token changes nothing earlier; each tensor of a layer matters for the logits."""
    cfg = config(32, 40, [delta(2, 8, 12), attention(4, 2, 8, 12, 3, 6, 2, 0.7, 4.0, 20)], max_positions=64)
    w = make_weights(cfg, 4, 3)
    rng = np.random.default_rng(0)
    toks = rng.integers(0, 40, 20)
    base = O.forward(cfg, w, toks)
    other = toks.copy()
    other[15] = (other[15] + 1) % 40
    moved = O.forward(cfg, w, other)
    assert np.array_equal(base[:15], moved[:15]) and not np.allclose(base[15:], moved[15:])
    for name in w:
        if name in ("embed", "head"):
            continue
        changed = dict(w)
        changed[name] = w[name] + 0.25 * rng.normal(size=w[name].shape)
        assert logits_error(O.forward(cfg, changed, toks), base) > 1e-4, name
