"""Small random models of the hybrid designs for the tests: configurations, weights, model folders."""
import json
import os

import numpy as np

from oracle import hybrid_oracle as O


def bf16_bits(a):
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def bf16_round(a):
    return (bf16_bits(a).astype(np.uint32) << 16).view(np.float32)


def attention(heads, kv_heads, dim, vdim, conv, size, keep, scale, softcap, ff):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "softcap": softcap,
                      "mask": {"size": size, "keep_first": keep}}}


def delta(heads, dim, ff):
    return {"type": "general_delta", "mlp": {"kind": "dense", "ff": ff} if ff else None, "mixer": {"heads": heads, "dim": dim}}


def config(width, vocab, layers, max_positions=512, eps=1e-5):
    return {"architecture": "Bidonex", "width": width, "vocab": vocab, "max_positions": max_positions, "norm": {"eps": eps}, "layers": layers}


# Sizes are unequal on purpose: key and value head sizes, ranks and widths off the powers of two, several window forms.
CONFIGS = {
    "mixed": (config(136, 203, [delta(3, 40, 150), attention(6, 2, 48, 24, 4, 37, 5, 0.3, 9.0, 200), delta(2, 64, 96),
                                attention(5, 1, 32, 40, 2, 64, 0, 0.15, 30.0, 77)]), 24),
    "odd": (config(75, 90, [attention(3, 3, 20, 36, 3, 1, 3, 0.5, 5.0, 0), delta(1, 7, 33), delta(5, 33, 0), attention(4, 4, 9, 5, 1, 11, 20, 1.0, 2.0, 51)],
                   eps=3e-4), 5),
    "wide_heads": (config(160, 128, [attention(2, 1, 136, 256, 5, 90, 12, 0.08, 15.0, 64), delta(1, 160, 130), attention(9, 1, 64, 128, 2, 30, 2, 0.125, 50.0, 64)]), 40),
}


def make_weights(cfg, rank, seed, matrix_scale=1.0):
    """Random tensors rounded to bf16 (what a file holds), as float32."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, *shape, gain=1.0):
        w[name] = rng.normal(0, gain * matrix_scale / np.sqrt(shape[-1]), shape)

    mat("embed", V, D, gain=np.sqrt(D))
    mat("pos", cfg["max_positions"], D, gain=0.5 * np.sqrt(D))
    mat("head", V, D)

    def norm(name, n):
        w[name] = 1 + 0.2 * rng.normal(size=n)
        w[name + ".b"] = 0.1 * rng.normal(size=n)

    norm("final.norm", D)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        norm(p + "norm1", D)
        H, d = m["heads"], m["dim"]
        if l["type"] == "attention":
            G, vd, t = m["kv_heads"], m["vdim"], m["conv"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * vd)):
                mat(p + "mix." + n, rows, D)
                w[p + f"mix.{n}.conv"] = rng.normal(0, 0.7, (rows, t))
            w[p + "mix.temp"] = 0.5 + rng.random(H)
            w[p + "mix.r1"] = 0.2 + rng.random(H)
            w[p + "mix.r2"] = 0.05 + rng.random(H)
            w[p + "mix.sink"] = rng.normal(0, 1.5, H)
            mat(p + "mix.o", D, H * vd, gain=1.5)
        else:
            for n in "rkvga":
                mat(p + "mix." + n, H * d, D)
            w[p + "mix.a.b"] = 0.5 * rng.normal(size=H * d)
            mat(p + "mix.w1", rank, D)
            mat(p + "mix.w2", H * d, rank, gain=2.0)
            w[p + "mix.w0"] = rng.normal(-2.0, 1.5, H * d)
            w[p + "mix.norm"] = 1 + 0.2 * rng.normal(size=H * d)
            mat(p + "mix.o", D, H * d)
        if l["mlp"]:
            mat(p + "mlp.up", l["mlp"]["ff"], D)
            mat(p + "mlp.down", D, l["mlp"]["ff"])
    return {n: bf16_round(v) for n, v in w.items()}


def write_model(folder, cfg, weights, pkg):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    pkg.model.write_safetensors(os.path.join(folder, "model.safetensors"), {n: bf16_bits(a) for n, a in weights.items()})
    return folder


def logits_error(got, want):
    """Root mean square over the vocabulary of the difference (mean taken off), relative to the rms of the wanted logits; worst row."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(-1, keepdims=True)
    c = want - want.mean(-1, keepdims=True)
    return float(np.sqrt((d * d).mean(-1)).max() / np.sqrt((c * c).mean()))


__all__ = ["O", "CONFIGS", "attention", "bf16_bits", "bf16_round", "config", "delta", "logits_error", "make_weights", "write_model"]
