"""Small random models of the latent attention / gated delta rule design for the tests: configurations and weights."""
import numpy as np

from _hybrid import bf16_bits, bf16_round, logits_error, write_model
from oracle import latent_oracle as L


def ff(width):
    return {"kind": "dense", "ff": width} if width else None


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, mlp, base=500.0, yarn=None):
    """The form with a query latent, sinks, gate and halves turned together (YaRN optional)."""
    rot = {"base": base, "dims": rot_dim}
    if yarn:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "latent_attention", "mlp": ff(mlp),
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale, "rot": rot}}


def latent_2(heads, dim, rot_dim, vdim, kv_rank, scale, mlp, base=500.0):
    return {"type": "latent_attention_2", "mlp": ff(mlp),
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}}


def gated(heads, kv_heads, dim, vdim, conv, mlp):
    return {"type": "channel_delta", "mlp": ff(mlp), "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def config(width, vocab, layers, scale=1.0, eps=1e-5):
    return {"architecture": "Tetilorn", "width": width, "vocab": vocab, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


# (configuration, low-rank widths of the decay and the gate).  Sizes are unequal on purpose: head sizes, latents and ranks off the
# powers of two, value heads that share keys, feed-forwards behind any kind of layer, several scalings and their absence.
CONFIGS = {
    "mixed": (config(132, 203, [gated(6, 2, 40, 56, 3, 150), latent(5, 24, 12, 40, 52, 36, 0.2, 96, yarn=(4.0, 64, 16.0, 1.0)), gated(3, 3, 64, 24, 5, 0),
                                latent_2(4, 48, 8, 20, 70, 0.15, 0), latent(2, 33, 20, 17, 88, 50, 0.17, 60)], 0.7), 13, 30),
    "odd": (config(75, 90, [latent_2(3, 7, 2, 5, 9, 0.4, 33), gated(2, 1, 9, 33, 2, 0), gated(1, 1, 33, 7, 1, 21),
                            latent(1, 20, 6, 70, 31, 6, 0.3, 0, base=40.0, yarn=(32.0, 8, 3.0, 2.5))], 2.5, 3e-4), 5, 1),
    "wide": (config(160, 128, [latent(20, 16, 32, 24, 144, 72, 0.2, 64, base=1e4, yarn=(2.0, 4096, 32.0, 1.0)), gated(4, 2, 130, 160, 4, 130),
                               latent_2(34, 128, 64, 136, 200, 0.07, 0), gated(2, 2, 96, 128, 4, 0)], 1.0, 1e-6), 40, 24),
}


def make_weights(cfg, rank_a, rank_g, seed, matrix_scale=1.0):
    """Random tensors rounded to bf16 (what a file holds), as float32."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, rows, cols, gain=1.0):
        w[name] = rng.normal(0, gain * matrix_scale / np.sqrt(cols), (rows, cols))

    def norm(name, n):
        w[name] = 1 + 0.2 * rng.normal(size=n)

    mat("embed", V, D, gain=np.sqrt(D))
    norm("final.norm", D)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", l["mixer"]
        norm(f"l{i}.norm1", D)
        H, d = m["heads"], m["dim"]
        if l["type"] == "channel_delta":
            G, vd, t = m["kv_heads"], m["vdim"], m["conv"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * vd)):
                mat(p + n, rows, D)
                w[p + n + ".conv"] = rng.normal(0, 0.7, (rows, t))
            mat(p + "b", H, D, gain=2.0)
            mat(p + "a1", rank_a, D)
            mat(p + "a2", H * d, rank_a, gain=1.5)
            w[p + "A_log"] = rng.normal(-1.0, 1.0, H)
            w[p + "dt_bias"] = rng.normal(-2.0, 1.0, H * d)
            mat(p + "g1", rank_g, D)
            mat(p + "g2", H * vd, rank_g, gain=1.5)
            norm(p + "norm", vd)
            mat(p + "o", D, H * vd)
        else:
            r, vd, R = m["rot_dim"], m["vdim"], m["kv_rank"]
            if l["type"] == "latent_attention":
                Q = m["q_rank"]
                mat(p + "dq", Q, D)
                norm(p + "dq.norm", Q)
                mat(p + "uq", H * (d + r), Q, gain=1.5)
                w[p + "sink"] = rng.normal(0, 1.5, H)
                mat(p + "g", H * vd, D)
            else:
                mat(p + "q", H * (d + r), D, gain=1.5)
            mat(p + "dkv", R + r, D)
            norm(p + "dkv.norm", R)
            mat(p + "uk", H * d, R)
            mat(p + "uv", H * vd, R)
            mat(p + "o", D, H * vd, gain=1.5)
        if l["mlp"]:
            norm(f"l{i}.norm2", D)
            mat(f"l{i}.mlp.up", l["mlp"]["ff"], D)
            mat(f"l{i}.mlp.down", D, l["mlp"]["ff"])
    return {n: bf16_round(v) for n, v in w.items()}


__all__ = ["CONFIGS", "L", "bf16_bits", "bf16_round", "config", "ff", "gated", "latent", "latent_2", "logits_error", "make_weights", "write_model"]
