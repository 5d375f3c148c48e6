"""Plain float64 restatement of the latent attention / gated delta rule decoder ("Tetilorn" design).

One function per mechanism, loops over positions where the mechanism is defined position by position; nothing here is
shared with the product path.  Weights are a dict name -> float array, the configuration is the parsed config.json.

Notation: x residual stream, h = RMS(x) * w; rows are positions t = 0 .. T-1 (first + t with an offset).
"""
import math

import numpy as np

F = np.float64


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


# ------------------------------------------------------------------ rotary positions
def frequencies(dims, base, scaling=None):
    """-> frequency per pair, amplitude of cos and sin."""
    i = np.arange(dims // 2, dtype=F)
    f = base ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0

    def where(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(where(scaling["fast"])), 0)
    hi = min(math.ceil(where(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, pos, freq, amp, interleaved):
    """x [T, n, d]: pairs among the first 2 len(freq) channels, neighbours (interleaved) or halves apart; pos [T]."""
    n = len(freq)
    a = np.asarray(pos, F)[:, None] * freq
    c, s = (np.cos(a) * amp)[:, None], (np.sin(a) * amp)[:, None]
    y = x.copy()
    first, second = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if interleaved else (slice(0, n), slice(n, 2 * n))
    u, v = x[..., first], x[..., second]
    y[..., first], y[..., second] = u * c - v * s, v * c + u * s
    return y


# ------------------------------------------------------------------ latent attention
def attend(q, qr, k, kr, v, scale, sink=None):
    """q, k [T, H, dim], qr [T, H, r], kr [T, r] (one for all heads), v [T, H, vdim]; sink [H] or None."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        for h in range(H):
            s = (k[:i + 1, h] @ q[i, h] + kr[:i + 1] @ qr[i, h]) * scale
            m = s.max() if sink is None else max(s.max(), sink[h])
            e = np.exp(s - m)
            out[i, h] = (e @ v[:i + 1, h]) / (e.sum() + (0.0 if sink is None else math.exp(sink[h] - m)))
    return out


def latent_mixer(h, w, pre, m, eps, interleaved, low_rank_q, sink, gate):
    H, d, r, vd, R, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], h.shape[0]
    rot = m["rot"]
    freq, amp = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    if low_rank_q:
        q = rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T
    else:
        q = h @ w[pre + "q"].T
    q = q.reshape(T, H, d + r)
    down = h @ w[pre + "dkv"].T
    c = rms_norm(down[:, :R], w[pre + "dkv.norm"], eps)
    pos = np.arange(T)
    qr = rotate(q[:, :, d:], pos, freq, amp, interleaved)
    kr = rotate(down[:, None, R:], pos, freq, amp, interleaved)[:, 0]
    k = (c @ w[pre + "uk"].T).reshape(T, H, d)
    v = (c @ w[pre + "uv"].T).reshape(T, H, vd)
    o = attend(q[:, :, :d], qr, k, kr, v, m["scale"], w[pre + "sink"] if sink else None).reshape(T, H * vd)
    if gate:
        o = o * sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


# ------------------------------------------------------------------ gated delta rule, a decay per key channel
def causal_conv(u, w):
    """y[t, c] = sum_j w[c, j] u[t - taps + 1 + j, c], zeros in front of the sequence."""
    T, taps = u.shape[0], w.shape[1]
    y = np.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def channel_decay(z, a_log, dt_bias):
    """z [T, H, dim] -> decay in (0, 1), rates exp(a_log) per head."""
    return np.exp(-np.exp(a_log)[:, None] * softplus(z + dt_bias.reshape(z.shape[1:])))


def gated_scan(q, k, v, g, beta, S=None):
    """q, k [T, G, dim], v [T, H, vdim], g [T, H, dim], beta [T, H]; state S [H, dim, vdim].  -> o [T, H, vdim], S"""
    T, H, vd = v.shape
    per = H // q.shape[1]
    S = np.zeros((H, q.shape[2], vd)) if S is None else S.copy()
    o = np.zeros((T, H, vd))
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // per], q[t, h // per]
            S[h] *= g[t, h][:, None]
            S[h] += np.outer(kk, beta[t, h] * (v[t, h] - S[h].T @ kk))
            o[t, h] = S[h].T @ qq
    return o, S


def delta_mixer(h, w, pre, m, eps):
    H, G, d, vd, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (silu(causal_conv(h @ w[pre + n].T, w[pre + n + ".conv"])) for n in "qkv")
    q = unit(q.reshape(T, G, d)) * d ** -0.5
    k = unit(k.reshape(T, G, d))
    beta = sigmoid(h @ w[pre + "b"].T)
    g = channel_decay((h @ w[pre + "a1"].T @ w[pre + "a2"].T).reshape(T, H, d), w[pre + "A_log"], w[pre + "dt_bias"])
    o, _ = gated_scan(q, k, v.reshape(T, H, vd), g, beta)
    o = rms_norm(o, w[pre + "norm"], eps).reshape(T, H * vd)
    return (o * sigmoid(h @ w[pre + "g1"].T @ w[pre + "g2"].T)) @ w[pre + "o"].T


def mixer(kind, h, w, pre, m, eps):
    if kind == "latent_attention":
        return latent_mixer(h, w, pre, m, eps, interleaved=False, low_rank_q=True, sink=True, gate=True)
    if kind == "latent_attention_2":
        return latent_mixer(h, w, pre, m, eps, interleaved=True, low_rank_q=False, sink=False, gate=False)
    assert kind == "channel_delta", kind
    return delta_mixer(h, w, pre, m, eps)


def feed_forward(h, w, pre):
    return np.maximum(h @ w[pre + "up"].T, 0.0) ** 2 @ w[pre + "down"].T


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence from position 0; the residual stream after every layer goes to layers_out."""
    w = {n: np.asarray(v, F) for n, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + mixer(layer["type"], rms_norm(x, w[pre + "norm1"], eps), w, pre + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + feed_forward(rms_norm(x, w[pre + "norm2"], eps), w, pre + "mlp.")
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


def generate(cfg, w, prompt, n_new):
    """Greedy ids (first maximum), the whole sequence recomputed for every new id.  -> ids, smallest top-2 gap seen"""
    seq, gap = list(prompt), math.inf
    for _ in range(n_new):
        z = forward(cfg, w, seq)[-1]
        top = np.sort(z)[-2:]
        gap = min(gap, float(top[1] - top[0]))
        seq.append(int(np.argmax(z)))
    return seq[len(prompt):], gap
