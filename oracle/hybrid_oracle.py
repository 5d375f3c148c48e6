"""Plain float64 restatement of the parallel attention / delta-rule decoder ("Bidonex" design).

One function per mechanism, loops over positions where the mechanism is defined position by position; nothing here is
shared with the product path.  Weights are a dict name -> float array, the configuration is the parsed config.json.

Notation: x residual stream, h = LN(x); rows are positions t = 0 .. T-1.
"""
import math

import numpy as np

F = np.float64


def layer_norm(x, w, b, eps):
    mu = x.mean(-1, keepdims=True)
    c = x - mu
    return c / np.sqrt((c * c).mean(-1, keepdims=True) + eps) * w + b


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def gelu_erf(z):
    erf = np.vectorize(math.erf, otypes=[F])
    return 0.5 * z * (1.0 + erf(z / math.sqrt(2.0)))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


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


def visible(i, j, size, keep_first):
    """Sliding window of `size` positions that also keeps the first `keep_first` of the sequence."""
    return j <= i and (i - j < size or j < keep_first)


def attend(q, k, v, p, size, keep_first, scale, softcap):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim]; p: per-head temp, r1, r2, sink.  -> [T, H, vdim]"""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        js = np.array([j for j in range(i + 1) if visible(i, j, size, keep_first)])
        for h in range(H):
            g = h // (H // G)
            s = (k[js, g] @ q[i, h]) * scale * p["temp"][h]
            s = softcap * np.tanh(s / softcap)
            s = s - p["r1"][h] * np.log(1.0 + p["r2"][h] * (i - js))
            m = max(s.max(), p["sink"][h])
            e = np.exp(s - m)
            out[i, h] = (e @ v[js, g]) / (e.sum() + math.exp(p["sink"][h] - m))
    return out


def attention_mixer(h, w, pre, m, eps):
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (causal_conv(h @ w[pre + n].T, w[pre + n + ".conv"]) for n in "qkv")
    q = rms_unit(q.reshape(T, H, dim), eps)
    k = rms_unit(k.reshape(T, G, dim), eps)
    p = {n: w[pre + n] for n in ("temp", "r1", "r2", "sink")}
    o = attend(q, k, v.reshape(T, G, vdim), p, m["mask"]["size"], m["mask"]["keep_first"], m["scale"], m["softcap"])
    return o.reshape(T, H * vdim) @ w[pre + "o"].T


def delta_decay(h, w, pre):
    return np.exp(-math.exp(-0.5) * sigmoid(np.tanh(h @ w[pre + "w1"].T) @ w[pre + "w2"].T + w[pre + "w0"]))


def delta_scan(r, k, v, w, a, S=None):
    """Generalised delta rule, [T, H, dim] each; state S [H, key, value].  -> o [T, H, dim], S"""
    T, H, d = r.shape
    S = np.zeros((H, d, d)) if S is None else S.copy()
    o = np.zeros((T, H, d))
    for t in range(T):
        for h in range(H):
            u = k[t, h] / math.sqrt((k[t, h] ** 2).sum() + 1e-6)
            S[h] = w[t, h][:, None] * S[h] - np.outer(a[t, h] * u, u @ S[h]) + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ r[t, h]
    return o, S


def delta_mixer(h, w, pre, m, eps):
    H, d, T = m["heads"], m["dim"], h.shape[0]
    r, k, v = ((h @ w[pre + n].T).reshape(T, H, d) for n in "rkv")
    dec = delta_decay(h, w, pre).reshape(T, H, d)
    a = sigmoid(h @ w[pre + "a"].T + w[pre + "a.b"]).reshape(T, H, d)
    o, _ = delta_scan(r, k, v, dec, a)
    o = rms_unit(o, eps).reshape(T, H * d) * w[pre + "norm"]
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


MIXERS = {"attention": attention_mixer, "general_delta": delta_mixer}


def feed_forward(h, w, pre):
    return gelu_erf(h @ w[pre + "up"].T) @ w[pre + "down"].T


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence from position 0; the residual stream after every layer goes to layers_out."""
    w = {n: np.asarray(v, F) for n, v in w.items()}
    eps = cfg["norm"]["eps"]
    tokens = np.asarray(tokens)
    x = w["embed"][tokens] + w["pos"][:len(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        h = layer_norm(x, w[pre + "norm1"], w[pre + "norm1.b"], eps)
        y = MIXERS[layer["type"]](h, w, pre + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, w, pre + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


def generate(cfg, w, prompt, n_new):
    """Greedy ids (first maximum), the whole sequence recomputed for every new id.  -> ids, smallest top-2 gap seen"""
    seq, gap = list(prompt), math.inf
    for _ in range(n_new):
        z = forward(cfg, w, seq)[-1]
        top = np.sort(z)[-2:]
        gap = min(gap, float(top[1] - top[0]))
        seq.append(int(np.argmax(z)))
    return seq[len(prompt):], gap
