"""Plain numpy restatement (float64) of the Kogerax design, one function per mechanism, whole sequences only.

It shares no code with the engine. A model is a configuration dict (the content of config.json) and a dict of tensors by
name. Notation: T tokens, E width, eps the model's norm constant, rms(x) = sqrt(mean(x^2) + eps).

    block      x starts as scale * embedding row. Each sub-layer f reads x itself and only its output is normed:
               x <- x + m f(x) / rms(f(x)) (1 + w). The head reads x / rms(x) (1 + w).
    parallel   windowed attention and selective scan on the same input; half the sum of both, each over its rms times a weight
    attention  grouped heads, rotation of half-split pairs (frequencies stretched by wavelength), then unit q and k, a sliding window
    selective  convolution, silu, then per channel c and state n  S <- exp(dt_c A_cn) S + dt_c x_c B_n,  y_c = S_c . C + D_c x_c
    mlstm      S <- e^(f + m - m') S + e^(i - m') k v^T with a running maximum m' = max(f + m, i), m starting at 0
    mamba2     one decay per head: S <- e^(-e^A dt) S + dt B x^T,  y = S^T C + D x, gate, then norm in parts
    dense      gelu (tanh form) gated unit
    mixture    soft-max router over experts and identity outputs; a correction moves the choice only; chosen scores are
               normalised; clamped gated units; a shared unit behind a gate of its own
"""
import numpy as np

GATE_SLOPE = 1.702


def rms_unit(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot):
    """angle per position of every pair; with 'scaling', pairs of long wavelength turn `factor` times slower, blended in between"""
    n = rot["dims"] // 2
    f = float(rot["base"]) ** (-2.0 * np.arange(n) / rot["dims"]) if n else np.zeros(0)
    sc = rot.get("scaling")
    if sc:
        out = []
        for x in f:
            wave = 2.0 * np.pi / x
            if wave < sc["original"] / sc["high"]:
                out.append(x)
            elif wave > sc["original"] / sc["low"]:
                out.append(x / sc["factor"])
            else:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                out.append((1.0 - s) * x / sc["factor"] + s * x)
        f = np.array(out)
    return f


def rotate_half(x, rot):
    """x [T, heads, D], row t at position t: pairs (i, i + dims / 2)"""
    if not rot or not rot["dims"]:
        return x
    n = rot["dims"] // 2
    a = np.arange(x.shape[0])[:, None] * frequencies(rot)[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    out = x.copy()
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


def window_attention(h, mx, W, p, eps):
    T = h.shape[0]
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    G = mx.get("kv_heads", H)
    q = (h @ W[p + "q"].T).reshape(T, H, D)
    k = (h @ W[p + "k"].T).reshape(T, G, D)
    v = (h @ W[p + "v"].T).reshape(T, G, V)
    q, k = rms_unit(rotate_half(q, mx.get("rot")), eps), rms_unit(rotate_half(k, mx.get("rot")), eps)
    size = mx["mask"]["size"] if mx.get("mask") else T
    out = np.zeros((T, H, V))
    for t in range(T):
        lo = max(0, t - size + 1)
        for hh in range(H):
            g = hh // (H // G)
            s = k[lo:t + 1, g] @ q[t, hh] * mx["scale"]
            w = np.exp(s - s.max())
            out[t, hh] = (w / w.sum()) @ v[lo:t + 1, g]
    return out.reshape(T, H * V) @ W[p + "o"].T


def short_conv(x, w, b):
    """x [T, C], w [C, taps], last column on the current row, zeros before the start"""
    T, C = x.shape
    taps = w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, C)), x])
    return sum(pad[j:j + T] * w[:, j] for j in range(taps)) + b


def selective_scan(h, mx, W, p, eps):
    T = h.shape[0]
    n_in, N, R = mx["inner"], mx["state"], mx["dt_rank"]
    xz = h @ W[p + "in"].T
    x = silu(short_conv(xz[:, :n_in], W[p + "conv"], W[p + "conv.b"]))
    z = xz[:, n_in:]
    dbc = x @ W[p + "x"].T
    dt = softplus(dbc[:, :R] @ W[p + "dt"].T + W[p + "dt.b"])
    B, C = dbc[:, R:R + N], dbc[:, R + N:]
    A = -np.exp(W[p + "A_log"])
    S = np.zeros((n_in, N))
    y = np.zeros((T, n_in))
    for t in range(T):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + W[p + "D"] * x[t]
    return (y * silu(z)) @ W[p + "o"].T


def parallel(h, mx, W, p, eps):
    a = window_attention(h, mx["left"], W, p + "left.", eps)
    b = selective_scan(h, mx["right"], W, p + "right.", eps)
    return 0.5 * (rms_unit(a, eps) * W[p + "left.out"] + rms_unit(b, eps) * W[p + "right.out"])


def divisor(nq, m):
    return max(abs(nq), np.exp(-m)) + 1e-6


def mlstm(h, mx, W, p, eps):
    T = h.shape[0]
    H, D, V, cap = mx["heads"], mx["dim"], mx["vdim"], mx["gate_cap"]
    q = (h @ W[p + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ W[p + "k"].T).reshape(T, H, D)
    v = (h @ W[p + "v"].T).reshape(T, H, V)
    li = cap * np.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    lf = log_sigmoid(cap * np.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap))
    out = np.zeros((T, H, V))
    for hh in range(H):
        S, n, m = np.zeros((D, V)), np.zeros(D), 0.0
        for t in range(T):
            m2 = max(lf[t, hh] + m, li[t, hh])
            keep, add = np.exp(lf[t, hh] + m - m2), np.exp(li[t, hh] - m2)
            S = keep * S + add * np.outer(k[t, hh], v[t, hh])
            n = keep * n + add * k[t, hh]
            m = m2
            out[t, hh] = S.T @ q[t, hh] / divisor(n @ q[t, hh], m)
    y = rms_unit(out, eps).reshape(T, H * V) * W[p + "norm"]
    return (y * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def mamba2(h, mx, W, p, eps):
    T = h.shape[0]
    H, V, N, G = mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * V
    P = h @ W[p + "in"].T
    z, xbc, dt = P[:, :inner], P[:, inner:2 * inner + 2 * G * N], P[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x = xbc[:, :inner].reshape(T, H, V)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + W[p + "dt_bias"])
    rate = np.exp(W[p + "A_log"])
    y = np.zeros((T, H, V))
    for hh in range(H):
        g = hh // (H // G)
        S = np.zeros((N, V))
        for t in range(T):
            S = np.exp(-rate[hh] * dt[t, hh]) * S + dt[t, hh] * np.outer(B[t, g], x[t, hh])
            y[t, hh] = S.T @ C[t, g] + W[p + "D"][hh] * x[t, hh]
    y = y.reshape(T, inner) * silu(z)
    parts = mx["norm_groups"]
    y = rms_unit(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * W[p + "norm"]
    return y @ W[p + "o"].T


MIXERS = {"parallel": parallel, "mlstm": mlstm, "mamba2": mamba2}


def dense(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def clamped_unit(h, W, p, limit):
    g, u = np.minimum(h @ W[p + "gate"].T, limit), np.clip(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(GATE_SLOPE * g) * (u + 1.0)) @ W[p + "down"].T


def route(h, Wr, correction, top):
    """choices [T, top] (best first, the lower index among equals) and their normalised weights"""
    z = h @ Wr.T
    s = np.exp(z - z.max(axis=-1, keepdims=True))
    s = s / s.sum(axis=-1, keepdims=True)
    order = np.argsort(-(s + correction), axis=-1, kind="stable")[:, :top]
    w = np.take_along_axis(s, order, axis=-1)
    return order, w / (w.sum(axis=-1, keepdims=True) + 1e-20)


def mixture(h, mj, W, p):
    r = mj["router"]
    n = r["experts"]
    sel, wt = route(h, W[p + "router"], W[p + "correction"], r["top"])
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(sel[t], wt[t]):
            y[t] += w * (h[t] if e >= n else clamped_unit(h[t:t + 1], W, p + "e%d." % e, mj["expert"]["limit"])[0])
    if mj.get("shared"):
        y += sigmoid(h @ W[p + "shared.sg"].T) * clamped_unit(h, W, p + "shared.", mj["shared"]["limit"])
    return y


def feed_forward(h, mj, W, p):
    return dense(h, W, p) if mj["kind"] == "dense" else mixture(h, mj, W, p)


def forward(cfg, W, tokens):
    """logits [T, vocab] and the residual after every layer [layers, T, E]"""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    taps = []
    for i, lj in enumerate(cfg["layers"]):
        p = "l%d." % i
        x = x + m * rms_unit(MIXERS[lj["type"]](x, lj["mixer"], W, p + "mix.", eps), eps) * (1.0 + W[p + "norm1"])
        if lj.get("mlp"):
            x = x + m * rms_unit(feed_forward(x, lj["mlp"], W, p + "mlp."), eps) * (1.0 + W[p + "norm2"])
        taps.append(x)
    return (rms_unit(x, eps) * (1.0 + W["final.norm"])) @ W["head"].T, np.stack(taps)


def tensor_shapes(cfg):
    """tensor name -> shape of a model file of this design"""
    E, Vc = cfg["width"], cfg["vocab"]
    t = {"embed": [Vc, E]}
    for i, lj in enumerate(cfg["layers"]):
        p, mx = "l%d." % i, lj["mixer"]
        t[p + "norm1"] = [E]
        m = p + "mix."
        if lj["type"] == "parallel":
            a, b = mx["left"], mx["right"]
            H, G, D, V = a["heads"], a.get("kv_heads", a["heads"]), a["dim"], a["vdim"]
            t.update({m + "left.q": [H * D, E], m + "left.k": [G * D, E], m + "left.v": [G * V, E], m + "left.o": [E, H * V]})
            n, N, R, k = b["inner"], b["state"], b["dt_rank"], b["conv"]
            t.update({m + "right.in": [2 * n, E], m + "right.conv": [n, k], m + "right.conv.b": [n], m + "right.x": [R + 2 * N, n], m + "right.dt": [n, R],
                      m + "right.dt.b": [n], m + "right.A_log": [n, N], m + "right.D": [n], m + "right.o": [E, n], m + "left.out": [E], m + "right.out": [E]})
        elif lj["type"] == "mlstm":
            H, D, V = mx["heads"], mx["dim"], mx["vdim"]
            t.update({m + "q": [H * D, E], m + "k": [H * D, E], m + "v": [H * V, E], m + "g": [H * V, E], m + "o": [E, H * V], m + "norm": [H * V],
                      m + "i": [H, E], m + "i.b": [H], m + "f": [H, E], m + "f.b": [H]})
        else:
            H, V, N, G = mx["heads"], mx["vdim"], mx["state"], mx["groups"]
            C = H * V + 2 * G * N
            t.update({m + "in": [H * V + C + H, E], m + "conv": [C, mx["conv"]], m + "conv.b": [C], m + "dt_bias": [H], m + "A_log": [H], m + "D": [H],
                      m + "norm": [H * V], m + "o": [E, H * V]})
        mj, f = lj.get("mlp"), p + "mlp."
        if not mj:
            continue
        t[p + "norm2"] = [E]
        if mj["kind"] == "dense":
            t.update({f + "gate": [mj["ff"], E], f + "up": [mj["ff"], E], f + "down": [E, mj["ff"]]})
            continue
        rows = mj["router"]["experts"] + mj["router"].get("identity", 0)
        units = [("e%d." % e, mj["expert"]["ff"]) for e in range(mj["router"]["experts"])]
        if mj.get("shared"):
            units.append(("shared.", mj["shared"]["ff"]))
            t[f + "shared.sg"] = [1, E]
        for u, ff in units:
            t.update({f + u + "gate": [ff, E], f + u + "up": [ff, E], f + u + "down": [E, ff]})
        t.update({f + "router": [rows, E], f + "correction": [rows]})
    t["final.norm"] = [E]
    t["head"] = [Vc, E]
    return t


def random_model(cfg, seed=0):
    """random weights rounded to bfloat16 (what a model file holds): matrices ~ N(0, 1/in), zero-centred norm weights near 0, plain
    ones near 1, router rows spread so that the choice of experts is never a close call, decays from fast to slow"""
    import stack_oracle as so
    rng = np.random.default_rng(seed)
    W = {}
    for name, shp in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        z = rng.standard_normal(shp)
        if name == "embed":
            x = z / cfg["embedding"]["scale"]
        elif leaf in ("norm1", "norm2") or name == "final.norm":
            x = 0.2 * z
        elif leaf in ("norm", "out", "D"):
            x = 1.0 + 0.2 * z
        elif leaf == "router":
            x = z * (2.0 / np.sqrt(shp[1]))
        elif leaf == "correction":
            x = 0.15 * z
        elif leaf == "A_log":
            x = -1.5 + 1.2 * z
        elif name.endswith(".f.b"):
            x = 2.0 + z
        elif leaf == "dt_bias" or name.endswith(".dt.b"):
            x = -1.0 + z
        elif leaf == "conv":
            x = z * shp[1] ** -0.5
        elif len(shp) == 2:
            x = z / np.sqrt(shp[1])
        else:
            x = 0.3 * z
        W[name] = so.round_bf16(np.asarray(x, np.float32)).astype(np.float64).reshape(shp)
    return W


def write_model(d, cfg, W):
    import json
    import os
    import stack_oracle as so
    os.makedirs(d, exist_ok=True)
    so.save_safetensors(os.path.join(d, "model.safetensors"), {k: np.asarray(v, np.float32) for k, v in W.items()})
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    return d
