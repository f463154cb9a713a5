"""Plain numpy restatement (float64) of the Bozisun design, one function per mechanism, whole sequences only.

It shares no code with the engine. A model is a configuration dict (the content of config.json) and a dict of tensors by
name. Notation: T tokens, E width, eps the model's norm constant, unit(x) = x / sqrt(mean(x^2) + eps).

    embedding  token row plus, when the model has pairs, row (previous cp + current cc) mod buckets of a second table (the
               extra last row where a sequence has no previous token)
    layer      h = unit(x) w; x <- x + attention(h) + ff(h): one norm, both sub-layers read it. Then the token's own input of
               this layer: with e its slice of a per-token table, y = proj(gelu(gate x) e), x <- x + unit(y) w'
    attention  grouped heads, every earlier position; queries and keys normed per head (weight shared by the heads), then part of
               a head rotated (half-split pairs, YaRN: slow pairs turn slower, and all rotated entries grow by one factor);
               the concatenated heads are gated entry by entry from h
    dense      silu gated unit
    mixture    the largest router logits (with a bias) choose; their soft-max among themselves weighs
    span       a run of layers is passed several times with the same weights
    head       logits capped softly
"""
import numpy as np


def unit(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def pair_rows(tokens, pc):
    """row of the pair table for every token: hashed from the token before it and the token, the extra row at the start"""
    rows = [pc["buckets"]]
    for a, b in zip(tokens[:-1], tokens[1:]):
        rows.append((int(a) * pc["mul_prev"] + int(b) * pc["mul_cur"]) % pc["buckets"])
    return np.array(rows)


def embed(cfg, W, tokens):
    x = W["embed"][np.asarray(tokens)]
    pc = (cfg.get("embedding") or {}).get("bigram")
    if pc:
        x = x + W["bigram"][pair_rows(tokens, pc)]
    return x


def yarn_bounds(rot):
    """pair indices between which frequencies are blended"""
    sc, d = rot["scaling"], rot["dims"]

    def index(turns):
        return d * np.log(sc["original"] / (2.0 * np.pi * turns)) / (2.0 * np.log(rot["base"]))
    return max(np.floor(index(sc["fast"])), 0.0), min(np.ceil(index(sc["slow"])), d - 1.0)


def frequencies(rot):
    """angle per position of every pair, and the factor on the rotated entries"""
    n = rot["dims"] // 2
    i = np.arange(n)
    f = float(rot["base"]) ** (-2.0 * i / rot["dims"]) if n else np.zeros(0)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    lo, hi = yarn_bounds(rot)
    slow = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f * (slow / sc["factor"] + 1.0 - slow), 0.1 * np.log(sc["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, D], row t at position t"""
    if not rot or not rot["dims"]:
        return x
    n = rot["dims"] // 2
    f, mag = frequencies(rot)
    a = np.arange(x.shape[0])[:, None] * f[None, :]
    c, s = mag * np.cos(a)[:, None, :], mag * np.sin(a)[:, None, :]
    out = x.copy()
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


def queries_keys(h, mx, W, p, eps):
    T, H, G, D = h.shape[0], mx["heads"], mx.get("kv_heads", mx["heads"]), mx["dim"]
    q = unit((h @ W[p + "q"].T).reshape(T, H, D), eps) * W[p + "q.norm"]
    k = unit((h @ W[p + "k"].T).reshape(T, G, D), eps) * W[p + "k.norm"]
    return rotate(q, mx.get("rot")), rotate(k, mx.get("rot"))


def attention(h, mx, W, p, eps):
    T = h.shape[0]
    H, V = mx["heads"], mx["vdim"]
    G = mx.get("kv_heads", H)
    q, k = queries_keys(h, mx, W, p, eps)
    v = (h @ W[p + "v"].T).reshape(T, G, V)
    out = np.zeros((T, H, V))
    seen = np.tril(np.ones((T, T), bool))
    for hh in range(H):
        g = hh // (H // G)
        out[:, hh] = softmax(np.where(seen, q[:, hh] @ k[:, g].T * mx["scale"], -np.inf)) @ v[:, g]
    return (out.reshape(T, H * V) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def gated(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, Wr, bias, top):
    """choices [T, top] (best first, the lower index among equals) and their weights"""
    z = h @ Wr.T + bias
    sel = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    return sel, softmax(np.take_along_axis(z, sel, axis=-1))


def mixture(h, mj, W, p):
    sel, wt = route(h, W[p + "router"], W[p + "router.b"], mj["router"]["top"])
    y = np.zeros_like(h)
    for e in range(mj["router"]["experts"]):
        t, k = np.nonzero(sel == e)
        if len(t):
            y[t] += wt[t, k][:, None] * gated(h[t], W, p + "e%d." % e)
    return y


def feed_forward(h, mj, W, p):
    return gated(h, W, p) if mj["kind"] == "dense" else mixture(h, mj, W, p)


def side(x, e, W, p, eps):
    """what the token's own input of this layer adds"""
    y = (gelu_tanh(x @ W[p + "gate"].T) * e) @ W[p + "proj"].T
    return unit(y, eps) * W[p + "norm"]


def run_order(cfg):
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


def forward(cfg, W, tokens):
    """logits [T, vocab] and the residual after every layer run [runs, T, E]"""
    W = {k: np.asarray(v, dtype=np.float64) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    dim = (cfg.get("token_side") or {}).get("dim", 0)
    x = embed(cfg, W, tokens)
    taps = []
    for i in run_order(cfg):
        lj, p = cfg["layers"][i], "l%d." % i
        h = unit(x, eps) * W[p + "norm1"]
        y = attention(h, lj["mixer"], W, p + "mix.", eps)
        if lj.get("mlp"):
            y = y + feed_forward(h, lj["mlp"], W, p + "mlp.")
        x = x + y
        if dim:
            x = x + side(x, W["side.embed"][np.asarray(tokens), i * dim:(i + 1) * dim], W, p + "side.", eps)
        taps.append(x)
    return soft_cap((unit(x, eps) * W["final.norm"]) @ W["head"].T, cfg.get("logit_softcap", 0.0)), np.stack(taps)


def tensor_shapes(cfg):
    """tensor name -> shape of a model file of this design"""
    E, Vc, n = cfg["width"], cfg["vocab"], len(cfg["layers"])
    t = {"embed": [Vc, E]}
    pc, ts = (cfg.get("embedding") or {}).get("bigram"), cfg.get("token_side")
    if pc:
        t["bigram"] = [pc["buckets"] + 1, E]
    if ts:
        t["side.embed"] = [Vc, n * ts["dim"]]
    for i, lj in enumerate(cfg["layers"]):
        p, mx = "l%d." % i, lj["mixer"]
        m = p + "mix."
        H, D, V = mx["heads"], mx["dim"], mx["vdim"]
        G = mx.get("kv_heads", H)
        t.update({p + "norm1": [E], m + "q": [H * D, E], m + "k": [G * D, E], m + "v": [G * V, E], m + "q.norm": [D], m + "k.norm": [D], m + "g": [H * V, E], m + "o": [E, H * V]})
        mj, f = lj.get("mlp"), p + "mlp."
        if mj:
            units = [("", mj["ff"])] if mj["kind"] == "dense" else [("e%d." % e, mj["expert"]["ff"]) for e in range(mj["router"]["experts"])]
            for u, ff in units:
                t.update({f + u + "gate": [ff, E], f + u + "up": [ff, E], f + u + "down": [E, ff]})
            if mj["kind"] == "moe":
                t.update({f + "router": [mj["router"]["experts"], E], f + "router.b": [mj["router"]["experts"]]})
        if ts:
            t.update({p + "side.gate": [ts["dim"], E], p + "side.proj": [E, ts["dim"]], p + "side.norm": [E]})
    t.update({"final.norm": [E], "head": [Vc, E]})
    return t


def random_model(cfg, seed=0):
    """random weights rounded to bfloat16 (what a model file holds): matrices ~ N(0, 1/in), norm weights near 1, router rows spread so
    that the choice of experts is rarely a close call"""
    import stack_oracle as so
    rng = np.random.default_rng(seed)
    W = {}
    for name, shp in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        z = rng.standard_normal(shp)
        if name == "embed":
            x = z
        elif name == "bigram":
            x = 0.7 * z
        elif name == "side.embed":
            x = z
        elif leaf in ("norm", "norm1"):
            x = 1.0 + 0.2 * z
        elif leaf == "router":
            x = z * (2.0 / np.sqrt(shp[1]))
        elif leaf == "b":
            x = z
        else:
            x = z / np.sqrt(shp[1])
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
