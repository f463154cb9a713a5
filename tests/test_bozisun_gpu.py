"""The Bozisun design on the GPU against the plain numpy restatement in tests/bozisun_oracle.py: every mechanism alone (with the
residual after the layer), whole prompts against token-by-token decoding and portions down to two tokens, contexts that are cleared
and used again, several live contexts stepping in turn, who notices a changed token (through the pair table, the token inputs and
the attention), far keys that stand out, the first tokens of a sequence, repeated spans with a cache per pass, long decoding through
the replayed graph, other sizes (scalar and vector load paths, rows beyond the one-launch layer end, grouped and ungrouped heads,
every band of the frequency scaling, parts of the design left out, values that are 1), bfloat16, greedy generation through the
bridge's job loop and the trace runner. Small random models in a temporary folder; float32 is the sharp comparison."""
import copy

import numpy as np
import pytest

import bozisun_oracle as bo
import stack_oracle as so
from booster_b200 import _lib, engine

pytestmark = pytest.mark.gpu

TOL32 = 2e-4


def err(got, want):
    """root mean square of the difference with its mean taken off, over the root mean square of the expected row; worst row"""
    return float(row_errs(got, want).max())


def row_errs(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / (np.sqrt((w * w).mean(-1)) + 1e-30)


def dense(ff=20):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=20):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def att(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.4, rot=4, base=100.0, scaling=(4.0, 2.0, 0.25, 64), mlp=None):
    mx = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        mx["rot"] = {"base": base, "dims": rot}
        if scaling:
            mx["rot"]["scaling"] = dict(zip(("factor", "fast", "slow", "original"), scaling))
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def config(layers, width=48, vocab=61, eps=1e-5, pairs=(37, 11, 5), side=10, loop=None, cap=9.0):
    cfg = {"architecture": "Bozisun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if pairs:
        cfg["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))}
    if side:
        cfg["token_side"] = {"dim": side}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if cap:
        cfg["logit_softcap"] = cap
    return cfg


class Pair:
    """the same random model in the framework and in the oracle"""

    def __init__(self, tmp_path, cfg, seed=0, dtype="float32", n_ctx=512, edit=None):
        self.cfg = cfg
        self.w = bo.random_model(cfg, seed)
        if edit:
            edit(self.w)
        self.dir = bo.write_model(str(tmp_path / f"b{seed}_{dtype}_{abs(hash(str(cfg))) % 10**8}"), cfg, self.w)
        self.model = engine.Model(self.dir, dtype=dtype)
        self.ctx = engine.Context(self.model, n_ctx)

    def close(self):
        self.ctx.close()
        self.model.close()

    def tokens(self, n, seed=1):
        return np.random.default_rng(seed).integers(0, self.cfg["vocab"], size=n).tolist()

    def expected(self, toks, cfg=None, w=None, residuals=False):
        lg, taps = bo.forward(cfg or self.cfg, w or self.w, toks)
        return (lg, taps) if residuals else lg

    def run(self, toks, cuts=None, ctx=None):
        """logits of every position, the token stream cut into steps of the given sizes (None: one step)"""
        ctx = ctx or self.ctx
        ctx.kv_clear()
        out, pos, i = [], 0, 0
        cuts = list(cuts) if cuts else [len(toks)]
        while pos < len(toks):
            n = min(cuts[i % len(cuts)], len(toks) - pos)
            out.append(ctx.decode_rows(toks[pos:pos + n], pos, list(range(n))))
            pos += n
            i += 1
        return np.concatenate(out)


def bf16(x):
    return so.round_bf16(np.asarray(x, np.float32)).astype(np.float64)


ALL_CUTS = ([1], [2], [3], [4], [5], [6, 7], [8, 9], [5, 1, 9, 2])
PLAIN = dict(pairs=None, side=0, cap=0.0)
ALONE = {"attention": config([att()], **PLAIN), "attention-ungrouped-unscaled": config([att(heads=3, kv_heads=3, dim=5, vdim=7, rot=4, scaling=None)], **PLAIN),
         "attention-one-key-head-unrotated": config([att(heads=6, kv_heads=1, dim=12, vdim=16, rot=0)], **PLAIN), "attention-whole-head-rotated": config([att(heads=2, kv_heads=2, dim=16, vdim=1, rot=16)], **PLAIN),
         "dense": config([att(mlp=dense())], **PLAIN), "mixture": config([att(mlp=moe())], **PLAIN), "mixture-of-one": config([att(mlp=moe(experts=1, top=1, ff=9))], **PLAIN),
         "mixture-all-chosen": config([att(mlp=moe(experts=5, top=5))], **PLAIN), "mixture-of-many": config([att(mlp=moe(experts=70, top=40, ff=4))], **PLAIN),
         "pairs": config([att()], pairs=(7, 3, 2), side=0, cap=0.0), "one-bucket": config([att()], pairs=(1, 1, 1), side=0, cap=0.0), "token-input": config([att()], pairs=None, side=16, cap=0.0),
         "token-input-of-one+dense": config([att(mlp=dense(9))], pairs=None, side=1, cap=0.0), "cap": config([att(mlp=dense())], pairs=None, side=0, cap=2.0),
         "span": config([att(mlp=dense())], pairs=None, side=0, cap=0.0, loop=(0, 1, 3)), "everything": config([att(mlp=moe())], loop=(0, 1, 2))}


@pytest.mark.parametrize("name", list(ALONE))
def test_each_mechanism_alone_with_the_residual_after_the_layer(tmp_path, name):
    cfg = ALONE[name]
    p = Pair(tmp_path, cfg)
    toks = p.tokens(29)
    want, res = p.expected(toks, residuals=True)
    p.ctx.set_taps(True)
    got = p.ctx.decode_rows(toks, 0, list(range(len(toks))))
    taps = p.ctx.layer_taps(len(toks))
    p.ctx.kv_clear()
    one = []
    for i in range(5):                                    # and through the steps of one token
        p.ctx.decode_rows(toks[i:i + 1], i, [0])
        one.append(p.ctx.layer_taps(1))
    p.ctx.set_taps(False)
    assert taps.shape[0] == len(bo.run_order(cfg))
    for a, b, c in zip(taps, res, np.concatenate(one, 1)):
        assert np.abs(a - b).max() < 1e-4 * max(1.0, np.abs(b).max()) and np.abs(c - b[:5]).max() < 1e-4 * max(1.0, np.abs(b).max())
    assert err(got, want) < TOL32
    for cuts in ALL_CUTS:
        assert err(p.run(toks, cuts), want) < TOL32, cuts
    p.close()


FULL = [att(mlp=dense()), att(heads=6, kv_heads=3, dim=12, vdim=8, rot=6, mlp=moe()), att(heads=2, kv_heads=1, dim=16, vdim=12, rot=16, base=500.0, scaling=(8.0, 4.0, 0.5, 40)),
        att(heads=3, kv_heads=3, dim=10, vdim=20, rot=10, scaling=None, mlp=moe(experts=5, top=3, ff=16)), att(rot=0, mlp=dense(33))]


def full(**kw):
    kw.setdefault("loop", (1, 4, 2))
    return config(FULL, **kw)


def test_small_mechanisms_matter(tmp_path):
    """the oracle without one of the small mechanisms is far from the framework: none of them is a no-op in these models"""
    cfg = config([att(heads=4, scale=1.0, rot=8, mlp=moe()), att(mlp=dense())], loop=(0, 1, 2))
    p = Pair(tmp_path, cfg)
    toks = p.tokens(61)
    got = p.run(toks)
    assert err(got, p.expected(toks)) < TOL32
    for key in ("bigram", "side.embed", "l0.norm1", "l0.mix.q", "l0.mix.g", "l0.mlp.router", "l0.mlp.router.b", "l0.side.gate", "l0.side.norm", "l1.side.proj", "l1.mix.g"):
        w2 = dict(p.w); w2[key] = np.zeros_like(p.w[key])
        assert err(got, p.expected(toks, w=w2)) > 20 * TOL32, key
    for key in ("l0.norm1", "l1.norm1", "final.norm", "l0.mix.q.norm", "l0.mix.k.norm", "l1.side.norm"):
        w2 = dict(p.w); w2[key] = p.w[key] * np.linspace(0.5, 1.5, p.w[key].size).reshape(p.w[key].shape)
        assert err(got, p.expected(toks, w=w2)) > 20 * TOL32, key
    mix = lambda c: c["layers"][0]["mixer"]
    for edit in (lambda c: mix(c)["rot"].update(base=50.0), lambda c: mix(c)["rot"].update(dims=6), lambda c: mix(c)["rot"].pop("scaling"), lambda c: mix(c)["rot"]["scaling"].update(factor=3.0),
                 lambda c: mix(c)["rot"]["scaling"].update(fast=0.5), lambda c: mix(c)["rot"]["scaling"].update(slow=2.0), lambda c: mix(c)["rot"]["scaling"].update(original=6), lambda c: mix(c).update(scale=0.9),
                 lambda c: c["layers"][0]["mlp"]["router"].update(top=3), lambda c: c["norm"].update(eps=1e-1), lambda c: c.update(logit_softcap=7.0), lambda c: c.update(logit_softcap=0.0),
                 lambda c: c["loop"].update(times=1), lambda c: c["loop"].update(stop=2), lambda c: c["embedding"]["bigram"].update(mul_prev=5, mul_cur=11), lambda c: c["embedding"].pop("bigram")):
        c2 = copy.deepcopy(cfg); edit(c2)
        assert err(got, p.expected(toks, cfg=c2)) > 20 * TOL32, c2
    # and one function at a time, restated wrongly on purpose
    keep = {n: getattr(bo, n) for n in ("gelu_tanh", "silu", "sigmoid", "frequencies", "pair_rows", "route", "side")}

    def weights_over_all(h, Wr, bias, top):
        sel, _ = keep["route"](h, Wr, bias, top)
        return sel, np.take_along_axis(bo.softmax(h @ Wr.T + bias), sel, -1)

    def choice_without_bias(h, Wr, bias, top):
        sel, _ = keep["route"](h, Wr, 0 * bias, top)
        return sel, bo.softmax(np.take_along_axis(h @ Wr.T + bias, sel, -1))
    for name, f in (("gelu_tanh", bo.silu), ("silu", bo.gelu_tanh), ("sigmoid", lambda z: 1.0 / (1.0 + np.exp(-1.2 * z))), ("frequencies", lambda r: (keep["frequencies"](r)[0], 1.0)), ("route", weights_over_all), ("route", choice_without_bias),
                    ("pair_rows", lambda t, pc: np.concatenate([[0], keep["pair_rows"](t, pc)[1:]])), ("side", lambda x, e, W, q, eps: keep["side"](bo.unit(x, eps), e, W, q, eps))):
        setattr(bo, name, f)
        try:
            assert err(got, p.expected(toks)) > 20 * TOL32, name
        finally:
            setattr(bo, name, keep[name])
    p.close()


def test_whole_prompt_token_by_token_and_portions_agree(tmp_path):
    p = Pair(tmp_path, full())
    toks = p.tokens(75)
    want, res = p.expected(toks, residuals=True)
    p.ctx.set_taps(True)
    p.ctx.decode_rows(toks, 0, [])
    taps = p.ctx.layer_taps(len(toks))
    p.ctx.set_taps(False)
    assert taps.shape[0] == len(res) == len(FULL) + 3
    for a, b in zip(taps, res):
        assert np.abs(a - b).max() < 1e-4 * max(1.0, np.abs(b).max())
    assert err(p.run(toks), want) < TOL32
    for cuts in ALL_CUTS + ([3, 2, 7, 1, 5], [37, 2, 2, 30], [6, 1, 1, 11], [17, 16, 15], [1, 2]):      # [1]: every token through the replayed one-token graph
        assert err(p.run(toks, cuts), want) < TOL32, cuts
    p.close()


def test_cleared_context_is_as_good_as_new_and_contexts_do_not_meet(tmp_path):
    p = Pair(tmp_path, full())
    a, b = p.tokens(60, seed=3), p.tokens(29, seed=4)
    fresh = engine.Context(p.model, 512)
    ref_b = p.run(b, [5, 1, 1, 9], ctx=fresh)
    p.run(a, [7, 1])                                  # fills cache rows; its last token must not pair with the next sequence's first
    again = p.run(b, [5, 1, 1, 9])                    # run() clears first: the same context, used again
    assert np.array_equal(again, ref_b)
    assert err(again, p.expected(b)) < TOL32
    # two live sequences of unequal length stepping in turn, each as if alone
    p.ctx.kv_clear(); fresh.kv_clear()
    ga, gb, pa, pb = [], [], 0, 0
    for na, nb in ((9, 3), (1, 1), (4, 13), (1, 2), (45, 10)):
        ga.append(p.ctx.decode_rows(a[pa:pa + na], pa, list(range(na)))); pa += na
        gb.append(fresh.decode_rows(b[pb:pb + nb], pb, list(range(nb)))); pb += nb
    assert err(np.concatenate(ga), p.expected(a)) < TOL32
    assert err(np.concatenate(gb), p.expected(b)) < TOL32
    fresh.close()
    p.close()


@pytest.mark.parametrize("path", ["pairs", "token-input", "attention"])
def test_who_notices_a_changed_token(tmp_path, path):
    """which positions change when token j does: itself (its own inputs), itself and the next one (the pair table; also where a portion
    or a one-token step begins), itself and every later one (the attention)"""
    cfg = config([att(mlp=dense()), att(heads=2, kv_heads=2, mlp=moe(top=1))], width=32, vocab=40, pairs=(211, 40, 1) if path == "pairs" else None)

    def edit(w):
        if path != "attention":
            for i in range(2):
                w["l%d.mix.o" % i] = np.zeros_like(w["l%d.mix.o" % i])
    p = Pair(tmp_path, cfg, seed=2, edit=edit)
    n = 70
    toks = p.tokens(n, seed=5)
    for cuts in (None, [40, 1], [2, 3, 5, 1, 7, 11]):
        base = p.run(toks, cuts)
        for j in (0, 3, 9, 39, 44, 69):
            other = list(toks); other[j] = (toks[j] + 1) % 40
            got = p.run(other, cuts)
            for q in range(n):
                changes = q == j or (path == "pairs" and q == j + 1) or (path == "attention" and q > j)
                assert np.array_equal(got[q], base[q]) != changes, (cuts, j, q)
    assert err(p.run(toks), p.expected(toks)) < TOL32
    p.close()


def test_pair_rows(tmp_path):
    """the first token's extra row, rows that differ in the order of a pair, multipliers whose products need more than 32 bits"""
    for pc in ((50, 3, 7), (509, 1 << 29, (1 << 29) + 12345), (1021, 4294967291, 2654435761), (3, 0, 1), (64, 1, 0)):
        cfg = config([att(mlp=dense())], width=32, vocab=2000, pairs=pc, side=0)
        p = Pair(tmp_path, cfg, seed=pc[0], n_ctx=64)
        toks = p.tokens(40, seed=pc[0])
        toks[5:9] = [1999, 1998, 1999, 0]
        want = p.expected(toks)
        for cuts in (None, [1], [2], [7, 1]):
            assert err(p.run(toks, cuts), want) < TOL32, (pc, cuts)
        w2 = dict(p.w); w2["bigram"] = p.w["bigram"].copy(); w2["bigram"][pc[0]] = 0.0
        assert row_errs(p.expected(toks, w=w2), want)[0] > 20 * TOL32
        p.close()


def test_far_keys_stand_out(tmp_path):
    """one odd token among alike ones draws every later query: the logits 300 positions on rest on it, in prompts, in decoding and with
    portions that start anywhere; an oracle that loses the key is far away"""
    cfg = config([att(heads=4, kv_heads=2, dim=16, vdim=8, rot=4, scale=1.5, mlp=dense())], width=32, vocab=40, pairs=None)

    def edit(w):
        e = w["embed"].copy()
        e[:39] = e[0] + 0.3 * e[:39]
        w["embed"] = bf16(e)
        alike, odd = e[0] * w["l0.norm1"], e[39] * w["l0.norm1"]
        k = w["l0.mix.k"]
        for g in range(2):                                # the odd token's key points where the alike tokens' queries do
            q = w["l0.mix.q"][32 * g:32 * g + 16] @ alike
            rows = slice(16 * g, 16 * g + 16)
            k[rows] = 0.3 * k[rows] + np.outer(q / np.linalg.norm(q), odd / np.linalg.norm(odd))
            w["l0.mix.q"][32 * g + 16:32 * g + 32] = w["l0.mix.q"][32 * g:32 * g + 16]
        w["l0.mix.k"] = bf16(k); w["l0.mix.v"] = bf16(2.0 * w["l0.mix.v"])
    p = Pair(tmp_path, cfg, seed=6, n_ctx=400, edit=edit)
    plain = np.random.default_rng(9).integers(0, 39, size=340).tolist()
    for at in (0, 3, 15, 16, 127, 128):
        odd = list(plain); odd[at] = 39
        want, base = p.expected(odd), p.expected(plain)
        late = row_errs(base, want)[300:]
        assert np.median(late) > 50 * TOL32
        for cuts in (None, [300, 1], [2, 129, 3, 64], [1, 150, 1, 150]):
            assert err(p.run(odd, cuts), want) < TOL32, (at, cuts)
    assert err(p.run(odd[:40], [1]), want[:40]) < TOL32          # the first tokens of a sequence
    p.close()


@pytest.mark.parametrize("shape", [(1, 16, 8), (2, 64, 64), (3, 128, 128), (4, 132, 20), (5, 8, 256), (6, 256, 128), (8, 32, 128), (9, 64, 4), (17, 4, 4)], ids=str)
def test_few_token_attention_over_many_slices(tmp_path, shape):
    """queries per key head below, at and beyond what a block takes together, one or two 16-byte chunks per lane, several strips per warp
    and several blocks per head: single tokens and short portions far into a sequence"""
    R, dim, vdim = shape
    cfg = config([att(heads=2 * R, kv_heads=2, dim=dim, vdim=vdim, rot=4, scale=1.5 / np.sqrt(dim)), att(heads=R, kv_heads=1, dim=dim, vdim=vdim, rot=4, scale=4.0 / np.sqrt(dim))], width=32, vocab=40)
    p = Pair(tmp_path, cfg, seed=R, n_ctx=2048)
    toks = p.tokens(700, seed=R)
    want = p.expected(toks)
    for cuts in ([661] + [1] * 39, [655, 7, 6, 5, 4, 3, 2, 1, 7, 7]):
        got = p.run(toks, cuts)
        assert err(got, want) < 2 * TOL32, cuts
    assert err(p.run(toks[:120], [1, 2, 3, 4, 5, 6, 7]), want[:120]) < TOL32      # from the first token on
    p.close()


def test_steep_scores_and_angles(tmp_path):
    """peaked attention: positions one off, or another factor on the rotated entries, are far away"""
    cfg = config([att(heads=4, kv_heads=1, dim=8, rot=8, scale=3.0, mlp=dense())], width=32, vocab=40)
    p = Pair(tmp_path, cfg, seed=3)
    toks = p.tokens(150, seed=3)
    want = p.expected(toks)
    keep = bo.rotate
    bo.rotate = lambda x, rot: keep(np.concatenate([x[:1], x]), rot)[1:] if x.shape[1] == 4 else keep(x, rot)      # queries one position on
    try:
        assert err(p.expected(toks), want) > 50 * TOL32
    finally:
        bo.rotate = keep
    for cuts in (None, [110, 1], [7, 2], [31, 1, 33, 2]):
        assert err(p.run(toks, cuts), want) < TOL32, cuts
    p.close()


def test_frequency_bands(tmp_path):
    """frequencies kept, blended and slowed all occur; a blend that ends at the last pair, one of no width, one cut at the first pair"""
    bands = [(1000.0, 16, (6.0, 8.0, 1.0, 60)), (1000.0, 16, (6.0, 3.0, 3.0, 60)), (50.0, 16, (2.5, 1.0, 0.001, 60)), (10000.0, 18, (16.0, 400.0, 1.0, 300)), (1000.0, 2, (4.0, 32.0, 1.0, 512))]
    for seed, (base, dims, sc) in enumerate(bands):
        rot = {"base": base, "dims": dims, "scaling": dict(zip(("factor", "fast", "slow", "original"), sc))}
        if seed == 0:
            f, g = bo.frequencies({"base": base, "dims": dims})[0], bo.frequencies(rot)[0]
            kept, slowed = np.isclose(g, f), np.isclose(g, f / 6.0)
            assert kept.any() and slowed.any() and not (kept | slowed).all()
        L = att(heads=2, kv_heads=2, dim=18, vdim=8, scale=1.0, rot=0)
        L["mixer"]["rot"] = rot
        p = Pair(tmp_path, config([L], pairs=None), seed=seed)
        toks = p.tokens(120)
        want = p.expected(toks)
        for cuts in (None, [100, 1], [3, 14]):
            assert err(p.run(toks, cuts), want) < TOL32, (seed, cuts)
        p.close()


def test_router_choices(tmp_path):
    """logits far apart (weights of exactly one and zero), the bias alone deciding, every expert chosen"""
    for seed, (top, gain, shift) in enumerate([(2, 60.0, 0.0), (3, 0.0, 4.0), (1, 1.0, 0.0), (6, 3.0, 1.0)]):
        cfg = config([att(mlp=moe(experts=6, top=top))])

        def edit(w):
            w["l0.mlp.router"] = bf16(gain * w["l0.mlp.router"]); w["l0.mlp.router.b"] = bf16(w["l0.mlp.router.b"] + shift * np.arange(6) - 100.0)
        p = Pair(tmp_path, cfg, seed=seed, edit=edit)
        toks = p.tokens(40)
        want = p.expected(toks)
        for cuts in (None, [1], [3], [7, 2]):
            assert err(p.run(toks, cuts), want) < TOL32, (top, gain, cuts)
        p.close()


@pytest.mark.parametrize("loop", [None, (0, 5, 2), (0, 1, 4), (4, 5, 3), (2, 2, 5), (1, 3, 1)], ids=str)
def test_repeated_spans(tmp_path, loop):
    """each pass of a span keeps keys and values of its own; the same slice of the token's inputs serves every pass"""
    p = Pair(tmp_path, full(loop=loop))
    toks = p.tokens(50)
    want = p.expected(toks)
    for cuts in (None, [30, 1], [2, 9]):
        assert err(p.run(toks, cuts), want) < TOL32, cuts
    p.close()


def test_long_decoding_through_the_graph(tmp_path):
    p = Pair(tmp_path, full())
    toks = p.tokens(400, seed=11)
    want = p.expected(toks)
    got = p.run(toks, [4] + [1] * 400)
    assert err(got, want) < 2 * TOL32
    p.close()


@pytest.mark.parametrize("width,vocab", [(36, 50), (40, 77), (64, 130), (37, 53)], ids=["scalar-loads", "width-40", "vector-loads", "odd-width"])
@pytest.mark.parametrize("side", [1, 12, 40])
def test_other_sizes(tmp_path, width, vocab, side):
    layers = [att(heads=6, kv_heads=2, dim=9, vdim=5, rot=2, mlp=moe(experts=3, top=3, ff=7)), att(heads=4, kv_heads=4, dim=16, vdim=40, rot=6, mlp=moe(experts=16, top=4, ff=64)),
              att(heads=1, kv_heads=1, dim=4, vdim=4, rot=4), att(heads=8, kv_heads=1, dim=64, vdim=5, rot=64, mlp=dense(1)), att(heads=2, kv_heads=1, dim=1, vdim=1, rot=0, mlp=moe(experts=1, top=1, ff=24)),
              att(heads=3, kv_heads=1, dim=130, vdim=200, rot=30, scale=0.1, mlp=dense(130)), att(heads=1, kv_heads=1, dim=300, vdim=256, rot=300, scale=0.05)]
    p = Pair(tmp_path, config(layers, width=width, vocab=vocab, eps=1e-6, side=side, loop=(1, 3, 2)), seed=width)
    toks = p.tokens(70, seed=width)
    want = p.expected(toks)
    assert err(p.run(toks), want) < TOL32
    assert err(p.run(toks, [13, 2, 1]), want) < TOL32
    p.close()


def test_wide_rows(tmp_path):
    """rows longer than what the joins keep in registers, and longer than what the one-launch layer end takes"""
    for width, side in ((2500, 24), (1031, 7), (10300, 8), (4104, 0)):
        layers = [att(heads=2, kv_heads=1, mlp=moe(experts=2, top=2, ff=8)), att(mlp=dense(8))]
        p = Pair(tmp_path, config(layers, width=width, vocab=40, side=side), seed=1, n_ctx=160)
        toks = p.tokens(60, seed=1)
        want = p.expected(toks)
        assert err(p.run(toks), want) < TOL32
        assert err(p.run(toks[:30], [20, 1, 1, 3]), want[:30]) < TOL32
        p.close()


def random_config(rng):
    """a random arrangement of layers with random sizes: nothing may rest on one model's values"""
    pick = lambda values: int(rng.choice(values))

    def ff():
        u = rng.random()
        if u < 0.2:
            return None
        if u < 0.5:
            return dense(pick([8, 30, 64, 136]))
        n = pick([1, 2, 5, 8, 12])
        return moe(experts=n, top=pick(range(1, min(n, 5) + 1)), ff=pick([8, 24, 64, 100]))
    layers = []
    for _ in range(pick([1, 2, 3, 4, 6])):
        kv, d = pick([1, 2, 3]), pick([4, 6, 16, 32, 64, 128])
        rot = pick([r for r in (0, 2, 4, 16, 32, 64, 128) if r <= d])
        layers.append(att(heads=kv * pick([1, 2, 4, 5]), kv_heads=kv, dim=d, vdim=pick([4, 8, 48, 128, 200]), scale=float(rng.choice([0.1, 0.3])), rot=rot, base=float(rng.choice([100.0, 1e4, 5e5])),
                          scaling=None if rng.random() < 0.3 else (float(rng.choice([2.0, 8.0, 40.0])), 32.0, 1.0, pick([64, 512, 4096])), mlp=ff()))
    n = len(layers)
    a = pick(range(n))
    loop = None if rng.random() < 0.3 else (a, pick(range(a, n)) + 1, pick([1, 2, 3]))
    return config(layers, width=pick([24, 36, 64, 100, 136]), vocab=pick([37, 100, 257, 513]), eps=float(rng.choice([1e-6, 1e-5])), loop=loop, cap=float(rng.choice([0.0, 5.0, 30.0])),
                  pairs=None if rng.random() < 0.2 else (pick([1, 64, 1021]), pick([1, 13, 513]), pick([1, 9, 257])), side=pick([0, 4, 8, 17, 64]))


@pytest.mark.parametrize("seed", range(12))
def test_random_configurations(tmp_path, seed):
    rng = np.random.default_rng(900 + seed)
    cfg = random_config(rng)
    n = int(rng.choice([70, 150, 330]))
    p = Pair(tmp_path, cfg, seed=seed, n_ctx=n + 4)
    toks = p.tokens(n, seed=seed)
    want = p.expected(toks)
    assert err(p.run(toks), want) < 2 * TOL32, cfg
    assert err(p.run(toks, [n - 20] + [1] * 20), want) < 2 * TOL32, cfg
    assert err(p.run(toks, [2, 67, 3, 129, 1, 5]), want) < 2 * TOL32, cfg
    p.close()


def test_a_step_longer_than_one_pass(tmp_path):
    """a 1100-token step runs as several passes of the layers: cached keys and the previous token cross the passes' edges"""
    p = Pair(tmp_path, full(), n_ctx=1104)
    toks = p.tokens(1100, seed=5)
    want = p.expected(toks)
    assert err(p.run(toks), want) < 2 * TOL32
    assert err(p.run(toks, [509, 2, 3, 586]), want) < 2 * TOL32
    p.close()


def test_bfloat16_prompt_kernels_and_decode(tmp_path):
    """wide enough for the tensor-core products, also the segmented ones of the routed mixture and both of the token inputs"""
    layers = [att(heads=4, kv_heads=2, dim=32, vdim=32, rot=16, mlp=dense(256)), att(heads=8, kv_heads=1, dim=32, vdim=16, rot=32, mlp=moe(experts=4, top=2, ff=64)),
              att(heads=2, kv_heads=2, dim=64, vdim=64, rot=0, mlp=moe(experts=3, top=2, ff=128))]
    cfg = config(layers, width=128, vocab=160, side=128, loop=(0, 2, 2))
    p = Pair(tmp_path, cfg, dtype="bfloat16")
    toks = p.tokens(300, seed=2)
    keep, gaps = bo.route, []

    def watched(h, Wr, bias, top):                     # how close the choice of experts is, position by position
        c = np.sort(h @ Wr.T + bias, axis=-1)
        gaps.append(c[:, -top] - c[:, -top - 1])
        return keep(h, Wr, bias, top)
    bo.route = watched
    try:
        want = p.expected(toks)
    finally:
        bo.route = keep
    clear = np.min(gaps, axis=0) > 0.1
    assert clear.mean() > 0.3
    # token by token: mat-vec kernels with float32 activations on the stored bfloat16 weights: as sharp as float32
    assert err(p.run(toks[:60], [1]), want[:60]) < TOL32
    assert err(p.run(toks[:60], [3, 4, 2]), want[:60]) < TOL32
    # longer portions: tensor-core products round the activation operand to bfloat16
    for cuts in (None, [280, 1], [5, 17, 133]):
        e = row_errs(p.run(toks, cuts), want)
        # where rounding cannot change the choice of an expert
        assert np.median(e) < 3e-2 and np.median(e[clear]) < 2e-2 and np.quantile(e[clear], 0.9) < 0.1, (cuts, float(np.median(e)), np.sort(e[clear])[-9:])
    p.close()


def test_greedy_generation_through_the_bridge(tmp_path, monkeypatch):
    """initContext / doInference on a folder model: decimal-id prompt, standard chain at temperature 0 (arg-max on the device),
    prompt through the prompt kernels, generation through the one-token graph: the ids the oracle generates greedily"""
    monkeypatch.setenv("BOOSTER_B200_DTYPE", "float32")
    p = Pair(tmp_path, full())
    prompt, n_gen = p.tokens(21, seed=6), 12
    seq, ids = list(prompt), []
    for _ in range(n_gen):
        lg = p.expected(seq)[-1]
        srt = np.sort(lg)
        assert srt[-1] - srt[-2] > 1e-3               # no near-tie: float32 must pick the same id
        ids.append(int(np.argmax(lg)))
        seq.append(ids[-1])
    L = _lib.lib()
    L.init(b"", b"")
    ctx = L.initContext(7, p.dir.encode(), 1, 0, 100, 0, 0, 0, 64, n_gen, 0, 0.0, 0.0, 0.0, 1, 1.0, 1.0, 1.0, 0, 0, 200, 1.0, 1.0, 1.0, 42, b"")
    assert ctx, _lib.last_error()
    for job in (b"bozisun-job", b"bozisun-again"):       # twice on one pod: the second job starts its sequence anew
        n = L.doInference(7, ctx, job, b"", " ".join(map(str, prompt)).encode())
        out = [int(x) for x in L.status(job).decode().split()]
        assert out[:len(prompt)] == prompt and out[len(prompt):] == ids
        assert n == len(prompt) + n_gen - 1 and L.getPromptTokenCount(job) == len(prompt)
    # the device-resident loop of the token-level interface gives the same ids, in one burst and in several
    for bursts in ([n_gen - 1], [1, 1, 2, n_gen - 5]):
        p.ctx.kv_clear()
        out, pos = [int(np.argmax(p.ctx.decode(prompt, 0)))], len(prompt)
        for b in bursts:
            out += p.ctx.generate_greedy(out[-1], pos, b).tolist()
            pos += b
        assert out == ids
        after = p.ctx.decode([ids[-1]], pos)          # a host-fed token pairs with the burst's last one
        assert err(after[None], p.expected(seq)[-1][None]) < TOL32
    assert p.ctx.L.b200_kernel_launches(p.ctx.h) > 0
    p.close()


def test_trace_runner_replays_steps(tmp_path):
    """bin/trace_run on a folder model of this design: wanted rows per step, a finished request's context used again"""
    import json
    import os
    import subprocess
    import sys
    cfg = full()
    w = bo.random_model(cfg, 5)
    d = bo.write_model(str(tmp_path / "m"), cfg, w)
    rng = np.random.default_rng(3)
    a, b = rng.integers(0, cfg["vocab"], size=40).tolist(), rng.integers(0, cfg["vocab"], size=23).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:31], "want": [0, 7, 30]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[31:33], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[33:40], "want": [6, 1]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[:22], "want": [0, 21]}], "end": []},
             {"step": 4, "entries": [{"id": "b", "tokens": b[22:], "want": [0]}], "end": ["b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(x) + "\n" for x in steps).encode(), stdout=subprocess.PIPE, stderr=subprocess.PIPE, timeout=600)
    assert r.returncode == 0, r.stderr.decode()[-2000:]
    assert [l for l in r.stdout.decode().split("\n") if l.startswith("done")] == ["done %d" % i for i in range(5)]
    assert not (out / "1.f32").exists()
    wa, wb = bo.forward(cfg, w, a)[0], bo.forward(cfg, w, b)[0]
    for n, want in ((0, wa[[0, 7, 30]]), (2, wa[[39, 34]]), (3, wb[[0, 21]]), (4, wb[[22]])):
        got = np.fromfile(str(out / ("%d.f32" % n)), "<f4").reshape(len(want), cfg["vocab"])
        assert err(got, want) < TOL32, n


def test_bad_models_fail_loudly(tmp_path):
    cfg = config([att(mlp=moe()), att(mlp=dense())], loop=(0, 1, 2))
    w = bo.random_model(cfg)

    def fails(match, edit, drop=None):
        c2 = copy.deepcopy(cfg)
        edit(c2)
        w2 = {k: v for k, v in w.items() if k != drop}
        with pytest.raises(_lib.B200Error, match=match):
            engine.Model(bo.write_model(str(tmp_path / "bad"), c2, w2))
    fails("not part of the Bozisun design", lambda c: c["layers"][1].update(type="retention"))
    fails("not part of the Bozisun design", lambda c: c["layers"][1]["mlp"].update(kind="poly"))
    fails("not part of the Bozisun design", lambda c: c["layers"][0]["mlp"].update(shared={"ff": 4}))
    fails("takes no mask", lambda c: c["layers"][0]["mixer"].update(mask={"size": 4}))
    fails("missing", lambda c: None, drop="l1.mix.q.norm")
    fails("missing", lambda c: None, drop="l0.mlp.router.b")
    fails("missing|rows", lambda c: None, drop="l0.mix.g")
    fails("missing", lambda c: None, drop="bigram")
    fails("missing", lambda c: None, drop="l1.side.proj")
    fails("shape", lambda c: c["embedding"]["bigram"].update(buckets=38))
    fails("multiple of kv_heads", lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    fails("exceeds the experts", lambda c: c["layers"][0]["mlp"]["router"].update(top=9))
    fails("within the layers", lambda c: c["loop"].update(stop=3))
    fails("must be even", lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10))
