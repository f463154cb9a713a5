"""The Kogerax design on the GPU against the plain numpy restatement in tests/kogerax_oracle.py: every mechanism alone (with and
without each feed-forward, with the residual after the layer), whole prompts against token-by-token decoding and portions down to
two tokens, contexts that are cleared and used again, several live contexts stepping in turn, what every position sees through the
attention's window (by changing one token and looking at who notices), far tokens through the recurrences, the first tokens of a
sequence, long decoding through the replayed graph, other sizes (scalar and vector load paths, one to many state entries,
grouped and ungrouped heads, partial and no rotation, every band of the frequency scaling, identity outputs, no shared unit, no
feed-forward, values that are 1), bfloat16, greedy generation through the bridge's job loop and the trace runner. Small random
models in a temporary folder; float32 is the sharp comparison."""
import copy

import numpy as np
import pytest

import kogerax_oracle as ko
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


def moe(experts=6, top=2, ff=20, limit=1.2, identity=2, shared=12, shared_limit=0.9):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if identity:
        m["router"]["identity"] = identity
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def par(heads=4, kv_heads=2, dim=8, vdim=6, size=9, scale=0.4, rot=4, base=100.0, scaling=(4.0, 1.0, 4.0, 64), inner=20, state=6, dt_rank=3, conv=3, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}
    if rot:
        left["rot"] = {"base": base, "dims": rot}
        if scaling:
            left["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "parallel", "mixer": {"left": left, "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}, "mlp": mlp}


def mlstm(heads=3, dim=8, vdim=6, cap=10.0, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def ssd(heads=4, vdim=6, state=8, groups=2, norm_groups=2, conv=4, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}, "mlp": mlp}


def config(layers, width=48, vocab=61, eps=1e-5, mult=0.7, scale=3.0):
    return {"architecture": "Kogerax", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


class Pair:
    """the same random model in the framework and in the oracle"""

    def __init__(self, tmp_path, cfg, seed=0, dtype="float32", n_ctx=512, edit=None):
        self.cfg = cfg
        self.w = ko.random_model(cfg, seed)
        if edit:
            edit(self.w)
        self.dir = ko.write_model(str(tmp_path / f"k{seed}_{dtype}_{abs(hash(str(cfg))) % 10**8}"), cfg, self.w)
        self.model = engine.Model(self.dir, dtype=dtype)
        self.ctx = engine.Context(self.model, n_ctx)

    def close(self):
        self.ctx.close()
        self.model.close()

    def tokens(self, n, seed=1):
        return np.random.default_rng(seed).integers(0, self.cfg["vocab"], size=n).tolist()

    def expected(self, toks, cfg=None, w=None, residuals=False):
        lg, taps = ko.forward(cfg or self.cfg, w or self.w, toks)
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


ALONE = {"parallel": par(), "parallel-ungrouped-unscaled+dense": par(heads=3, kv_heads=3, dim=5, vdim=7, size=4, rot=4, scaling=None, inner=13, state=1, dt_rank=1, conv=1, mlp=dense(9)),
         "parallel-plain+moe": par(heads=2, kv_heads=1, dim=12, vdim=16, rot=0, size=1, inner=32, state=16, dt_rank=8, conv=4, mlp=moe()),
         "mlstm": mlstm(), "mlstm-one-head+dense": mlstm(heads=1, dim=5, vdim=9, cap=2.0, mlp=dense()), "mlstm-wide+moe": mlstm(heads=2, dim=20, vdim=33, mlp=moe(identity=0, top=3)),
         "mamba2": ssd(), "mamba2-one-group+moe": ssd(heads=3, vdim=5, state=9, groups=1, norm_groups=1, conv=2, mlp=moe(experts=3, top=4, shared=0)),
         "mamba2-own-groups+dense": ssd(heads=4, vdim=8, state=20, groups=4, norm_groups=4, conv=1, mlp=dense(24))}


@pytest.mark.parametrize("name", list(ALONE))
def test_each_mixer_alone_with_the_residual_after_the_layer(tmp_path, name):
    p = Pair(tmp_path, config([ALONE[name]]))
    toks = p.tokens(29)
    want, res = p.expected(toks, residuals=True)
    p.ctx.set_taps(True)
    got = p.ctx.decode_rows(toks, 0, list(range(len(toks))))
    taps = p.ctx.layer_taps(len(toks))
    p.ctx.set_taps(False)
    assert taps.shape[0] == 1 and np.abs(taps[0] - res[0]).max() < 1e-4 * max(1.0, np.abs(res[0]).max())
    assert err(got, want) < TOL32
    for cuts in ([1], [2], [3], [5, 1, 9]):
        assert err(p.run(toks, cuts), want) < TOL32, cuts
    p.close()


FULL = [par(mlp=dense()), mlstm(mlp=moe()), ssd(mlp=moe(experts=4, top=1, ff=16, shared=24, identity=1)), par(heads=2, kv_heads=2, dim=16, vdim=12, size=16, rot=16, inner=24, state=16, mlp=moe(experts=5, top=3)),
        ssd(heads=2, vdim=16, state=4, groups=1, norm_groups=1), mlstm(heads=2, dim=16, vdim=8, mlp=moe(experts=9, top=3, shared=0))]


def test_small_mechanisms_matter(tmp_path):
    """the oracle without one of the small mechanisms is far from the framework: none of them is a no-op in these models"""
    cfg = config([par(mlp=moe()), mlstm(mlp=dense()), ssd(mlp=moe(top=1, identity=4))])
    p = Pair(tmp_path, cfg)
    toks = p.tokens(41)
    got = p.run(toks)
    assert err(got, p.expected(toks)) < TOL32
    for key in ("l0.norm1", "l0.norm2", "l1.norm1", "final.norm", "l0.mix.right.conv.b", "l0.mix.right.dt.b", "l0.mix.right.D", "l0.mix.right.A_log", "l0.mix.left.out", "l0.mix.right.out", "l0.mlp.router", "l0.mlp.shared.sg",
                "l1.mix.i", "l1.mix.i.b", "l1.mix.f", "l1.mix.f.b", "l1.mix.g", "l2.mix.conv.b", "l2.mix.dt_bias", "l2.mix.A_log", "l2.mix.D", "l2.mlp.correction"):
        w2 = dict(p.w); w2[key] = np.zeros_like(p.w[key])
        assert err(got, p.expected(toks, w=w2)) > 20 * TOL32, key
    for key in ("l1.mix.norm", "l2.mix.norm", "l0.mix.right.conv", "l2.mix.conv"):
        w2 = dict(p.w); w2[key] = p.w[key] * np.linspace(0.5, 1.5, p.w[key].size).reshape(p.w[key].shape)
        assert err(got, p.expected(toks, w=w2)) > 20 * TOL32, key
    left = lambda c: c["layers"][0]["mixer"]["left"]
    for edit in (lambda c: left(c)["rot"].update(base=50.0), lambda c: left(c)["rot"].update(dims=8), lambda c: left(c)["rot"].pop("scaling"), lambda c: left(c)["mask"].update(size=10), lambda c: left(c)["mask"].update(size=8),
                 lambda c: left(c).update(scale=0.3), lambda c: c["layers"][1]["mixer"].update(gate_cap=3.0), lambda c: c["layers"][2]["mixer"].update(norm_groups=1), lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.8),
                 lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0.5), lambda c: c["layers"][0]["mlp"]["router"].update(top=3), lambda c: c["norm"].update(eps=1e-1), lambda c: c.update(residual_mult=0.6),
                 lambda c: c["embedding"].update(scale=2.5)):
        c2 = copy.deepcopy(cfg); edit(c2)
        assert err(got, p.expected(toks, cfg=c2)) > 20 * TOL32, c2
    # and one function at a time, restated wrongly on purpose
    keep = {n: getattr(ko, n) for n in ("gelu_tanh", "GATE_SLOPE", "route")}

    def weights_with_correction(h, Wr, corr, top):
        sel, _ = keep["route"](h, Wr, corr, top)
        z = h @ Wr.T
        s = np.exp(z - z.max(-1, keepdims=True)); s = s / s.sum(-1, keepdims=True) + corr
        w = np.take_along_axis(s, sel, -1)
        return sel, w / w.sum(-1, keepdims=True)
    for name, f in (("gelu_tanh", ko.silu), ("GATE_SLOPE", 1.0), ("route", weights_with_correction)):
        setattr(ko, name, f)
        try:
            assert err(got, p.expected(toks)) > 20 * TOL32, name
        finally:
            setattr(ko, name, keep[name])
    p.close()


def test_identity_outputs(tmp_path):
    """all choices identity (their correction is large), none, and a mixture of both, in prompts and in decoding"""
    for top, shift in ((2, 5.0), (2, -5.0), (3, 0.0), (1, 5.0)):
        cfg = config([ssd(mlp=moe(experts=4, top=top, identity=3, shared=8 if top == 2 else 0))])

        def edit(w):
            c = w["l0.mlp.correction"].copy(); c[4:] += shift
            w["l0.mlp.correction"] = bf16(c)
        p = Pair(tmp_path, cfg, seed=int(10 * top + shift), edit=edit)
        toks = p.tokens(40)
        want, res = p.expected(toks, residuals=True)
        for cuts in (None, [1], [3], [7, 2]):
            assert err(p.run(toks, cuts), want) < TOL32, (top, shift, cuts)
        p.close()


def test_running_maximum_and_divisor(tmp_path):
    """input gates that jump (a new maximum rescales what is held), forget gates from shut to open, and read-outs small enough for the
    other side of the divisor: each against the oracle in one step, token by token and across the long-portion path"""
    for seed, (ib, fb, gain) in enumerate([(0.0, 0.0, 6.0), (-6.0, 6.0, 3.0), (6.0, -6.0, 3.0), (-9.0, 8.0, 0.5), (3.0, 20.0, 1.0)]):
        cfg = config([mlstm(heads=2, dim=8, vdim=10, cap=8.0 + seed, mlp=dense())], eps=0.3)      # a large eps: the read-out's own size matters

        def edit(w):
            w["l0.mix.i"] = bf16(w["l0.mix.i"] * gain); w["l0.mix.f"] = bf16(w["l0.mix.f"] * gain)
            w["l0.mix.i.b"] = bf16(np.full(2, ib)); w["l0.mix.f.b"] = bf16(np.full(2, fb))
        p = Pair(tmp_path, cfg, seed=seed, edit=edit)
        toks = p.tokens(300)
        want = p.expected(toks)
        for cuts in (None, [1], [130, 2, 40, 128]):
            assert err(p.run(toks, cuts), want) < TOL32, (ib, fb, gain, cuts)
        if seed == 0:                                     # both sides of the divisor are in use, and leaving one out shows
            keep = ko.divisor
            for f in (lambda nq, m: np.exp(-m), lambda nq, m: abs(nq) + 1e-6):
                ko.divisor = f
                try:
                    assert err(p.expected(toks), want) > 20 * TOL32
                finally:
                    ko.divisor = keep
        p.close()


def test_whole_prompt_token_by_token_and_portions_agree(tmp_path):
    p = Pair(tmp_path, config(FULL))
    toks = p.tokens(75)
    want, res = p.expected(toks, residuals=True)
    p.ctx.set_taps(True)
    p.ctx.kv_clear()
    p.ctx.decode_rows(toks, 0, [])
    taps = p.ctx.layer_taps(len(toks))
    p.ctx.set_taps(False)
    assert taps.shape[0] == len(res) == len(FULL)
    for a, b in zip(taps, res):
        assert np.abs(a - b).max() < 1e-4 * max(1.0, np.abs(b).max())
    assert err(p.run(toks), want) < TOL32
    assert err(p.run(toks, [1]), want) < TOL32        # every token through the replayed one-token graph
    for cuts in ([2], [3, 2, 7, 1, 5], [37, 2, 2, 30], [6, 1, 1, 11], [4], [9, 8], [1, 2]):
        assert err(p.run(toks, cuts), want) < TOL32, cuts
    p.close()


def test_portions_around_the_switch_to_chunks(tmp_path):
    """portions just below, at and above the length from which the matrix-state recurrences run chunk by chunk, whole and ragged chunks,
    each continued by the walk and by single tokens"""
    p = Pair(tmp_path, config([mlstm(mlp=dense()), ssd(), par(inner=40, state=16), ssd(heads=2, vdim=70, state=33, groups=1, norm_groups=1), mlstm(heads=2, dim=36, vdim=130)]), n_ctx=420)
    toks = p.tokens(400, seed=7)
    want = p.expected(toks)
    for cuts in (None, [127, 1], [128, 1, 2], [129, 127, 3], [160, 31, 1], [255, 145], [2, 398], [191, 1, 1, 193]):
        assert err(p.run(toks, cuts), want) < TOL32, cuts
    p.close()


def test_cleared_context_is_as_good_as_new_and_contexts_do_not_meet(tmp_path):
    p = Pair(tmp_path, config(FULL))
    a, b = p.tokens(60, seed=3), p.tokens(29, seed=4)
    fresh = engine.Context(p.model, 512)
    ref_b = p.run(b, [5, 1, 1, 9], ctx=fresh)
    p.run(a, [7, 1])                                  # fills cache rows, matrix states, maxima and convolution histories
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


@pytest.mark.parametrize("size", [1, 2, 9, 16, 17, 33, 200])
def test_who_notices_a_changed_token(tmp_path, size):
    """a model whose only path between positions is the attention's window (the scan's branch is weighed with zero): when token j
    changes, exactly the positions j .. j + size - 1 change, in a whole prompt, in decoding and in portions that start anywhere"""
    cfg = config([par(size=size)], width=32, vocab=40)

    def edit(w):
        w["l0.mix.right.out"] = np.zeros_like(w["l0.mix.right.out"])
    p = Pair(tmp_path, cfg, seed=2, edit=edit)
    n = 70
    toks = p.tokens(n, seed=5)
    for cuts in (None, [40, 1], [2, 3, 5, 1, 7, 11]):
        base = p.run(toks, cuts)
        for j in (0, 3, 17, 32, 44):
            other = list(toks); other[j] = (toks[j] + 1) % 40
            got = p.run(other, cuts)
            for q in range(n):
                assert np.array_equal(got[q], base[q]) != (0 <= q - j < size), (cuts, j, q)
    assert err(p.run(toks), p.expected(toks)) < TOL32
    p.close()


@pytest.mark.parametrize("size", [1, 2, 9, 33])
def test_window_edges_with_steep_scores(tmp_path, size):
    """peaked attention: an oracle whose window is one token off, or whose angles are off, is far away"""
    cfg = config([par(size=size, dim=8, rot=8, scale=2.5, mlp=dense())], width=32, vocab=40)
    p = Pair(tmp_path, cfg, seed=size)
    toks = p.tokens(150, seed=size)
    want = p.expected(toks)
    for d in (1, -1):
        if size + d > 0:
            c2 = copy.deepcopy(cfg); c2["layers"][0]["mixer"]["left"]["mask"]["size"] = size + d
            assert err(p.expected(toks, cfg=c2), want) > 50 * TOL32
    for cuts in (None, [110, 1], [size, 1, size + 1, 2, 31], [7, 2]):
        assert err(p.run(toks, cuts), want) < TOL32, cuts
    p.close()


def test_frequency_bands(tmp_path):
    """frequencies below, inside and above the blended band all occur, and reading any band differently shows"""
    rot = {"base": 1000.0, "dims": 16, "scaling": {"factor": 6.0, "low": 1.0, "high": 5.0, "original": 60}}
    plain, scaled = ko.frequencies({"base": 1000.0, "dims": 16}), ko.frequencies(rot)
    kept, slowed = np.isclose(scaled, plain), np.isclose(scaled, plain / 6.0)
    assert kept.any() and slowed.any() and not (kept | slowed).all()
    L = par(heads=2, kv_heads=2, dim=18, vdim=8, size=60, scale=1.0, rot=0)
    L["mixer"]["left"]["rot"] = rot
    cfg = config([L])
    p = Pair(tmp_path, cfg, seed=4)
    toks = p.tokens(120)
    want = p.expected(toks)
    for key, val in (("factor", 3.0), ("low", 2.0), ("high", 3.0), ("original", 30)):
        c2 = copy.deepcopy(cfg); c2["layers"][0]["mixer"]["left"]["rot"]["scaling"][key] = val
        assert err(p.expected(toks, cfg=c2), want) > 20 * TOL32, key
    for cuts in (None, [100, 1], [3, 14]):
        assert err(p.run(toks, cuts), want) < TOL32, cuts
    p.close()


@pytest.mark.parametrize("kind", ["parallel", "mlstm", "mamba2"])
def test_far_tokens_reach_through_the_state(tmp_path, kind):
    """slow decays: a token at position 3 moves the logits 300 positions later, in prompts, in decoding and across portions; the odd
    token stands out (its embedding row is large, the others' are alike)"""
    L = {"parallel": par(size=3, inner=24, state=4), "mlstm": mlstm(heads=2, dim=8, vdim=8), "mamba2": ssd(heads=2, vdim=12, state=8, groups=1, norm_groups=1)}[kind]
    cfg = config([L], width=32, vocab=40, mult=1.0)

    def edit(w):
        e = w["embed"].copy()
        e[:39] = e[0] + 0.3 * e[:39]
        e[39] *= 12.0
        w["embed"] = bf16(e)
        if kind == "parallel":
            w["l0.mix.right.A_log"] = bf16(np.full_like(w["l0.mix.right.A_log"], -7.0))
        elif kind == "mamba2":
            w["l0.mix.A_log"] = bf16(np.full_like(w["l0.mix.A_log"], -7.0))
        else:
            w["l0.mix.f"] = bf16(0.1 * w["l0.mix.f"]); w["l0.mix.f.b"] = np.full_like(w["l0.mix.f.b"], 8.0)
            w["l0.mix.i"] = bf16(np.outer([0.4, 0.5], e[39] / np.linalg.norm(e[39])))      # the odd token's input gate opens wide
    p = Pair(tmp_path, cfg, seed=6, n_ctx=400, edit=edit)
    plain = np.random.default_rng(9).integers(0, 39, size=330).tolist()
    odd = list(plain); odd[3] = 39
    want, base = p.expected(odd), p.expected(plain)
    late = row_errs(base, want)[300:]
    assert late.min() > 5 * TOL32 and np.median(late) > 50 * TOL32
    for cuts in (None, [300, 1], [2, 129, 3, 64], [1, 150, 1, 150]):
        assert err(p.run(odd, cuts), want) < TOL32, cuts
    assert err(p.run(odd[:40], [1]), want[:40]) < TOL32          # the first tokens of a sequence
    assert err(p.run(plain, [31, 32, 33, 1]), base) < TOL32
    p.close()


def test_long_decoding_through_the_graph(tmp_path):
    p = Pair(tmp_path, config(FULL))
    toks = p.tokens(300, seed=11)
    want = p.expected(toks)
    got = p.run(toks, [4] + [1] * 300)
    assert err(got, want) < 2 * TOL32
    p.close()


@pytest.mark.parametrize("width,vocab", [(36, 50), (40, 77), (64, 130), (37, 53)], ids=["scalar-loads", "width-40", "vector-loads", "odd-width"])
def test_other_sizes(tmp_path, width, vocab):
    layers = [par(heads=6, kv_heads=2, dim=9, vdim=5, size=3, rot=2, inner=17, state=2, dt_rank=5, conv=2, mlp=moe(experts=3, top=3, ff=7, shared=3, identity=1)),
              mlstm(heads=5, dim=9, vdim=5, cap=4.0),
              ssd(heads=6, vdim=4, state=7, groups=3, norm_groups=3, conv=5, mlp=dense(33)),
              par(heads=4, kv_heads=4, dim=16, vdim=40, size=40, rot=6, inner=64, state=40, dt_rank=4, conv=4, mlp=moe(experts=16, top=4, ff=64, shared=64, identity=5)),
              ssd(heads=1, vdim=48, state=1, groups=1, norm_groups=1, conv=1),
              mlstm(heads=1, dim=70, vdim=1, mlp=moe(experts=1, top=1, ff=24, identity=0)),
              par(heads=4, kv_heads=1, dim=64, vdim=5, size=7, rot=64, inner=8, state=100, dt_rank=9, mlp=moe(experts=2, top=2, identity=1, shared=0)),
              ssd(heads=8, vdim=1, state=130, groups=8, norm_groups=2, conv=3),
              mlstm(heads=3, dim=1, vdim=16),
              par(heads=1, kv_heads=1, dim=4, vdim=4, size=5, rot=4, inner=300, state=200, dt_rank=2, conv=6)]
    p = Pair(tmp_path, config(layers, width=width, vocab=vocab, eps=1e-6, mult=1.0, scale=1.0), seed=width)
    toks = p.tokens(70, seed=width)
    want = p.expected(toks)
    assert err(p.run(toks), want) < TOL32
    assert err(p.run(toks, [13, 2, 1]), want) < TOL32
    p.close()


def test_wide_rows(tmp_path):
    """rows longer than what the join and the gated norm keep in registers, many heads, odd and even widths"""
    for width in (2500, 1031):
        layers = [ssd(heads=8, vdim=300, state=4, groups=2, norm_groups=1), par(heads=2, kv_heads=1, dim=8, vdim=8, inner=1100, state=3, mlp=moe(experts=2, top=2, ff=8, identity=1, shared=4)), mlstm(heads=2, dim=200, vdim=260)]
        p = Pair(tmp_path, config(layers, width=width, vocab=40), seed=1, n_ctx=160)
        toks = p.tokens(150, seed=1)
        want = p.expected(toks)
        assert err(p.run(toks), want) < TOL32
        assert err(p.run(toks[:30], [20, 1, 1, 3]), want[:30]) < TOL32
        p.close()


def random_config(rng):
    """a random arrangement of the mixers with random sizes: nothing may rest on one model's values"""
    pick = lambda values: int(rng.choice(values))

    def ff():
        u = rng.random()
        if u < 0.2:
            return None
        if u < 0.45:
            return dense(pick([8, 30, 64, 136]))
        n, ident = pick([1, 2, 5, 8, 12]), pick([0, 1, 3])
        return moe(experts=n, top=pick(range(1, min(n + ident, 5) + 1)), ff=pick([8, 24, 64, 100]), limit=float(rng.choice([0.5, 1.5, 7.0])), identity=ident, shared=pick([0, 8, 40, 136]),
                   shared_limit=float(rng.choice([0.7, 3.0])))
    layers = []
    for _ in range(pick([2, 3, 4, 6])):
        kind = pick([0, 1, 2])
        if kind == 0:
            kv, d = pick([1, 2, 3]), pick([4, 6, 16, 32, 64, 128])
            rot = pick([r for r in (0, 2, 4, 16, 32, 64, 128) if r <= d])
            layers.append(par(heads=kv * pick([1, 2, 4]), kv_heads=kv, dim=d, vdim=pick([4, 8, 48, 128, 200]), size=pick([1, 3, 16, 50, 128, 1000]), scale=float(rng.choice([0.1, 0.3])), rot=rot,
                              base=float(rng.choice([100.0, 1e4, 5e5])), scaling=None if rng.random() < 0.4 else (float(rng.choice([2.0, 8.0])), 1.0, 4.0, pick([64, 512, 4096])),
                              inner=pick([16, 50, 128, 260]), state=pick([1, 4, 8, 16, 24, 64]), dt_rank=pick([1, 4, 8, 24]), conv=pick([1, 2, 4]), mlp=ff()))
        elif kind == 1:
            layers.append(mlstm(heads=pick([1, 2, 4]), dim=pick([4, 12, 32, 64, 128]), vdim=pick([4, 16, 48, 64, 130]), cap=float(rng.choice([2.0, 15.0, 30.0])), mlp=ff()))
        else:
            g = pick([1, 2, 3])
            h = g * pick([1, 2, 4])
            layers.append(ssd(heads=h, vdim=pick([4, 16, 48, 64, 100]), state=pick([4, 8, 32, 60, 128]), groups=g, norm_groups=pick([1, g, h]), conv=pick([1, 2, 4]), mlp=ff()))
    return config(layers, width=pick([24, 36, 64, 100, 136]), vocab=pick([37, 100, 257, 513]), eps=float(rng.choice([1e-6, 1e-5])), mult=float(rng.choice([0.3, 1.0, 1.5])), scale=float(rng.choice([1.0, 5.0, 12.0])))


@pytest.mark.parametrize("seed", range(10))
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
    """a 700-token step runs as two passes of the layers: cached keys, states, maxima and convolution histories cross the pass's edge"""
    p = Pair(tmp_path, config(FULL), n_ctx=704)
    toks = p.tokens(700, seed=5)
    want = p.expected(toks)
    assert err(p.run(toks), want) < 2 * TOL32
    assert err(p.run(toks, [509, 2, 3, 186]), want) < 2 * TOL32
    p.close()


def test_bfloat16_prompt_kernels_and_decode(tmp_path):
    """wide enough for the tensor-core products, also the segmented ones of the routed mixture"""
    layers = [par(heads=4, kv_heads=2, dim=32, vdim=32, size=40, rot=16, inner=192, state=16, dt_rank=8, conv=4, mlp=dense(256)),
              mlstm(heads=4, dim=32, vdim=64, mlp=moe(experts=4, top=2, ff=64, shared=64)),
              ssd(heads=4, vdim=32, state=32, groups=1, norm_groups=1, mlp=moe(experts=3, top=2, ff=128, identity=1, shared=128))]
    cfg = config(layers, width=128, vocab=160)
    p = Pair(tmp_path, cfg, dtype="bfloat16")
    toks = p.tokens(300, seed=2)
    keep, gaps = ko.route, []

    def watched(h, Wr, corr, top):                     # how close the choice of experts is, position by position
        z = h @ Wr.T
        s = np.exp(z - z.max(-1, keepdims=True))
        c = np.sort(s / s.sum(-1, keepdims=True) + corr, axis=-1)
        gaps.append(c[:, -top] - c[:, -top - 1])
        return keep(h, Wr, corr, top)
    ko.route = watched
    try:
        want = p.expected(toks)
    finally:
        ko.route = keep
    clear = np.min(gaps, axis=0) > 0.02
    assert clear.mean() > 0.5
    # token by token: mat-vec kernels with float32 activations on the stored bfloat16 weights: as sharp as float32
    assert err(p.run(toks[:60], [1]), want[:60]) < TOL32
    assert err(p.run(toks[:60], [3, 4, 2]), want[:60]) < TOL32
    # longer portions: tensor-core products round the activation operand to bfloat16
    for cuts in (None, [280, 1], [5, 17, 133]):
        e = row_errs(p.run(toks, cuts), want)
        # where rounding cannot change the choice of an expert
        assert np.median(e) < 2e-2 and e[clear].max() < 0.1, (cuts, float(np.median(e)), float(e[clear].max()), np.argsort(-e)[:5], np.sort(-e)[:5])
    p.close()


def test_greedy_generation_through_the_bridge(tmp_path, monkeypatch):
    """initContext / doInference on a folder model: decimal-id prompt, standard chain at temperature 0 (arg-max on the device),
    prompt through the prompt kernels, generation through the one-token graph: the ids the oracle generates greedily"""
    monkeypatch.setenv("BOOSTER_B200_DTYPE", "float32")
    p = Pair(tmp_path, config(FULL[:4]))
    prompt, n_gen = p.tokens(21, seed=6), 10
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
    n = L.doInference(7, ctx, b"kogerax-job", b"", " ".join(map(str, prompt)).encode())
    out = [int(x) for x in L.status(b"kogerax-job").decode().split()]
    assert out[:len(prompt)] == prompt and out[len(prompt):] == ids
    assert n == len(prompt) + n_gen - 1 and L.getPromptTokenCount(b"kogerax-job") == len(prompt)
    # the device-resident loop of the token-level interface gives the same ids
    p.ctx.kv_clear()
    first = int(np.argmax(p.ctx.decode(prompt, 0)))
    dev = p.ctx.generate_greedy(first, len(prompt), n_gen - 1).tolist()
    assert [first] + dev == ids
    after = p.ctx.decode([ids[-1]], len(prompt) + n_gen - 1)
    assert err(after[None], p.expected(seq)[-1][None]) < TOL32
    assert p.ctx.L.b200_kernel_launches(p.ctx.h) > 0
    p.close()


def test_trace_runner_replays_steps(tmp_path):
    """bin/trace_run on a folder model of this design: wanted rows per step, a finished request's context used again"""
    import json
    import os
    import subprocess
    import sys
    cfg = config(FULL[:3])
    w = ko.random_model(cfg, 5)
    d = ko.write_model(str(tmp_path / "m"), cfg, w)
    rng = np.random.default_rng(3)
    a, b = rng.integers(0, cfg["vocab"], size=40).tolist(), rng.integers(0, cfg["vocab"], size=23).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:31], "want": [0, 7, 30]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[31:33], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[33:40], "want": [6, 1]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[:22], "want": [21]}], "end": []},
             {"step": 4, "entries": [{"id": "b", "tokens": b[22:], "want": [0]}], "end": ["b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(x) + "\n" for x in steps).encode(), stdout=subprocess.PIPE, stderr=subprocess.PIPE, timeout=600)
    assert r.returncode == 0, r.stderr.decode()[-2000:]
    assert [l for l in r.stdout.decode().split("\n") if l.startswith("done")] == ["done %d" % i for i in range(5)]
    assert not (out / "1.f32").exists()
    wa, wb = ko.forward(cfg, w, a)[0], ko.forward(cfg, w, b)[0]
    for n, want in ((0, wa[[0, 7, 30]]), (2, wa[[39, 34]]), (3, wb[[21]]), (4, wb[[22]])):
        got = np.fromfile(str(out / ("%d.f32" % n)), "<f4").reshape(len(want), cfg["vocab"])
        assert err(got, want) < TOL32, n


def test_bad_models_fail_loudly(tmp_path):
    cfg = config([par(mlp=moe()), mlstm(), ssd(mlp=dense())])
    w = ko.random_model(cfg)

    def fails(match, edit, drop=None):
        c2 = copy.deepcopy(cfg)
        edit(c2)
        w2 = {k: v for k, v in w.items() if k != drop}
        with pytest.raises(_lib.B200Error, match=match):
            engine.Model(ko.write_model(str(tmp_path / "bad"), c2, w2))
    fails("not part of the Kogerax design", lambda c: c["layers"][1].update(type="retention"))
    fails("missing", lambda c: None, drop="l1.mix.f.b")
    fails("missing", lambda c: None, drop="l0.mlp.correction")
    fails("multiple of kv_heads", lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3))
    fails("multiple of groups", lambda c: c["layers"][2]["mixer"].update(groups=3))
    fails("multiple of norm_groups", lambda c: c["layers"][2]["mixer"].update(norm_groups=7))
    fails("exceeds the experts", lambda c: c["layers"][0]["mlp"]["router"].update(top=9))
    fails("gate_cap", lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0))
    fails("not part of the Kogerax design", lambda c: c["layers"][2]["mlp"].update(kind="poly"))
