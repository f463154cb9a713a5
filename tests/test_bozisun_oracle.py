"""The numpy restatement of the Bozisun design checked against itself and by hand (CPU): causality, the pair table's rows, the frequency
bands and the factor beside them, the rotation's pairs, grouped heads and the entry-wise gate, the router's choice and weights, the token
input, the order of the runs, the model writer."""
import numpy as np

import bozisun_oracle as bo
import stack_oracle as so
from test_bozisun_gpu import att, config, dense, full, moe


def test_later_tokens_do_not_reach_back():
    cfg = full()
    w = bo.random_model(cfg, 1)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], size=40).tolist()
    lg = bo.forward(cfg, w, toks)[0]
    for n in (1, 2, 17, 39):
        assert np.allclose(bo.forward(cfg, w, toks[:n])[0], lg[:n], rtol=0, atol=1e-9)


def test_pair_rows_by_hand():
    pc = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert bo.pair_rows([4, 1, 4], pc).tolist() == [10, (12 + 7) % 10, (3 + 28) % 10]
    assert bo.pair_rows([9], pc).tolist() == [10]


def test_frequencies_by_hand():
    f, m = bo.frequencies({"base": 10000.0, "dims": 4})
    assert np.allclose(f, [1.0, 0.01]) and m == 1.0
    rot = {"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0, "fast": 32.0, "slow": 1.0, "original": 4096}}
    # pair index at t turns: 8 ln(4096 / (2 pi t)) / (2 ln 10000) = 1.31 at 32, 2.81 at 1
    assert bo.yarn_bounds(rot) == (1.0, 3.0)
    f, m = bo.frequencies(rot)
    assert np.allclose(f, [1.0, 0.1, 0.01 * (0.5 / 4 + 0.5), 0.001 / 4]) and np.isclose(m, 0.1 * np.log(4.0) + 1.0)
    rot["scaling"].update(fast=1e9, slow=1e-9)                    # both ends cut: from the first pair to dims - 1
    assert bo.yarn_bounds(rot) == (0.0, 7.0)
    rot["scaling"].update(fast=5.0, slow=5.0, original=5.0 * 2 * np.pi * 10.0)      # an edge of no width at pair 1
    assert np.allclose(bo.frequencies(rot)[0], [1.0, 0.1, 0.01 / 4, 0.001 / 4])


def test_rotation_turns_half_split_pairs():
    x = np.zeros((2, 1, 5)); x[:, 0, 0] = 1.0; x[:, 0, 4] = 7.0
    y = bo.rotate(x, {"base": 100.0, "dims": 4})
    assert np.allclose(y[0], x[0]) and np.allclose(y[1, 0], [np.cos(1.0), 0, np.sin(1.0), 0, 7.0])


def test_attention_by_hand():
    """two query heads on one key head: at position 0 the value itself; equal scores: the values' mean; the gate entry by entry"""
    mx = {"heads": 2, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0}
    h = np.array([[1.0, 2.0], [3.0, -1.0]])
    W = {"q": np.ones((4, 2)), "k": np.zeros((2, 2)), "q.norm": np.ones(2), "k.norm": np.ones(2), "v": np.array([[1.0, 0.0], [0.0, 1.0]]), "g": np.array([[0, 0], [1.0, 0], [0, 1.0], [-1.0, 0]]), "o": np.eye(4)}
    y = bo.attention(h, mx, W, "", 1e-9)
    s = bo.sigmoid
    assert np.allclose(y[0], [0.5 * 1, s(1.0) * 2, s(2.0) * 1, s(-1.0) * 2])
    assert np.allclose(y[1], [0.5 * 2, s(3.0) * 0.5, s(-1.0) * 2, s(-3.0) * 0.5])


def test_router_choice_and_weights():
    sel, w = bo.route(np.ones((1, 1)), np.array([[1.0], [2.0], [3.0], [4.0]]), np.array([2.5, 0.0, 0.0, -9.0]), 2)
    assert sel.tolist() == [[0, 2]] and np.allclose(w, [[1 / (1 + np.exp(-0.5)), 1 / (1 + np.exp(0.5))]])
    sel, w = bo.route(np.zeros((1, 1)), np.zeros((4, 1)), np.zeros(4), 3)
    assert sel.tolist() == [[0, 1, 2]] and np.allclose(w, 1 / 3)                # the lowest index first among equals


def test_both_sub_layers_read_one_norm_and_the_token_input_comes_last():
    cfg = config([att(mlp=dense())], side=3, pairs=(5, 2, 1))
    w = bo.random_model(cfg, 5)
    toks = [3, 1, 4, 1, 5]
    x = w["embed"][toks] + w["bigram"][[5, 7 % 5, 6 % 5, 9 % 5, 7 % 5]]
    h = x / np.sqrt((x * x).mean(-1, keepdims=True) + 1e-5) * w["l0.norm1"]
    x = x + bo.attention(h, cfg["layers"][0]["mixer"], w, "l0.mix.", 1e-5) + bo.gated(h, w, "l0.mlp.")
    y = (bo.gelu_tanh(x @ w["l0.side.gate"].T) * w["side.embed"][toks]) @ w["l0.side.proj"].T
    x = x + y / np.sqrt((y * y).mean(-1, keepdims=True) + 1e-5) * w["l0.side.norm"]
    assert np.allclose(bo.forward(cfg, w, toks)[1][0], x)


def test_run_order_and_slices():
    cfg = config([att(), att(), att()], loop=(1, 3, 2))
    assert bo.run_order(cfg) == [0, 1, 2, 1, 2]
    w = bo.random_model(cfg, 3)
    toks = [7, 8, 9]
    base = bo.forward(cfg, w, toks)[1]
    w2 = dict(w); w2["side.embed"] = w["side.embed"].copy(); w2["side.embed"][:, 20:] += 1.0      # the third layer's slice
    moved = [not np.allclose(a, b) for a, b in zip(bo.forward(cfg, w2, toks)[1], base)]
    assert moved == [False, False, True, True, True]


def test_soft_cap():
    assert np.allclose(bo.soft_cap(np.array([0.0, 1e9, -1e9]), 5.0), [0.0, 5.0, -5.0]) and bo.soft_cap(3.0, 0.0) == 3.0


def test_mixture_sums_the_weighted_choices():
    cfg = config([att(mlp=moe(experts=3, top=2, ff=5))], width=6)
    w = bo.random_model(cfg, 2)
    h = np.random.default_rng(1).standard_normal((4, 6))
    y = bo.mixture(h, cfg["layers"][0]["mlp"], w, "l0.mlp.")
    sel, wt = bo.route(h, w["l0.mlp.router"], w["l0.mlp.router.b"], 2)
    for t in range(4):
        assert np.allclose(y[t], sum(a * bo.gated(h[t:t + 1], w, "l0.mlp.e%d." % e)[0] for e, a in zip(sel[t], wt[t])))


def test_model_writer_round_trips(tmp_path):
    cfg = full()
    w = bo.random_model(cfg, 3)
    d = bo.write_model(str(tmp_path / "m"), cfg, w)
    back = so.load_safetensors(d + "/model.safetensors")
    assert set(back) == set(w) == set(bo.tensor_shapes(cfg))
    for k in w:
        assert list(np.shape(back[k])) == bo.tensor_shapes(cfg)[k] and np.array_equal(np.asarray(back[k], np.float64), w[k])
