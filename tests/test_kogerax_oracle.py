"""The numpy restatement of the Kogerax design checked against itself and by hand (CPU): causality, the window's reach, the frequency
bands, the running maximum's independence of its own value, both scans against closed forms, the router's choice and weights, the
clamped unit, the join's scale, the model writer."""
import numpy as np

import kogerax_oracle as ko
import stack_oracle as so
from test_kogerax_gpu import FULL, config, dense, mlstm, moe, par, ssd


def test_later_tokens_do_not_reach_back():
    cfg = config(FULL)
    w = ko.random_model(cfg, 1)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], size=40).tolist()
    full = ko.forward(cfg, w, toks)[0]
    for n in (1, 2, 17, 39):
        assert np.allclose(ko.forward(cfg, w, toks[:n])[0], full[:n], rtol=0, atol=1e-9)


def test_window_reaches_size_tokens():
    for size in (1, 4):
        cfg = config([par(size=size)])
        w = ko.random_model(cfg, 2)
        w["l0.mix.right.out"] = np.zeros_like(w["l0.mix.right.out"])
        toks = list(range(12))
        other = list(toks); other[3] = 50
        moved = np.abs(ko.forward(cfg, w, toks)[0] - ko.forward(cfg, w, other)[0]).max(-1) > 0
        assert moved.tolist() == [0 <= t - 3 < size for t in range(12)]


def test_frequencies_by_hand():
    f = ko.frequencies({"base": 10000.0, "dims": 4})
    assert np.allclose(f, [1.0, 0.01])
    sc = {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100.0}
    g = ko.frequencies({"base": 10000.0, "dims": 4, "scaling": sc})
    assert np.allclose(g, [1.0, 0.0025])                          # wavelengths 6.28 < 25 and 628 > 100
    sc["original"] = 1256.0                                       # 628.3 lies between 314 and 1256: original / wavelength = 2
    s = (1256.0 / (2 * np.pi / 0.01) - 1.0) / 3.0
    assert np.allclose(ko.frequencies({"base": 10000.0, "dims": 4, "scaling": sc})[1], (1 - s) * 0.0025 + s * 0.01)


def test_rotation_turns_half_split_pairs():
    x = np.zeros((2, 1, 5)); x[:, 0, 0] = 1.0; x[:, 0, 4] = 7.0
    y = ko.rotate_half(x, {"base": 100.0, "dims": 4})
    assert np.allclose(y[0], x[0]) and np.allclose(y[1, 0], [np.cos(1.0), 0, np.sin(1.0), 0, 7.0])


def test_running_maximum_is_only_a_scale():
    """apart from the divisor's floor, e^m cancels: the read-out is sum_j w_j (k_j . q) v_j over |sum_j w_j (k_j . q)| with plain gates"""
    rng = np.random.default_rng(3)
    T, E, D, V = 9, 6, 4, 3
    mx = {"heads": 1, "dim": D, "vdim": V, "gate_cap": 5.0}
    W = {k: rng.standard_normal(s) for k, s in (("q", (D, E)), ("k", (D, E)), ("v", (V, E)), ("g", (V, E)), ("i", (1, E)), ("f", (1, E)), ("i.b", 1), ("f.b", 1))}
    W["i.b"] = W["i.b"] + 4.0                                      # large input gates: |n . q| beats e^(-m)
    W["q"] = 30.0 * W["q"]
    W["norm"], W["o"] = np.ones(V), np.eye(V)
    h = rng.standard_normal((T, E))
    got = ko.mlstm(h, mx, W, "", 1e-12) / ko.sigmoid(h @ W["g"].T)
    q, k, v = h @ W["q"].T * D ** -0.5, h @ W["k"].T, h @ W["v"].T
    li = 5.0 * np.tanh((h @ W["i"].T + W["i.b"])[:, 0] / 5.0)
    lf = ko.log_sigmoid(5.0 * np.tanh((h @ W["f"].T + W["f.b"])[:, 0] / 5.0))
    for t in range(T):
        w = np.array([np.exp(li[j] + lf[j + 1:t + 1].sum()) for j in range(t + 1)]) * (k[:t + 1] @ q[t])
        o = w @ v[:t + 1]
        o = o / np.sqrt(np.mean(o * o))                            # the norm takes the divisor's size away, not its absence of sign
        assert np.allclose(got[t], o, atol=1e-5), t


def test_scans_against_closed_forms():
    rng = np.random.default_rng(4)
    T, E = 7, 5
    h = rng.standard_normal((T, E))
    # one channel and one state entry, no convolution, no skip: y_t = C_t sum_j exp(A sum_(i in j+1..t) dt_i) dt_j x_j B_j
    W = {"in": rng.standard_normal((2, E)), "conv": np.ones((1, 1)), "conv.b": np.zeros(1), "x": rng.standard_normal((3, 1)), "dt": rng.standard_normal((1, 1)), "dt.b": np.array([0.3]),
         "A_log": np.array([[-0.4]]), "D": np.zeros(1), "o": np.eye(1)}
    got = ko.selective_scan(h, {"inner": 1, "state": 1, "dt_rank": 1, "conv": 1}, W, "", 1e-6)[:, 0]
    x = ko.silu(h @ W["in"][0])
    low, B, C = np.outer(x, W["x"][:, 0]).T
    dt = ko.softplus(low * W["dt"][0, 0] + 0.3)
    A = -np.exp(-0.4)
    for t in range(T):
        y = C[t] * sum(np.exp(A * dt[j + 1:t + 1].sum()) * dt[j] * x[j] * B[j] for j in range(t + 1))
        assert np.isclose(got[t], y * ko.silu(h[t] @ W["in"][1]))
    # mamba2 with one head: y_t = sum_j exp(-rate sum dt) dt_j (B_j . C_t) x_j + D x_t, gate before the norm
    mx = {"heads": 1, "vdim": 2, "state": 3, "groups": 1, "norm_groups": 1, "conv": 1}
    W = {"in": rng.standard_normal((2 + 8 + 1, E)), "conv": np.ones((8, 1)), "conv.b": np.zeros(8), "dt_bias": np.array([0.1]), "A_log": np.array([-1.0]), "D": np.array([0.7]),
         "norm": np.ones(2), "o": np.eye(2)}
    got = ko.mamba2(h, mx, W, "", 1e-9)
    P = h @ W["in"].T
    z, xbc, dt = P[:, :2], ko.silu(P[:, 2:10]), ko.softplus(P[:, 10] + 0.1)
    for t in range(T):
        y = sum(np.exp(-np.exp(-1.0) * dt[j + 1:t + 1].sum()) * dt[j] * (xbc[j, 2:5] @ xbc[t, 5:8]) * xbc[j, :2] for j in range(t + 1)) + 0.7 * xbc[t, :2]
        y = y * ko.silu(z[t])
        assert np.allclose(got[t], y / np.sqrt(np.mean(y * y) + 1e-9))


def test_convolution_by_hand():
    x = np.array([[1.0], [2.0], [3.0]])
    assert np.allclose(ko.short_conv(x, np.array([[10.0, 1.0]]), np.array([0.5]))[:, 0], [1.5, 12.5, 23.5])


def test_router_choice_and_weights():
    Wr = np.log(np.array([[1.0], [2.0], [3.0], [4.0]]))
    sel, w = ko.route(np.ones((1, 1)), Wr, np.array([0.4, 0.0, 0.0, 0.0]), 2)
    assert sel.tolist() == [[0, 3]] and np.allclose(w, [[0.2, 0.8]])          # chosen with the correction, weighed without
    sel, _ = ko.route(np.ones((1, 1)), np.zeros((4, 1)), np.zeros(4), 3)
    assert sel.tolist() == [[0, 1, 2]]                                          # the lowest index first among equals


def test_clamped_unit_and_identity():
    W = {"gate": np.array([[5.0]]), "up": np.array([[-5.0]]), "down": np.array([[1.0]])}
    y = ko.clamped_unit(np.ones((1, 1)), W, "", 0.5)
    assert np.isclose(y[0, 0], 0.5 * ko.sigmoid(1.702 * 0.5) * 0.5)           # (u + 1) with u = -0.5
    W["gate"] = np.array([[-5.0]])                                              # the gate has no lower clamp
    assert np.isclose(ko.clamped_unit(np.ones((1, 1)), W, "", 0.5)[0, 0], -5.0 * ko.sigmoid(-8.51) * 0.5)
    mj = {"router": {"experts": 1, "identity": 1, "top": 1}, "expert": {"limit": 1.0}}
    w = {"router": np.array([[0.0], [9.0]]), "correction": np.zeros(2)}
    assert np.allclose(ko.mixture(np.full((1, 1), 2.5), mj, w, ""), 2.5)


def test_sub_layers_read_the_residual_and_are_normed_on_the_way_out():
    cfg = config([mlstm(mlp=dense())], mult=0.25)
    w = ko.random_model(cfg, 5)
    toks = [3, 1, 4, 1, 5]
    x = w["embed"][toks] * cfg["embedding"]["scale"]
    y = ko.mlstm(x, cfg["layers"][0]["mixer"], w, "l0.mix.", cfg["norm"]["eps"])
    x = x + 0.25 * y / np.sqrt((y * y).mean(-1, keepdims=True) + cfg["norm"]["eps"]) * (1 + w["l0.norm1"])
    y = ko.dense(x, w, "l0.mlp.")
    x = x + 0.25 * y / np.sqrt((y * y).mean(-1, keepdims=True) + cfg["norm"]["eps"]) * (1 + w["l0.norm2"])
    assert np.allclose(ko.forward(cfg, w, toks)[1][0], x)


def test_model_writer_round_trips(tmp_path):
    cfg = config([par(mlp=moe()), mlstm(), ssd(mlp=dense())])
    w = ko.random_model(cfg, 3)
    d = ko.write_model(str(tmp_path / "m"), cfg, w)
    back = so.load_safetensors(d + "/model.safetensors")
    assert set(back) == set(w) == set(ko.tensor_shapes(cfg))
    for k in w:
        assert list(np.shape(back[k])) == ko.tensor_shapes(cfg)[k] and np.array_equal(np.asarray(back[k], np.float64), w[k])
