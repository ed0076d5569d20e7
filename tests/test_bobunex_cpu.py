"""CPU: the float64 restatement of the Bobunex design agrees with itself over cuts (whole prompt, portions, token by token) for every test
configuration, and its parts do what their definitions say on inputs whose answer is known."""
import math

import numpy as np
import pytest

from tests import bobunex_oracle as O
from tests.bobunex_configs import CONFIGS, bands, drawn, left, right


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_oracle_cuts_agree(name):
    cfg = CONFIGS[name]()
    W = O.random_weights(cfg, 3)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 23).tolist()
    whole = O.forward(cfg, W, O.Sequence(cfg), toks)
    assert whole.shape == (23, cfg["vocab"]) and np.isfinite(whole).all()
    for cuts in ([1], range(1, 23), [2, 4, 5, 12, 14, 21]):
        seq, out, a = O.Sequence(cfg), [], 0
        for b in list(cuts) + [23]:
            out.append(O.forward(cfg, W, seq, toks[a:b]))
            a = b
        assert np.abs(np.concatenate(out) - whole).max() < 1e-9


def test_drawn_configurations_are_well_formed():
    for seed in range(40):
        cfg = drawn(seed)
        W = O.random_weights(cfg, seed)
        lg = O.forward(cfg, W, O.Sequence(cfg), [1, 2, 3])
        assert lg.shape == (3, cfg["vocab"]) and np.isfinite(lg).all()


def test_input_convolution_adds_its_input_and_ends_on_the_current_token():
    h = np.array([[1.0], [10.0], [100.0]])
    st = {}
    assert np.allclose(O.input_conv(h, np.array([[0.0, 0.0, 2.0]]), st, "t")[:, 0], [3.0, 30.0, 300.0])
    assert np.allclose(st["t"], [[10.0], [100.0]])
    assert np.allclose(O.input_conv(h, np.array([[1.0, 0.0, 0.0]]), {}, "t")[:, 0], [1.0, 10.0, 101.0])
    assert np.allclose(O.input_conv(h, np.array([[1.0, 0.0, 0.0]]), st, "t")[:, 0], [11.0, 110.0, 101.0])


def test_residual_gate_and_gelu():
    assert np.allclose(O.residual_gate(np.zeros((1, 2)), np.eye(2), np.array([0.0, math.log(3.0)])), [[0.5, 0.75]])
    z = np.array([-3.0, 0.0, 1.0, 10.0])
    exact = np.array([0.5 * v * (1.0 + math.erf(v / math.sqrt(2.0))) for v in z])
    assert np.abs(O.gelu_tanh(z) - exact).max() < 1e-3 and O.gelu_tanh(z)[3] == pytest.approx(10.0)


def test_visible_positions():
    assert O.visible(0, 3, 2) == [0]
    assert O.visible(2, 3, 2) == [0, 1, 2]
    assert O.visible(9, 3, 2) == [0, 1, 7, 8, 9]               # 6 is three away and outside, the first two stay
    assert O.visible(4, 3, 2) == [0, 1, 2, 3, 4]
    assert O.visible(5, 1, 0) == [5]
    assert O.visible(3, 2, 100) == [0, 1, 2, 3]


def test_capped_scores_and_the_zero_sink():
    assert O.capped(np.array([0.0, 1e6, -1e6]), 5.0).tolist() == [0.0, 5.0, -5.0]
    p = O.softmax_with_zero_sink(np.array([0.0, 0.0, 0.0]))
    assert np.allclose(p, 0.25)                                # the sink takes a share
    assert np.allclose(O.softmax_with_zero_sink(np.array([-800.0])), 0.0)
    assert np.allclose(O.softmax_with_zero_sink(np.array([800.0, 0.0])), [1.0, 0.0])


def test_rotation_half_pairs_first_dims_only():
    v = np.arange(1.0, 9.0).reshape(1, 1, 8)
    r = O.rotate_half(v, [1], {"base": 100.0, "dims": 4})
    a0, a1 = 1.0, 100.0 ** -0.5
    assert np.allclose(r[0, 0, 4:], v[0, 0, 4:])
    assert np.allclose(r[0, 0, :4], [1 * np.cos(a0) - 3 * np.sin(a0), 2 * np.cos(a1) - 4 * np.sin(a1), 3 * np.cos(a0) + 1 * np.sin(a0), 4 * np.cos(a1) + 2 * np.sin(a1)])


def test_frequency_bands():
    """frequencies 1, 10^-0.5, 10^-1, ...: over 100 positions they turn 15.9, 5.03, 1.59, 0.503, ... times"""
    f = O.rot_frequencies({"base": 100.0, "dims": 8, "scaling": bands(8.0, 100, low=1.0, high=4.0)})
    plain = 100.0 ** (-np.arange(4) / 4.0)
    assert np.allclose(f[:2], plain[:2]) and np.allclose(f[3], plain[3] / 8.0)
    s = (100.0 * plain[2] / (2 * math.pi) - 1.0) / 3.0
    assert np.isclose(f[2], plain[2] * ((1 - s) / 8.0 + s)) and plain[2] / 8.0 < f[2] < plain[2]


def test_query_norm_spans_all_heads():
    """one root mean square over both heads: a head of small rows stays small beside a head of large ones"""
    mx = left(2, 1, 2, 1, 4, 0, 0, softcap=1e6, scale=1.0)
    W = {"q": np.array([[1.0], [1.0], [100.0], [100.0]]), "k": np.ones((2, 1)), "v": np.ones((1, 1)), "q.norm": np.ones(4), "k.norm": np.ones(2),
         "g": np.full((2, 1), 1e3), "o": np.eye(2)}
    out = O.window_attention(np.ones((1, 1)), W, "", mx, 0.0, {}, [0])
    rms = math.sqrt((2 * 1.0 + 2 * 1e4) / 4)
    want = [1.0 / (1.0 + math.exp(-2.0 / rms)), 1.0 / (1.0 + math.exp(-200.0 / rms))]       # one key, value 1: exp(s) / (1 + exp(s))
    assert np.allclose(out[0], want)


def test_memory_scan_two_steps_by_hand():
    q = np.ones((2, 1, 1))
    k = np.array([[[2.0]], [[3.0]]])
    v = np.array([[[5.0]], [[7.0]]])
    i, f = np.array([[1.0], [-2.0]]), np.array([[-0.5], [-0.25]])
    st = {}
    o = O.memory_scan(q, k, v, i, f, st)
    # m: max(-0.5 + 0, 1) = 1, then max(0.75, -2) = 0.75
    n1, S1 = 2.0, 10.0
    keep, write = 1.0, math.exp(-2.75)
    n2, S2 = keep * n1 + write * 3.0, keep * S1 + write * 21.0
    assert np.allclose(o[:, 0, 0], [S1 / (max(n1, math.exp(-1.0)) + 1e-6), S2 / (max(n2, math.exp(-0.75)) + 1e-6)])
    assert np.allclose(st["m"], 0.75) and np.allclose(st["n"], n2) and np.allclose(st["S"], S2)


def test_memory_maximum_starts_at_zero():
    """a weak first write leaves m at log f, not at the input gate: the denominator's floor e^-m shows it"""
    st = {}
    o = O.memory_scan(np.ones((1, 1, 1)), np.ones((1, 1, 1)), np.ones((1, 1, 1)), np.array([[-6.0]]), np.array([[-0.1]]), st)
    assert np.allclose(st["m"], -0.1)
    w = math.exp(-6.0 + 0.1)
    assert np.isclose(o[0, 0, 0], w / (math.exp(0.1) + 1e-6))


def test_branches_are_normed_apart_and_averaged():
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 5)
    mx, eps, h = cfg["layers"][0]["mixer"], 1e-5, np.random.default_rng(2).standard_normal((4, cfg["width"]))
    a = O.window_attention(h, W, "l0.mix.left.", mx["left"], eps, {}, range(4))
    b = O.matrix_memory(h, W, "l0.mix.right.", mx["right"], eps, {})
    both = O.two_branches(h, W, "l0.mix.", mx, eps, {}, range(4))
    assert np.allclose(both, 0.5 * (O.rms_unit(a, eps) * W["l0.mix.left.out"] + O.rms_unit(b, eps) * W["l0.mix.right.out"]))
    W2 = dict(W, **{"l0.mix.right.o": W["l0.mix.right.o"] * 64.0})          # the norm takes a branch's size out
    assert np.abs(O.two_branches(h, W2, "l0.mix.", mx, eps, {}, range(4)) - both).max() < 1e-3


def test_gate_logits_are_capped():
    mx = right(1, 2, 2, cap=2.0)
    W = {"q": np.ones((2, 1)), "k": np.ones((2, 1)), "v": np.ones((2, 1)), "i": np.array([[1e4]]), "i.b": np.zeros(1), "f": np.array([[-1e4]]), "f.b": np.zeros(1),
         "norm": np.ones(2), "g": np.zeros((2, 1)), "o": np.eye(2)}
    st = {}
    O.matrix_memory(np.ones((1, 1)), W, "", mx, 1e-5, st)
    assert np.allclose(st["m"], 2.0)
    assert np.isclose(O.log_sigmoid(np.array(-2.0)), math.log(1.0 / (1.0 + math.exp(2.0))))
