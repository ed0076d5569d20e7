"""CPU: the float64 restatement of the Gusedra design agrees with itself over cuts (whole prompt, portions, token by token) for every test
configuration, and its parts do what their definitions say on inputs whose answer is known."""
import math

import numpy as np
import pytest

from tests import gusedra_oracle as O
from tests.gusedra_configs import CONFIGS, buckets, drawn, slopes


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


def test_layer_norm_uses_the_mean_of_squared_deviations():
    y = O.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 2.0]), np.array([10.0, 20.0]), 3.0)
    assert np.allclose(y, [[10.0 - 1.0, 20.0 + 1.0]])              # deviations -1, 1; sqrt(1 + 3) = 2


def test_sublayer_is_normed_before_and_behind_and_scaled():
    cfg = {"norm": {"eps": 0.0}, "residual_mult": 0.5}
    W = {"norm1": np.ones(2), "norm1.b": np.zeros(2), "norm1b": np.ones(2), "norm1b.b": np.array([0.0, 1.0]), "ls1": np.array([4.0, 8.0])}
    seen = []
    x = O.add_sublayer(np.array([[7.0, 9.0]]), lambda h: seen.append(h) or np.array([[100.0, 300.0]]), cfg, W, "", "1")
    assert np.allclose(seen[0], [[-1.0, 1.0]])
    assert np.allclose(x, [[7.0 + 0.5 * 4.0 * -1.0, 9.0 + 0.5 * 8.0 * 2.0]])


def test_visible_positions():
    assert O.visible(0, {"size": 3}) == [0]
    assert O.visible(9, {"size": 3, "keep_first": 2}) == [0, 1, 7, 8, 9]       # 6 is three away and outside, the first two stay
    assert O.visible(4, {"size": 3, "keep_first": 2}) == [0, 1, 2, 3, 4]
    assert O.visible(5, {"size": 1}) == [5]
    assert O.visible(3, {"size": 2, "keep_first": 100}) == [0, 1, 2, 3]
    assert O.visible(3, None) == [0, 1, 2, 3]


def test_slopes():
    assert [O.slope(h, 8) for h in range(8)] == [2.0 ** -(h + 1) for h in range(8)]
    assert O.slope(5, 6) == 2.0 ** -8 and np.isclose(O.slope(0, 3), 2.0 ** (-8.0 / 3.0))


def test_buckets():
    assert [O.bucket(n, 8, 64) for n in range(4)] == [0, 1, 2, 3]
    # half = 4, factors of 64 / 4 = 16 in four buckets: borders at 4, 8, 16, 32
    assert [O.bucket(n, 8, 64) for n in (4, 7, 8, 15, 16, 31, 32, 63, 64, 10 ** 6)] == [4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    b = [O.bucket(n, 20, 90) for n in range(200)]
    assert b[:10] == list(range(10)) and b == sorted(b) and b[-1] == 19 and b[89] == 19 and b[10] == 10


def test_sink_counts_once_and_carries_no_value():
    p = O.softmax_with_sink(np.array([0.0, 0.0]), math.log(2.0))
    assert np.allclose(p, 0.25)
    assert np.allclose(O.softmax_with_sink(np.array([-800.0]), 0.0), 0.0) and np.allclose(O.softmax_with_sink(np.array([800.0, 0.0]), 0.0), [1.0, 0.0])


def test_slope_attention_by_hand():
    """two keys with score 0: the nearer one ahead by one slope, the sink behind"""
    mx = slopes(1, 1, 1, 1, scale=1.0)[1]
    W = {"q": np.zeros((1, 1)), "o": np.ones((1, 1)), "sink": np.array([0.3])}
    kv = {"K": np.ones((2, 1, 1)), "V": np.array([[[5.0]], [[7.0]]])}
    s = 2.0 ** -8
    d = math.exp(0.3) + 1.0 + math.exp(-s)
    assert np.isclose(O.slope_attention(np.ones((1, 1)), W, "", mx, kv, [1])[0, 0], (7.0 + 5.0 * math.exp(-s)) / d)


def test_bucket_attention_by_hand():
    """the bias is not scaled; the gate multiplies value by value before the output matrix"""
    mx = buckets(1, 1, 1, 2, n=4, reach=8, scale=100.0)[1]
    W = {"q": np.zeros((1, 1)), "o": np.array([[1.0, 10.0]]), "rel": np.array([[0.0], [math.log(3.0)], [0.0], [0.0]]), "g": np.array([[0.0], [math.log(3.0)]])}
    kv = {"K": np.ones((2, 1, 1)), "V": np.array([[[4.0, 8.0]], [[0.0, 4.0]]])}
    a, b = 0.75 * 4.0, 0.75 * 8.0 + 0.25 * 4.0
    assert np.isclose(O.bucket_attention(np.ones((1, 1)), W, "", mx, kv, [1])[0, 0], 0.5 * a + 0.75 * 10.0 * b)


def test_routing():
    r = {"top": 2, "scale": 3.0}
    z = np.log(np.array([0.1, 0.2, 0.3, 0.4]))
    got = O.route(z, np.zeros(4), r)
    assert [i for i, _ in got] == [3, 2] and np.allclose([w for _, w in got], [1.2, 0.9])
    got = O.route(z, np.array([0.5, 0.0, 0.0, 0.0]), r)            # the correction chooses and does not weigh
    assert [i for i, _ in got] == [0, 3] and np.allclose([w for _, w in got], [0.3, 1.2])
    got = O.route(z, np.array([0.5, -9.0, 0.0, 0.0]), dict(r, groups={"count": 2, "keep": 1}))
    assert [i for i, _ in got] == [0, 1]                           # a bad neighbour is still a member of the best group, and what is outside it is not


def test_identity_outputs_pass_the_input_on():
    ml = {"router": {"experts": 1, "top": 2, "scale": 2.0, "identity": 1}, "expert": {"ff": 1}}
    W = {"router": np.zeros((2, 2)), "correction": np.zeros(2), "e0.gate": np.array([[1.0, 0.0]]), "e0.up": np.array([[0.0, 1.0]]), "e0.down": np.array([[1.0], [2.0]])}
    h = np.array([[1.0, 3.0]])
    e = 3.0 / (1.0 + math.exp(-1.0))
    assert np.allclose(O.expert_mixture(h, W, "", ml), [[e + 1.0, 2.0 * e + 3.0]])


def test_a_later_layer_reads_an_earlier_layers_cells():
    cfg = CONFIGS["shared_cells"]()
    W = O.random_weights(cfg, 4)
    seq = O.Sequence(cfg)
    O.forward(cfg, W, seq, [1, 2, 3])
    assert ["K" in k for k in seq.kv] == [True, False, True, False, False] and "l1.mix.k" not in W


def test_dense_feed_forward_squares_what_is_positive():
    W = {"up": np.array([[1.0], [-1.0]]), "down": np.array([[1.0, 100.0]])}
    assert np.allclose(O.dense_ff(np.array([[3.0], [-2.0]]), W, ""), [[9.0], [400.0]])
