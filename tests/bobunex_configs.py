"""Small Bobunex configurations for the tests (sizes chosen to differ from each other: heads, key / value heads, head and value sizes of
both branches, windows, kept tokens, rotated dimensions with and without scaled frequencies, caps, taps)."""
import math


def bands(factor, original, low=1.0, high=4.0):
    return {"factor": factor, "low": low, "high": high, "original": original}


def left(heads, kv_heads, dim, vdim, window, keep, rot_dims, softcap=20.0, base=10000.0, scaling=None, scale=None):
    rot = {"base": base, "dims": rot_dims}
    if scaling:
        rot["scaling"] = scaling
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window, "keep_first": keep}, "rot": rot, "softcap": softcap,
            "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}


def right(heads, dim, vdim, cap=15.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def model(width, vocab, layers, taps=4, eps=1e-5, embed_scale=2.0):
    """layers: [(left, right, ff or None)]"""
    return {"architecture": "Bobunex", "width": width, "vocab": vocab, "canon": {"taps": taps}, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "layers": [{"type": "parallel", "mixer": {"left": a, "right": b}, "mlp": {"kind": "dense", "ff": ff} if ff else None} for a, b, ff in layers]}


def mixed_small():
    """three unlike layers, the middle one without feed-forward; odd sizes, windows shorter and longer than the prompts"""
    return model(72, 170, [(left(4, 2, 12, 10, 9, 3, 8, scaling=bands(3.0, 60)), right(3, 8, 14), 90),
                           (left(3, 1, 10, 14, 16, 5, 10, softcap=6.0, base=300.0), right(2, 17, 9, cap=4.0), None),
                           (left(2, 2, 20, 7, 64, 2, 4, scale=0.5), right(5, 6, 12), 52)], taps=3)


def attention_only():
    """what the logits show most is the attention: large scores, tight caps, short windows, no feed-forward"""
    return model(64, 120, [(left(4, 2, 16, 12, 7, 2, 16, softcap=3.0, base=50.0, scale=1.0), right(1, 4, 4), None),
                           (left(6, 3, 12, 20, 12, 4, 6, softcap=8.0, base=100.0, scaling=bands(8.0, 40, low=0.5, high=3.0), scale=0.8), right(1, 4, 4), None)])


def memory_only():
    """what the logits show most is the matrix memory: several heads, more states than a warp, uneven value sizes"""
    return model(48, 100, [(left(1, 1, 4, 4, 4, 0, 0), right(6, 24, 8), None), (left(1, 1, 4, 4, 4, 1, 2), right(3, 33, 25, cap=2.0), 40)], taps=2)


def memory_wide():
    """memories whose long portions run as matmuls in served mode, beside a small attention"""
    return model(64, 110, [(left(1, 1, 8, 8, 5, 1, 4), right(3, 24, 20), 48), (left(1, 1, 8, 8, 5, 0, 0), right(2, 64, 33, cap=8.0), None)])


def deep_memory():
    """one memory with more rows than the other recurrences take, rows not a multiple of anything"""
    return model(40, 60, [(left(1, 1, 8, 8, 4, 1, 0), right(1, 301, 12), 24), (left(1, 1, 8, 8, 4, 1, 0), right(2, 264, 20), None)], taps=5)


def ones():
    """values that happen to be 1 or equal: one head, one state, one tap, window 1, nothing kept, nothing rotated, factors of 1"""
    return model(32, 40, [(left(1, 1, 1, 1, 1, 0, 0, scale=1.0, softcap=1.0), right(1, 1, 1, cap=1.0), 1),
                          (left(1, 1, 8, 8, 8, 8, 8, scaling=bands(1.0, 16)), right(1, 8, 8), 32),
                          (left(2, 2, 8, 8, 1, 1, 2, scaling=bands(2.0, 16, low=2.0, high=2.0)), right(2, 8, 8), None)], taps=1, embed_scale=1.0)


def far_keys():
    """a window of 50 with 4 kept tokens over prompts of hundreds, peaky softmaxes"""
    return model(64, 300, [(left(2, 1, 24, 16, 50, 4, 12, softcap=30.0, scale=1.2), right(2, 8, 8), None),
                           (left(4, 2, 8, 8, 110, 9, 8, softcap=15.0, scale=1.5), right(2, 8, 8), None)])


def wide_heads():
    """head sizes that are multiples of 8: in served mode long portions take the tensor-core (matmul) form of the attention"""
    return model(64, 160, [(left(4, 2, 32, 16, 70, 5, 16, scaling=bands(2.0, 128)), right(2, 16, 16), 96),
                           (left(8, 2, 16, 24, 300, 12, 8), right(4, 32, 24), 64),
                           (left(2, 1, 16, 16, 33, 0, 16, softcap=4.0), right(2, 64, 32), None)])


def medium():
    """wider layers: more query heads per key head, larger memories"""
    return model(128, 500, [(left(8, 2, 32, 24, 100, 6, 16, base=50000.0, scaling=bands(4.0, 256)), right(4, 32, 48), 200),
                            (left(6, 3, 40, 48, 40, 1, 40, softcap=10.0), right(2, 128, 64), 160),
                            (left(4, 4, 24, 32, 150, 17, 12), right(8, 16, 16, cap=6.0), None)])


def drawn(seed):
    """a configuration drawn from a seed: every size and constant varies"""
    import numpy as np
    r = np.random.default_rng(seed)
    pick = lambda xs: xs[int(r.integers(0, len(xs)))]
    layers = []
    for _ in range(int(r.integers(1, 5))):
        kv, rep, dim = pick([1, 2, 3]), pick([1, 2, 4]), pick([4, 6, 8, 16, 24, 40])
        rd = pick([0, 2, dim // 2 // 2 * 2, dim])
        lo = float(pick([0.5, 1.0, 2.0]))
        sc = bands(float(pick([1.5, 4.0, 16.0])), pick([16, 64, 512, 4096]), low=lo, high=lo * float(pick([1.5, 4.0]))) if rd and r.random() < 0.6 else None
        a = left(kv * rep, kv, dim, pick([3, 8, 12, 16, 40]), pick([1, 2, 5, 17, 64, 131, 1000]), pick([0, 1, 3, 8, 70]), rd, softcap=float(pick([2.0, 10.0, 50.0])),
                 base=pick([100.0, 10000.0, 1e6]), scaling=sc, scale=float(r.uniform(0.5, 2.0)) / math.sqrt(dim))
        b = right(pick([1, 2, 3, 5]), pick([1, 4, 7, 16, 40, 72]), pick([8, 9, 16, 40, 65]), cap=float(pick([1.0, 5.0, 15.0])))
        layers.append((a, b, pick([16, 50, 129]) if r.random() < 0.7 else None))
    return model(pick([24, 40, 53, 96, 136]), int(r.integers(30, 400)), layers, taps=int(r.integers(1, 7)), eps=pick([1e-6, 1e-5, 1e-3]), embed_scale=float(pick([1.0, 0.5, 7.5])))


CONFIGS = {f.__name__: f for f in (mixed_small, attention_only, memory_only, memory_wide, deep_memory, ones, far_keys, wide_heads, medium)}
