"""Small Gusedra configurations for the tests (sizes chosen to differ from each other: heads, key / value heads, head and value sizes, windows,
kept tokens, buckets and their reach, shared caches, experts, groups, identity outputs, widths that are no multiple of four)."""
import math


def slopes(heads, kv_heads, dim, vdim, window=None, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def buckets(heads, kv_heads, dim, vdim, window=None, keep=0, n=8, reach=40, scale=None, kv_from=None):
    """n: rows of the bucket table (what the tests draw its shape from; the library reads the tensor's)"""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.0 / math.sqrt(dim), "bias_max": reach, "buckets": n}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention_2", m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, groups=None, scale=1.0, shared=None):
    r = {"experts": experts, "top": top, "scale": scale, "identity": identity}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "router": r, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def model(width, vocab, layers, eps=1e-5, mult=0.5):
    """layers: [((type, mixer), feed-forward or None)]"""
    return {"architecture": "Gusedra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": [{"type": a[0], "mixer": a[1], "mlp": ml} for a, ml in layers]}


def mixed_small():
    """six unlike layers: both mixers, every kind of feed-forward and none, cells read by a later layer with another window, scale and query-head count"""
    return model(72, 170, [(slopes(6, 2, 12, 10, 9), dense(90)), (buckets(3, 1, 10, 14, 16, 5), moe(6, 3, 20, identity=3, groups=(3, 2), scale=1.7, shared=28)),
                           (slopes(4, 2, 12, 10, 14, scale=0.5, kv_from=0), None), (buckets(2, 2, 20, 7, 7, 2, n=6, reach=11), moe(5, 2, 12, scale=0.8)),
                           (slopes(5, 5, 8, 9, 64), moe(4, 4, 16, identity=2, shared=8)), (buckets(4, 2, 6, 8, 30, 3, n=4, reach=5, kv_from=None), dense(33))], mult=0.7)


def slope_only():
    """what the logits show most is the attention with slopes: large scores, short windows, heads that are no power of two, a layer without a window"""
    return model(64, 120, [(slopes(4, 2, 16, 12, 7, scale=0.8), None), (slopes(6, 3, 12, 20, 12, scale=0.6), None), (slopes(3, 1, 8, 8, scale=0.7), None)], mult=1.0)


def bucket_only():
    """the same for the attention with buckets: more buckets than the window is long, fewer, borders that fall on whole numbers, no window, no kept tokens"""
    return model(60, 110, [(buckets(4, 2, 16, 12, 9, 3, n=16, reach=64, scale=0.5), None), (buckets(3, 3, 8, 16, 20, 0, n=8, reach=64, scale=0.5), None),
                           (buckets(2, 1, 10, 10, n=10, reach=29, scale=0.5), None)], mult=1.0)


def experts_only():
    """what the logits show most are the mixtures: one group, many groups, identity outputs in their own group, all experts chosen, a width that is no multiple of four"""
    a = slopes(1, 1, 4, 4, 3)
    return model(50, 90, [(a, moe(9, 3, 24, identity=3, groups=(4, 2), scale=2.0, shared=10)), (a, moe(4, 2, 18, groups=(2, 1))), (a, moe(3, 5, 11, identity=2, scale=0.5, shared=7)),
                          (a, moe(40, 6, 9, identity=8, groups=(6, 3), scale=1.5))], mult=1.0)


def shared_cells():
    """one cache read by several layers, with and without a window, beside layers with their own"""
    return model(48, 100, [(slopes(4, 2, 8, 8, 20), dense(40)), (slopes(2, 2, 8, 8, kv_from=0), dense(24)), (buckets(4, 4, 8, 12, 10, 2), None), (slopes(8, 2, 8, 8, 5, kv_from=0), None),
                           (buckets(8, 4, 8, 12, 25, 1, kv_from=2), moe(4, 2, 16, shared=16))])


def ones():
    """values that happen to be 1 or equal: one head of one coordinate, a window of 1, one bucket above the first, one expert, one group"""
    return model(32, 40, [(slopes(1, 1, 1, 1, 1, scale=1.0), dense(1)), (buckets(1, 1, 8, 8, 1, 1, n=2, reach=2, scale=1.0), moe(1, 1, 32, groups=(1, 1))),
                          (slopes(2, 2, 8, 8, 8), moe(2, 1, 1, identity=1, groups=(3, 1), shared=1)), (buckets(2, 1, 8, 8, 8, 8, n=32, reach=17), None)], mult=1.0)


def far_keys():
    """windows over prompts of hundreds of tokens, kept first tokens, buckets that reach beyond the window"""
    return model(64, 300, [(slopes(2, 1, 24, 16, 50, scale=0.8), None), (buckets(4, 2, 8, 8, 80, 6, n=16, reach=300, scale=0.8), dense(50))], mult=1.0)


def wide_heads():
    """head sizes that are multiples of 8: in served mode long portions take the tensor-core (matmul) form of the attention"""
    return model(64, 160, [(slopes(4, 2, 32, 16, 70), moe(8, 3, 48, identity=4, groups=(2, 1), scale=1.3, shared=32)), (buckets(8, 2, 16, 24, 300, 12, n=20, reach=150), dense(96)),
                           (slopes(8, 2, 32, 16, 150, kv_from=0), moe(4, 2, 40)), (buckets(2, 1, 16, 16, 33, 3), None)])


def medium():
    """wider layers: more query heads per key head, larger experts, rows that TMA takes"""
    return model(128, 500, [(slopes(8, 2, 32, 24, 100), dense(200)), (buckets(6, 3, 40, 48, 60, 4, n=32, reach=128), moe(12, 4, 64, identity=4, groups=(4, 2), scale=2.5, shared=96)),
                            (slopes(4, 2, 32, 24, 40, kv_from=0), moe(6, 2, 56, shared=40))], mult=0.4)


def big_heads():
    """heads of up to 128 coordinates, value sizes unlike them, groups of three query heads, many rows per key: the tensor-core attention's widest tiles"""
    return model(64, 150, [(slopes(2, 1, 128, 128, 100), None), (buckets(3, 1, 96, 80, 170, 7, n=24, reach=200), dense(40)), (slopes(4, 4, 72, 40, scale=0.15), None),
                           (buckets(12, 4, 120, 8, 64, 130, n=12, reach=90, scale=0.12), None)], mult=0.6)


def drawn(seed):
    """a configuration drawn from a seed: every size and constant varies"""
    import numpy as np
    r = np.random.default_rng(seed)
    pick = lambda xs: xs[int(r.integers(0, len(xs)))]
    layers = []
    for i in range(int(r.integers(1, 6))):
        kv, rep, dim, vdim = pick([1, 2, 3]), pick([1, 2, 4]), pick([4, 6, 8, 16, 24, 40]), pick([3, 8, 12, 16, 40])
        window, scale, src = pick([1, 2, 5, 17, 64, 131, 1000, None]), float(r.uniform(0.4, 1.5)) / math.sqrt(dim), None
        kind = pick(["attention", "attention_2"])
        own = [j for j, (a, _) in enumerate(layers) if a[0] == kind and a[1].get("kv_from") is None]
        if own and r.random() < 0.4:
            src = pick(own)
            m = layers[src][0][1]
            kv, dim, vdim = m["kv_heads"], m["dim"], m["vdim"]
        if kind == "attention":
            a = slopes(kv * rep, kv, dim, vdim, window, scale, src)
        else:
            n = 2 * int(r.integers(1, 17))
            a = buckets(kv * rep, kv, dim, vdim, window, pick([0, 1, 3, 8, 70]), n=n, reach=n // 2 + int(r.integers(1, 200)), scale=scale, kv_from=src)
        ml = None
        if r.random() < 0.5:
            g = pick([1, 1, 2, 3, 4])
            per, keep = int(r.integers(2, 6)), int(r.integers(1, g + 1))
            ident = int(r.integers(0, per))
            ml = moe(g * per - ident, int(r.integers(1, min(keep * per, 6) + 1)), pick([8, 15, 24, 40]), identity=ident, groups=pick([(g, keep), (g, keep), None]) if g == 1 else (g, keep),
                     scale=float(pick([0.5, 1.0, 2.5])), shared=pick([None, 16, 21]))
        elif r.random() < 0.6:
            ml = dense(pick([16, 50, 129]))
        layers.append((a, ml))
    return model(pick([24, 40, 53, 96, 136]), int(r.integers(30, 400)), layers, eps=pick([1e-6, 1e-5, 1e-3]), mult=float(pick([0.2, 0.5, 1.0])))


CONFIGS = {f.__name__: f for f in (mixed_small, slope_only, bucket_only, experts_only, shared_cells, ones, far_keys, wide_heads, big_heads, medium)}
