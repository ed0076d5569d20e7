"""Plain, slow restatement of the Gusedra design in numpy float64 (test infrastructure only; shares no code with the library).

A model is (cfg, W): cfg the parsed config.json, W a dict name -> float64 array.  One function per mechanism; `Sequence` carries what a
sequence keeps between calls (every attention layer's cached keys and values), so the same functions serve whole prompts, portions and
token-by-token decoding.

Notation: x the residual stream [T, width], N a LayerNorm with weight and bias.  A sublayer f adds  m * ls * N'(f(N(x)))  to x, with one
number m for the model and one vector ls per sublayer.
"""
import functools
import math

import numpy as np

from tests.rapisun_oracle import bf16_round, write_model  # noqa: F401  (helpers for writing test models)


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def softmax(z):
    e = np.exp(z - z.max())
    return e / e.sum()


# ---- the layer's frame ----------------------------------------------------------------------------------------------------------------
def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w + b


def add_sublayer(x, f, cfg, W, p, n):
    """sublayer number n ("1" the mixer, "2" the feed-forward) of the layer with prefix p"""
    eps = cfg["norm"]["eps"]
    y = f(layer_norm(x, W[p + "norm" + n], W[p + "norm%s.b" % n], eps))
    y = layer_norm(y, W[p + "norm%sb" % n], W[p + "norm%sb.b" % n], eps)
    return x + cfg["residual_mult"] * (y * W[p + "ls" + n])


# ---- attention --------------------------------------------------------------------------------------------------------------------------
def visible(i, mask):
    """the positions a token at i reads: those less than `size` behind it and the sequence's first `keep_first`, none later than i"""
    if not mask:
        return list(range(i + 1))
    return [j for j in range(i + 1) if i - j < mask["size"] or j < mask.get("keep_first", 0)]


def slope(h, H):
    return 2.0 ** (-8.0 * (h + 1) / H)


@functools.lru_cache(maxsize=None)
def bucket(n, B, D):
    """distances below B/2 one by one, then B/2 buckets whose widths grow geometrically up to distance D, the last one open"""
    half = B // 2
    if n < half:
        return n
    return min(B - 1, half + math.floor(math.log(n / half) / math.log(D / half) * (B - half)))


def softmax_with_sink(s, sink):
    """exp(s_j) / (exp(sink) + sum exp(s)), formed without overflow"""
    m = max(float(s.max()), sink)
    e = np.exp(s - m)
    return e / (math.exp(sink - m) + e.sum())


def project_kv(h, W, pre, mx, st):
    T, G = h.shape[0], mx["kv_heads"]
    k, v = (h @ W[pre + "k"].T).reshape(T, G, mx["dim"]), (h @ W[pre + "v"].T).reshape(T, G, mx["vdim"])
    st["K"] = np.concatenate([st["K"], k], 0) if "K" in st else k
    st["V"] = np.concatenate([st["V"], v], 0) if "V" in st else v


def attend(h, W, pre, mx, kv, pos, bias, weigh):
    """[T, heads, vdim]: bias(h, distances) joins the scaled scores, weigh(scores, h) makes them weights"""
    H, G, D = mx["heads"], mx["kv_heads"], mx["dim"]
    T = h.shape[0]
    q = (h @ W[pre + "q"].T).reshape(T, H, D)
    o = np.zeros((T, H, mx["vdim"]))
    for t in range(T):
        js = np.array(visible(pos[t], mx.get("mask")))
        for hh in range(H):
            g = hh // (H // G)
            s = (kv["K"][js, g] @ q[t, hh]) * mx["scale"] + bias(hh, pos[t] - js)
            o[t, hh] = weigh(s, hh) @ kv["V"][js, g]
    return o


def slope_attention(h, W, pre, mx, kv, pos):
    """scores fall linearly with the distance; a learned logit per head joins the denominator"""
    sink = W[pre + "sink"]
    o = attend(h, W, pre, mx, kv, pos, lambda hh, n: -slope(hh, mx["heads"]) * n, lambda s, hh: softmax_with_sink(s, float(sink[hh])))
    return o.reshape(h.shape[0], -1) @ W[pre + "o"].T


def bucket_attention(h, W, pre, mx, kv, pos):
    """scores get a learned number per head and distance bucket; the heads' outputs are gated value by value"""
    rel = W[pre + "rel"]
    o = attend(h, W, pre, mx, kv, pos, lambda hh, n: np.array([rel[bucket(int(d), rel.shape[0], mx["bias_max"]), hh] for d in n]), lambda s, hh: softmax(s))
    return (o.reshape(h.shape[0], -1) * sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


# ---- feed-forwards ------------------------------------------------------------------------------------------------------------------------
def dense_ff(h, W, pre):
    return np.maximum(h @ W[pre + "up"].T, 0.0) ** 2 @ W[pre + "down"].T


def expert_ff(h, W, pre):
    g = h @ W[pre + "gate"].T
    return (g * sigmoid(g) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


def route(z, correction, r):
    """[(output, weight)] of one token: softmax scores; the corrected scores choose, first whole groups of neighbours by their best member,
    then the `top` best members of the kept groups; the weights are the uncorrected scores times a constant"""
    s = softmax(z)
    c = s + correction
    groups = (r.get("groups") or {}).get("count", 1)
    keep = (r.get("groups") or {}).get("keep", groups)
    per = len(z) // groups
    best = sorted(range(groups), key=lambda g: -c[g * per:(g + 1) * per].max())[:keep]
    allowed = [i for i in range(len(z)) if i // per in best]
    return [(i, s[i] * r.get("scale", 1.0)) for i in sorted(allowed, key=lambda i: -c[i])[:r["top"]]]


def expert_mixture(h, W, pre, ml):
    """the last `identity` outputs of the router pass the input on"""
    r = ml["router"]
    E = r["experts"]
    z = h @ W[pre + "router"].T
    out = expert_ff(h, W, pre + "shared.") if ml.get("shared") else np.zeros_like(h)
    for t in range(h.shape[0]):
        for i, w in route(z[t], W[pre + "correction"], r):
            out[t] += w * (expert_ff(h[t:t + 1], W, "%se%d." % (pre, i))[0] if i < E else h[t])
    return out


# ---- the model --------------------------------------------------------------------------------------------------------------------------
class Sequence:
    def __init__(self, cfg):
        self.n = 0
        self.kv = [dict() for _ in cfg["layers"]]


def mixer(h, cfg, W, il, seq, pos):
    jl = cfg["layers"][il]
    mx, pre, src = jl["mixer"], "l%d.mix." % il, jl["mixer"].get("kv_from")
    if src is None:
        project_kv(h, W, pre, mx, seq.kv[il])
        src = il
    f = {"attention": slope_attention, "attention_2": bucket_attention}[jl["type"]]
    return f(h, W, pre, mx, seq.kv[src], pos)


def forward(cfg, W, seq, tokens, trace=None):
    """logits [T, vocab] of the next `tokens` of the sequence; trace (a list) receives x as each layer leaves it"""
    pos = list(range(seq.n, seq.n + len(tokens)))
    x = W["embed"][np.asarray(tokens)]
    for il, jl in enumerate(cfg["layers"]):
        p, ml = "l%d." % il, jl.get("mlp")
        x = add_sublayer(x, lambda h: mixer(h, cfg, W, il, seq, pos), cfg, W, p, "1")
        if ml:
            ff = (lambda h: expert_mixture(h, W, p + "mlp.", ml)) if ml["kind"] == "moe" else (lambda h: dense_ff(h, W, p + "mlp."))
            x = add_sublayer(x, ff, cfg, W, p, "2")
        if trace is not None:
            trace.append(x.copy())
    seq.n += len(tokens)
    return layer_norm(x, W["final.norm"], W["final.norm.b"], cfg["norm"]["eps"]) @ W["head"].T


# ---- test models --------------------------------------------------------------------------------------------------------------------------
def tensor_shapes(cfg, buckets=8):
    """name -> shape of every tensor a model of this configuration holds; `buckets`: rows of the bucket tables"""
    Wd, s = cfg["width"], {}
    s["embed"] = (cfg["vocab"], Wd)
    s["head"] = (cfg["vocab"], Wd)
    s["final.norm"] = s["final.norm.b"] = (Wd,)
    for i, jl in enumerate(cfg["layers"]):
        p, mx, ml = "l%d." % i, jl["mixer"], jl.get("mlp")
        H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        for n in ("1", "2") if ml else ("1",):
            for t in ("norm" + n, "norm%s.b" % n, "norm%sb" % n, "norm%sb.b" % n, "ls" + n):
                s[p + t] = (Wd,)
        q = p + "mix."
        s.update({q + "q": (H * D, Wd), q + "o": (Wd, H * V)})
        if mx.get("kv_from") is None:
            s.update({q + "k": (G * D, Wd), q + "v": (G * V, Wd)})
        if jl["type"] == "attention":
            s[q + "sink"] = (H,)
        else:
            s.update({q + "rel": (mx.get("buckets", buckets), H), q + "g": (H * V, Wd)})
        q = p + "mlp."
        if ml and ml["kind"] == "dense":
            s.update({q + "up": (ml["ff"], Wd), q + "down": (Wd, ml["ff"])})
        elif ml:
            R = ml["router"]["experts"] + ml["router"].get("identity", 0)
            s.update({q + "router": (R, Wd), q + "correction": (R,)})
            parts = [("e%d." % e, ml["expert"]["ff"]) for e in range(ml["router"]["experts"])] + ([("shared.", ml["shared"]["ff"])] if ml.get("shared") else [])
            for e, F in parts:
                s.update({q + e + "gate": (F, Wd), q + e + "up": (F, Wd), q + e + "down": (Wd, F)})
    return s


def random_weights(cfg, seed):
    """bfloat16-representable random weights, float64"""
    rng = np.random.default_rng(seed)
    W = {}
    for name, s in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last == "b":
            w = 0.2 * rng.standard_normal(s)
        elif "norm" in last or last.startswith("ls"):
            w = 1.0 + 0.25 * rng.standard_normal(s)
        elif last == "sink":
            w = rng.uniform(-1.0, 2.0, s)
        elif last == "rel":
            w = rng.standard_normal(s)
        elif last == "correction":
            w = 0.15 * rng.standard_normal(s)
        elif name == "embed":
            w = rng.standard_normal(s)
        else:
            w = rng.standard_normal(s) * (1.4 / math.sqrt(s[-1]))
        W[name] = bf16_round(w)
    return W
