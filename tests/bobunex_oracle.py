"""Plain, slow restatement of the Bobunex design in numpy float64 (test infrastructure only; shares no code with the library).

A model is (cfg, W): cfg the parsed config.json, W a dict name -> float64 array.  One function per mechanism; `Sequence` carries what a
sequence keeps between calls (the input convolutions' tails, cached keys and values, the matrix memory with its normaliser and running
maximum), so the same functions serve whole prompts, portions and token-by-token decoding.

Notation: x the residual stream [T, width], N an RMS norm with a plain weight, C the input convolution (per channel, causal, its input
added).  A sublayer f adds  f(C(N(x))) * sigmoid(R N(x) + r)  to x.
"""
import math

import numpy as np

from tests.rapisun_oracle import bf16_round, write_model  # noqa: F401  (helpers for writing test models)


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


# ---- the layer's frame ----------------------------------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def input_conv(h, w, st, key):
    """h + causal per-channel convolution of h; w [width, taps], the last column on the current token; a fresh sequence has a tail of zeros"""
    taps = w.shape[1]
    ext = np.concatenate([st.get(key, np.zeros((taps - 1, h.shape[1]))), h], 0)
    out = h.copy()
    for t in range(h.shape[0]):
        for j in range(taps):
            out[t] += w[:, j] * ext[t + j]
    st[key] = ext[ext.shape[0] - (taps - 1):].copy()
    return out


def residual_gate(h, R, r):
    return sigmoid(h @ R.T + r)


def gelu_glu_ff(h, W, pre):
    return (gelu_tanh(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


# ---- attention branch -------------------------------------------------------------------------------------------------------------------
def rot_frequencies(rot):
    """base^(-2 i / dims); with rot["scaling"] waves longer than original / low are slowed down by the factor, waves shorter than
    original / high stay, and those between get a mix of both"""
    dims = rot["dims"]
    out = []
    sc = rot.get("scaling")
    for i in range(dims // 2):
        f = rot["base"] ** (-2.0 * i / dims)
        if sc:
            turns = sc["original"] * f / (2.0 * math.pi)           # turns over the original context = original / wavelength
            if turns > sc["high"]:
                pass
            elif turns < sc["low"]:
                f = f / sc["factor"]
            else:
                s = (turns - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return np.array(out, np.float64)


def rotate_half(v, pos, rot):
    """v [T, heads, dim]: coordinates i and i + dims/2 turn together by pos * f_i, the rest pass"""
    half = rot["dims"] // 2
    if half == 0:
        return v.copy()
    ang = np.asarray(pos, np.float64)[:, None] * rot_frequencies(rot)
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = v.copy()
    a, b = v[..., :half], v[..., half:2 * half]
    out[..., :half] = a * c - b * s
    out[..., half:2 * half] = b * c + a * s
    return out


def visible(i, size, keep):
    """the positions a token at i reads: the last `size` ones and the first `keep` of the sequence, none later than i"""
    return [j for j in range(i + 1) if i - j < size or j < keep]


def capped(s, cap):
    return cap * np.tanh(s / cap)


def softmax_with_zero_sink(s):
    """exp(s_j) / (1 + sum exp(s)), formed without overflow"""
    m = max(float(s.max()), 0.0)
    e = np.exp(s - m)
    return e / (math.exp(-m) + e.sum())


def window_attention(h, W, pre, mx, eps, st, pos):
    H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q = rms_norm(h @ W[pre + "q"].T, W[pre + "q.norm"], eps).reshape(T, H, D)          # one norm over all heads' rows
    k = rms_norm(h @ W[pre + "k"].T, W[pre + "k.norm"], eps).reshape(T, G, D)
    v = (h @ W[pre + "v"].T).reshape(T, G, V)
    q, k = rotate_half(q, pos, mx["rot"]), rotate_half(k, pos, mx["rot"])
    st["K"] = np.concatenate([st["K"], k], 0) if "K" in st else k
    st["V"] = np.concatenate([st["V"], v], 0) if "V" in st else v
    o = np.zeros((T, H, V))
    for t in range(T):
        js = visible(pos[t], mx["mask"]["size"], mx["mask"]["keep_first"])
        for hh in range(H):
            g = hh // (H // G)
            s = capped((st["K"][js, g] @ q[t, hh]) * mx["scale"], mx["softcap"])
            o[t, hh] = softmax_with_zero_sink(s) @ st["V"][js, g]
    o = o * sigmoid(h @ W[pre + "g"].T)[:, :, None]                                     # one number per head
    return o.reshape(T, H * V) @ W[pre + "o"].T


# ---- matrix-memory branch ---------------------------------------------------------------------------------------------------------------
def memory_scan(q, k, v, i, f, st):
    """per head: m' = max(f + m, i); S <- e^(f + m - m') S + e^(i - m') k v^T and, as if v were 1, n <- e^(f + m - m') n + e^(i - m') k;
    o = S^T q / (max(|n . q|, e^-m') + 1e-6).
    q, k [T, H, D], v [T, H, V], i, f [T, H] (logarithms of the gates); S, n, m start at zero."""
    T, H, D = q.shape
    V = v.shape[2]
    if "S" not in st:
        st["S"], st["n"], st["m"] = np.zeros((H, D, V)), np.zeros((H, D)), np.zeros(H)
    S, n, m = st["S"], st["n"], st["m"]
    o = np.zeros((T, H, V))
    for t in range(T):
        for h in range(H):
            new = max(f[t, h] + m[h], i[t, h])
            keep, write = math.exp(f[t, h] + m[h] - new), math.exp(i[t, h] - new)
            S[h] = keep * S[h] + write * np.outer(k[t, h], v[t, h])
            n[h] = keep * n[h] + write * k[t, h]
            m[h] = new
            o[t, h] = S[h].T @ q[t, h] / (max(abs(float(n[h] @ q[t, h])), math.exp(-new)) + 1e-6)
    return o


def matrix_memory(h, W, pre, mx, eps, st):
    H, D, V, cap = mx["heads"], mx["dim"], mx["vdim"], mx["gate_cap"]
    T = h.shape[0]
    q = (h @ W[pre + "q"].T).reshape(T, H, D) / math.sqrt(D)
    k = (h @ W[pre + "k"].T).reshape(T, H, D)
    v = (h @ W[pre + "v"].T).reshape(T, H, V)
    i = capped(h @ W[pre + "i"].T + W[pre + "i.b"], cap)
    f = log_sigmoid(capped(h @ W[pre + "f"].T + W[pre + "f.b"], cap))
    o = rms_unit(memory_scan(q, k, v, i, f, st), eps).reshape(T, H * V)                 # each head by its own root mean square
    return (o * W[pre + "norm"] * sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def two_branches(h, W, pre, mx, eps, st, pos):
    """the mean of attention and memory, after a norm over the width of either"""
    a = window_attention(h, W, pre + "left.", mx["left"], eps, st, pos)
    b = matrix_memory(h, W, pre + "right.", mx["right"], eps, st)
    return 0.5 * (rms_norm(a, W[pre + "left.out"], eps) + rms_norm(b, W[pre + "right.out"], eps))


# ---- the model --------------------------------------------------------------------------------------------------------------------------
class Sequence:
    def __init__(self, cfg):
        self.n = 0
        self.layers = [dict() for _ in cfg["layers"]]


def layer(x, cfg, W, il, st, pos):
    jl, eps, p = cfg["layers"][il], cfg["norm"]["eps"], "l%d." % il
    h = rms_norm(x, W[p + "norm1"], eps)
    y = two_branches(input_conv(h, W[p + "canon1"], st, "tail1"), W, p + "mix.", jl["mixer"], eps, st, pos)
    x = x + y * residual_gate(h, W[p + "rg1"], W[p + "rg1.b"])
    if jl.get("mlp"):
        h = rms_norm(x, W[p + "norm2"], eps)
        y = gelu_glu_ff(input_conv(h, W[p + "canon2"], st, "tail2"), W, p + "mlp.")
        x = x + y * residual_gate(h, W[p + "rg2"], W[p + "rg2.b"])
    return x


def forward(cfg, W, seq, tokens, trace=None):
    """logits [T, vocab] of the next `tokens` of the sequence; trace (a list) receives x as each layer leaves it"""
    T = len(tokens)
    pos = list(range(seq.n, seq.n + T))
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for il, st in enumerate(seq.layers):
        x = layer(x, cfg, W, il, st, pos)
        if trace is not None:
            trace.append(x.copy())
    seq.n += T
    return rms_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].T


# ---- test models --------------------------------------------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    """name -> shape of every tensor a model of this configuration holds"""
    Wd, taps, s = cfg["width"], cfg["canon"]["taps"], {}
    s["embed"] = (cfg["vocab"], Wd)
    s["head"] = (cfg["vocab"], Wd)
    s["final.norm"] = (Wd,)
    for i, jl in enumerate(cfg["layers"]):
        p, a, b = "l%d." % i, jl["mixer"]["left"], jl["mixer"]["right"]
        H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        for n in ("1", "2") if jl.get("mlp") else ("1",):
            s.update({p + "norm" + n: (Wd,), p + "canon" + n: (Wd, taps), p + "rg" + n: (Wd, Wd), p + "rg%s.b" % n: (Wd,)})
        q = p + "mix.left."
        s.update({q + "q": (H * D, Wd), q + "k": (G * D, Wd), q + "v": (G * V, Wd), q + "q.norm": (H * D,), q + "k.norm": (G * D,), q + "g": (H, Wd),
                  q + "o": (Wd, H * V), q + "out": (Wd,)})
        H, D, V = b["heads"], b["dim"], b["vdim"]
        q = p + "mix.right."
        s.update({q + "q": (H * D, Wd), q + "k": (H * D, Wd), q + "v": (H * V, Wd), q + "g": (H * V, Wd), q + "i": (H, Wd), q + "i.b": (H,), q + "f": (H, Wd),
                  q + "f.b": (H,), q + "norm": (H * V,), q + "o": (Wd, H * V), q + "out": (Wd,)})
        if jl.get("mlp"):
            F = jl["mlp"]["ff"]
            s.update({p + "mlp.gate": (F, Wd), p + "mlp.up": (F, Wd), p + "mlp.down": (Wd, F)})
    return s


def random_weights(cfg, seed):
    """bfloat16-representable random weights, float64"""
    rng = np.random.default_rng(seed)
    W = {}
    for name, s in tensor_shapes(cfg).items():
        if "norm" in name.rsplit(".", 1)[-1] or name.endswith(".out"):
            w = 1.0 + 0.2 * rng.standard_normal(s)
            if name.endswith("q.norm") or name.endswith("k.norm"):
                w = w * 1.5                                                             # peakier scores
        elif ".canon" in name:
            w = 0.35 * rng.standard_normal(s)
        elif name.endswith("f.b"):
            w = rng.uniform(-1.0, 5.0, s)                                               # some heads forget at once, some hold on for hundreds of tokens
        elif name.endswith("i.b"):
            w = rng.uniform(-3.0, 1.0, s)
        elif name.endswith("rg1.b") or name.endswith("rg2.b"):
            w = 0.5 + 0.5 * rng.standard_normal(s)
        elif name == "embed":
            w = rng.standard_normal(s)
        else:
            w = rng.standard_normal(s) * (1.2 / math.sqrt(s[-1]))
        W[name] = bf16_round(w)
    return W
