"""GPU: the Gusedra design through the library's own entry points (llama_decode on a llama_batch, llama_kv_cache_seq_rm, the
plain-generation scheduler, bin/trace_run) against the float64 oracle of tests/gusedra_oracle.py, on small random models written to a
folder (config.json + model.safetensors) and loaded like any other model.

float32 contexts are compared at 2e-4 of the logits' spread, which is what makes a window or a bucket's border one token off, a kept
token that is lost, a missing sink or a wrong cell show; bfloat16 contexts at 6e-2 (the median; single tokens may be several times as far
where rounding turns a close choice of experts).  Every schedule (whole prompt, portions, token by token, mixed batches, reused cells
and slots) is compared with the oracle AND, in float32, with the whole-prompt run."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from tests import gusedra_oracle as O
from tests.gusedra_configs import CONFIGS, drawn
from tests.test_gpu_rapisun import Served, row_err, spread, TOL32, TOL16

pytestmark = pytest.mark.gpu


def oracle_logits(cfg, W, toks):
    return O.forward(cfg, W, O.Sequence(cfg), list(toks))


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def close16(e, tol=TOL16):
    return np.median(e) < tol and np.quantile(e, 0.95) < 4 * tol and e.max() < 12 * tol


def spotlight(cfg, W, special_token, il=0, fi=3, fj=5, size=6.0):
    """Random weights would hide a key that enters or leaves a window among dozens.  This makes ONE token's key stand out in layer il's first
    head: the query is one coordinate reading an input feature that is positive for all tokens, the key the same coordinate reading a feature
    that is negative for all tokens but `special_token`; the special key's score is far above every other's."""
    W = dict(W)
    E = W["embed"].copy()
    E[:, fi], E[:, fj] = size, -size
    E[special_token, fj] = size
    W["embed"] = E
    p = "l%d." % il
    W[p + "norm1"], W[p + "norm1.b"] = np.ones_like(W[p + "norm1"]), 0 * W[p + "norm1.b"]
    mx = cfg["layers"][il]["mixer"]
    D = mx["dim"]
    for name, f in (("q", fi), ("k", fj)):
        M = W[p + "mix." + name].copy()
        M[:D, :] = 0.0
        M[D - 1, f] = 2.0
        W[p + "mix." + name] = M
    return W


# ---- each mechanism alone, float32 and bfloat16 -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["slope_only", "bucket_only", "experts_only", "shared_cells", "ones", "mixed_small", "far_keys", "wide_heads"])
@pytest.mark.parametrize("float32", [True, False])
def test_whole_prompt_matches_oracle(tmp_path, name, float32):
    cfg = CONFIGS[name]()
    W = O.random_weights(cfg, 11)
    toks = tokens(cfg, 37, 1)
    ref = oracle_logits(cfg, W, toks)
    s = Served(tmp_path, cfg, W, float32=float32)
    got = s.feed(0, toks, [])
    s.close()
    e = row_err(got, ref)
    assert e.max() < TOL32 if float32 else close16(e)


@pytest.mark.parametrize("seed", range(12))
def test_drawn_configurations(tmp_path, seed):
    """configurations drawn from a seed: a prompt long enough for the long-portion paths, whole and cut, in float32; whole in bfloat16"""
    cfg = drawn(100 + seed)
    W = O.random_weights(cfg, 200 + seed)
    toks = tokens(cfg, 280, 300 + seed)
    ref = oracle_logits(cfg, W, toks)
    # a drawn model may magnify rounding (a norm over few distinct values): how much is measured on the oracle itself, as the answer to weights moved
    # by 1e-7 of their size; the tolerances grow with it beyond a usual 15
    rng = np.random.default_rng(0)
    moved = {k: v * (1.0 + 1e-7 * rng.standard_normal(v.shape)) for k, v in W.items()}
    gain = max(1.0, float(np.median(row_err(oracle_logits(cfg, moved, toks[:80]), ref[:80])) / 1e-7) / 15.0)

    def close32(e):
        return np.quantile(e, 0.98) < TOL32 * gain
    s = Served(tmp_path / "a", cfg, W, n_ctx=900)
    whole = s.feed(0, toks, [])
    assert close32(row_err(whole, ref)), json.dumps(cfg)
    cut = s.feed(1, toks, [2, 131, 132, 260] + list(range(270, 280)))
    assert close32(row_err(cut, ref)) and close32(row_err(cut, whole)), json.dumps(cfg)
    s.close()
    s = Served(tmp_path / "b", cfg, W, float32=False, n_ctx=300)
    e = row_err(s.feed(0, toks, []), ref)
    assert np.median(e) < TOL16 * gain, json.dumps(cfg)
    s.close()


def test_residual_stream_after_every_layer(tmp_path, monkeypatch):
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 31)
    toks = tokens(cfg, 19, 5)
    trace = []
    O.forward(cfg, W, O.Sequence(cfg), toks, trace)
    dump = tmp_path / "dump"
    dump.mkdir()
    monkeypatch.setenv("PIB_HYBRID_DUMP", str(dump))
    s = Served(tmp_path / "m", cfg, W)
    s.feed(0, toks, [])
    s.close()
    for i, ref in enumerate(trace):
        got = np.fromfile(dump / ("d0_l%d.f32" % i), "<f4").reshape(ref.shape)
        assert np.abs(got - ref).max() < 1e-4 * max(1.0, np.abs(ref).max()), "layer %d" % i


def test_every_tensor_shows(tmp_path):
    """the oracle with any one tensor changed differs by far more than the tolerance, so the comparison with the library sees each"""
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 28)
    toks = tokens(cfg, 30, 9)
    ref = oracle_logits(cfg, W, toks)
    for name in sorted(W):
        if name.startswith("l1.") or name.startswith("l0.mix") or name.startswith("l4.m") or name.startswith("final"):
            W2 = dict(W)
            W2[name] = W[name] * 1.5 + np.linspace(-1.0, 1.0, W[name].size) if W[name].ndim == 1 else W[name] * np.linspace(0.5, 1.5, W[name].shape[0])[:, None]
            e = row_err(oracle_logits(cfg, W2, toks), ref)
            assert (e.max() if ".mlp." in name else np.median(e)) > 3 * TOL32, name          # an expert may serve few of the tokens
    s = Served(tmp_path, cfg, W)
    assert row_err(s.feed(0, toks, []), ref).max() < TOL32
    assert row_err(s.feed(1, toks, range(1, 30)), ref).max() < TOL32
    s.close()


# ---- prefill against token-by-token decoding, and portions down to two tokens ------------------------------------------------------------
@pytest.mark.parametrize("name", ["mixed_small", "slope_only", "bucket_only", "experts_only", "shared_cells", "ones"])
def test_cuts_do_not_matter(tmp_path, name):
    cfg = CONFIGS[name]()
    W = O.random_weights(cfg, 12)
    toks = tokens(cfg, 41, 2)
    ref = oracle_logits(cfg, W, toks)
    s = Served(tmp_path, cfg, W)
    whole = s.feed(0, toks, [])
    schedules = {"token by token": range(1, 41), "twos": range(2, 41, 2), "mixed sizes": [2, 4, 5, 12, 14, 15, 17, 30, 32],
                 "prompt then decode": [20] + list(range(21, 41)), "one, then the rest": [1], "threes after two": range(2, 41, 3)}
    for i, (label, cuts) in enumerate(schedules.items()):
        got = s.feed(1 + i, toks, cuts)
        s.end(1 + i)
        assert row_err(got, ref).max() < TOL32, label
        assert row_err(got, whole).max() < TOL32, label
    s.close()


def test_cuts_do_not_matter_bfloat16(tmp_path):
    cfg = CONFIGS["wide_heads"]()
    W = O.random_weights(cfg, 13)
    toks = tokens(cfg, 33, 3)
    ref = oracle_logits(cfg, W, toks)
    s = Served(tmp_path, cfg, W, float32=False)
    for i, cuts in enumerate([[], range(1, 33), [2, 4, 11, 13, 29]]):
        assert close16(row_err(s.feed(i, toks, cuts), ref))
    s.close()


# ---- the first tokens of a sequence -------------------------------------------
def test_first_tokens(tmp_path):
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 25)
    s = Served(tmp_path, cfg, W)
    for r, n in enumerate([1, 2, 3, 4]):
        toks = tokens(cfg, n, 40 + r)
        assert row_err(s.feed(r, toks, []), oracle_logits(cfg, W, toks)).max() < TOL32
    for r in range(4):
        s.end(r)
    # the same slots again, one token at a time: nothing of the earlier owners may be seen
    for r, n in enumerate([3, 1, 4, 2]):
        toks = tokens(cfg, n, 50 + r)
        assert row_err(s.feed(r, toks, range(1, n)), oracle_logits(cfg, W, toks)).max() < TOL32
    s.close()


# ---- window edges and kept tokens: one key that stands out, in prompts and in decoding ----------------------------------------------------------
@pytest.mark.parametrize("kind,place", [("slopes", "first"), ("slopes", "inside"), ("buckets", "kept"), ("buckets", "last kept"), ("buckets", "first not kept"), ("buckets", "inside")])
def test_one_key_stands_out_at_every_edge(tmp_path, kind, place):
    """one token's key carries the first head's output wherever it is seen.  A window one token longer, or one kept token more or fewer,
    must change the oracle's answer plainly; the library must agree with the oracle everywhere: whole, in portions whose edges lie around
    the window's, in decoded tokens, and in the tensor-core form of served mode"""
    cfg = CONFIGS["far_keys"]()
    cfg["layers"] = cfg["layers"][:1] if kind == "slopes" else cfg["layers"][1:]
    cfg["layers"][0]["mlp"] = None
    cfg["layers"][0]["mixer"]["dim"] = 16
    cfg["layers"][0]["mixer"]["vdim"] = 16
    mk = cfg["layers"][0]["mixer"]["mask"]
    size, keep = mk["size"], mk.get("keep_first", 0)
    W = spotlight(cfg, O.random_weights(cfg, 26), cfg["vocab"] - 1)
    toks = np.random.default_rng(7).integers(0, cfg["vocab"] - 1, 260).tolist()
    special = {"kept": 0, "first": 0, "last kept": keep - 1, "first not kept": keep, "inside": 90}[place]
    toks[special] = cfg["vocab"] - 1
    ref = oracle_logits(cfg, W, toks)
    edge = special + size                                         # the first position that the window no longer shows it to

    def moved(**kw):
        c = copy.deepcopy(cfg)
        c["layers"][0]["mixer"]["mask"].update(kw)
        return row_err(oracle_logits(c, W, toks), ref)
    if special < keep:
        assert np.quantile(moved(keep_first=special)[edge:], 0.05) > 0.02      # it is seen to the end
    else:
        assert moved(size=size + 1)[edge] > 0.02 and moved(size=size - 1)[edge - 1] > 0.02
    if place == "first not kept":
        assert np.quantile(moved(keep_first=keep + 1)[edge:], 0.05) > 0.02
    near = [edge - 2, edge - 1, edge, edge + 1, edge + 2]
    cuts = [c for c in sorted({special, special + 1, keep, 63, 64, 65} | set(near) | set(range(220, 260))) if c > 0]
    s = Served(tmp_path, cfg, W, n_ctx=1024)
    assert row_err(s.feed(0, toks, []), ref).max() < TOL32
    assert row_err(s.feed(1, toks, cuts), ref).max() < TOL32
    assert row_err(s.feed(2, toks, range(1, edge + 4)), ref).max() < TOL32
    s.close()
    s = Served(tmp_path, cfg, W, float32=False, n_ctx=1024)       # served mode: long portions run as tensor-core matmuls, with and without columns set apart for the kept tokens
    assert close16(row_err(s.feed(0, toks, []), ref))
    assert close16(row_err(s.feed(1, toks, [130]), ref))
    assert close16(row_err(s.feed(2, toks, cuts), ref))
    s.close()


def test_the_edge_of_a_window_over_shared_cells(tmp_path):
    """a layer that reads another layer's cells sees them through its OWN window: one key stands out, longer and shorter windows than the owner's"""
    cfg = CONFIGS["shared_cells"]()
    cfg["layers"] = cfg["layers"][:2] + [cfg["layers"][3]]
    for jl in cfg["layers"]:
        jl["mlp"] = None
    cfg["layers"][1]["mixer"]["mask"] = {"size": 33}
    W = O.random_weights(cfg, 36)
    W = spotlight(cfg, W, cfg["vocab"] - 1)
    for i in (1, 2):                                              # the readers' first head asks as the owner's does
        W["l%d.norm1" % i], W["l%d.norm1.b" % i] = W["l0.norm1"], W["l0.norm1.b"]
        M = W["l%d.mix.q" % i].copy()
        M[:8] = W["l0.mix.q"][:8]
        W["l%d.mix.q" % i] = M
    toks = np.random.default_rng(17).integers(0, cfg["vocab"] - 1, 90).tolist()
    toks[20] = cfg["vocab"] - 1
    ref = oracle_logits(cfg, W, toks)
    for i, size in ((1, 33), (2, 5)):
        c = copy.deepcopy(cfg)
        c["layers"][i]["mixer"]["mask"]["size"] = size + 1
        assert row_err(oracle_logits(c, W, toks), ref)[20 + size] > 20 * TOL32
    s = Served(tmp_path, cfg, W)
    for r, cuts in enumerate([[], [20, 21, 24, 25, 26, 52, 53, 54], range(1, 90)]):
        assert row_err(s.feed(0, toks, cuts), ref).max() < TOL32
        s.end(0)
    s.close()


def test_far_keys_among_hundreds(tmp_path):
    cfg = CONFIGS["far_keys"]()
    W = O.random_weights(cfg, 16)
    toks = tokens(cfg, 300, 6)
    ref = oracle_logits(cfg, W, toks)
    s = Served(tmp_path, cfg, W, n_ctx=640)
    assert row_err(s.feed(0, toks, []), ref).max() < TOL32
    assert row_err(s.feed(1, toks, [64, 128, 191, 192, 193, 194, 258, 259, 260, 261, 262] + list(range(263, 300))), ref).max() < TOL32
    s.close()


def test_sink_slope_and_buckets_show(tmp_path):
    """the oracle without its sink, with slopes of another head count, and with buckets that reach a little further differs plainly; the library does not"""
    cfg = CONFIGS["slope_only"]()
    W = O.random_weights(cfg, 29)
    toks = tokens(cfg, 40, 3)
    ref = oracle_logits(cfg, W, toks)
    W2 = dict(W)
    W2["l1.mix.sink"] = W["l1.mix.sink"] - 30.0
    assert np.median(row_err(oracle_logits(cfg, W2, toks), ref)) > 20 * TOL32
    orig = O.slope
    O.slope = lambda h, H: orig(h, H) * 1.02
    try:
        assert np.median(row_err(oracle_logits(cfg, W, toks), ref)) > 5 * TOL32
    finally:
        O.slope = orig
    s = Served(tmp_path / "a", cfg, W)
    assert row_err(s.feed(0, toks, []), ref).max() < TOL32
    s.close()
    cfg = CONFIGS["bucket_only"]()
    W = O.random_weights(cfg, 30)
    toks = tokens(cfg, 90, 4)
    ref = oracle_logits(cfg, W, toks)
    c = copy.deepcopy(cfg)
    c["layers"][2]["mixer"]["bias_max"] += 9
    assert np.median(row_err(oracle_logits(c, W, toks), ref)[40:]) > 5 * TOL32
    s = Served(tmp_path / "b", cfg, W)
    assert row_err(s.feed(0, toks, []), ref).max() < TOL32
    assert row_err(s.feed(1, toks, [7, 8, 40] + list(range(60, 90))), ref).max() < TOL32
    s.close()


def test_a_bucket_with_a_large_bias_shows_its_borders(tmp_path):
    """one bucket's bias stands far above all others: a distance more or less in it moves the first head's output; whole, cut, decoded, and as matmuls"""
    cfg = CONFIGS["wide_heads"]()
    cfg["layers"] = cfg["layers"][1:2]
    cfg["layers"][0]["mlp"] = None
    mx = cfg["layers"][0]["mixer"]
    W = O.random_weights(cfg, 35)
    R = W["l0.mix.rel"].copy()
    R[14] += 7.0
    W["l0.mix.rel"] = O.bf16_round(R)
    toks = tokens(cfg, 200, 5)
    ref = oracle_logits(cfg, W, toks)
    n = [d for d in range(200) if O.bucket(d, mx["buckets"], mx["bias_max"]) == 14]
    assert len(n) > 4
    orig = O.bucket
    for lo, hi in ((n[0] + 1, n[-1]), (n[0], n[-1] - 1)):        # the bucket one distance shorter on either side
        O.bucket = lambda d, B, D: orig(d, B, D) if lo <= d <= hi or d not in n else 3
        try:
            assert np.median(row_err(oracle_logits(cfg, W, toks), ref)[80:]) > 50 * TOL32
        finally:
            O.bucket = orig
    s = Served(tmp_path / "a", cfg, W, n_ctx=512)
    assert row_err(s.feed(0, toks, []), ref).max() < TOL32
    assert row_err(s.feed(1, toks, [60, 61, 130] + list(range(180, 200))), ref).max() < TOL32
    s.close()
    s = Served(tmp_path / "b", cfg, W, float32=False, n_ctx=512)
    assert close16(row_err(s.feed(0, toks, []), ref)) and close16(row_err(s.feed(1, toks, [150]), ref))
    s.close()


def test_negative_choice_scores_and_groups(tmp_path):
    """all choice scores far below zero: what is outside the kept groups must stay outside (it counts as minus infinity, not as nought); weights come from
    the uncorrected scores; identity outputs among the chosen; one token (routing and sorting in one launch), many tokens, and more tokens than that"""
    cfg = CONFIGS["experts_only"]()
    W = O.random_weights(cfg, 39)
    for i in range(4):
        W["l%d.mlp.correction" % i] = O.bf16_round(W["l%d.mlp.correction" % i] - 3.0)
    toks = tokens(cfg, 60, 6)
    ref = oracle_logits(cfg, W, toks)
    s = Served(tmp_path, cfg, W)
    for r, cuts in enumerate([[], range(1, 60), [16, 33, 34, 50], [17]]):
        assert row_err(s.feed(r, toks, cuts), ref).max() < TOL32
    s.close()


# ---- batches of unequal requests against each alone; cells and slots freed and used again -------------------------------------------------
def test_mixed_batches_and_reuse(tmp_path):
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 17)
    lens = [45, 9, 30, 2, 17, 26, 1, 38]
    reqs = [tokens(cfg, n, 20 + i) for i, n in enumerate(lens)]
    refs = [oracle_logits(cfg, W, t) for t in reqs]
    # 3 slots and 120 cells for 168 tokens: both have to come back and be used again, cells out of order
    s = Served(tmp_path, cfg, W, n_ctx=120, slots=3)
    rng = np.random.default_rng(7)
    got = [[] for _ in reqs]
    at = [0] * len(reqs)
    live, nxt = [], 0
    while nxt < len(reqs) or live:
        while nxt < len(reqs) and len(live) < 3:
            live.append(nxt)
            nxt += 1
        entries = []
        for r in live:
            left = len(reqs[r]) - at[r]
            n = min(left, int(rng.choice([1, 1, 2, 3, 7, 16])))
            if sum(len(t) for _, t in entries) + n > 120 - sum(at[q] for q in live):
                continue
            entries.append((r, reqs[r][at[r]:at[r] + n]))
        assert entries
        out = s.step(entries)
        for r, t in entries:
            got[r].append(out[r])
            at[r] += len(t)
        for r in list(live):
            if at[r] == len(reqs[r]):
                s.end(r)
                live.remove(r)
    for r in range(len(reqs)):
        assert row_err(np.concatenate(got[r]), refs[r]).max() < TOL32, "request %d" % r
    used, _ = s.ctx.kv_view()
    assert used == 0 and s.ctx.L.llama_pib_state_slots_free(s.ctx.ctx) == 3
    s.close()


def test_long_decoding(tmp_path):
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 19)
    toks = tokens(cfg, 150, 8)
    ref = oracle_logits(cfg, W, toks)
    s = Served(tmp_path, cfg, W)
    e = row_err(s.feed(0, toks, [6] + list(range(7, 150))), ref)
    s.close()
    assert e.max() < TOL32


@pytest.mark.parametrize("name", ["wide_heads", "big_heads"])
def test_long_portions_take_the_matmul_forms(tmp_path, name):
    """served mode: portions of 128 tokens and more run as tensor-core matmuls; shorter portions and decoded tokens stay with the per-token
    kernels.  Both against the oracle, against each other, and mixed in one batch"""
    cfg = CONFIGS[name]()
    W = O.random_weights(cfg, 23)
    toks, other = tokens(cfg, 450, 10), tokens(cfg, 60, 11)
    ref, ref_o = oracle_logits(cfg, W, toks), oracle_logits(cfg, W, other)
    s = Served(tmp_path, cfg, W, float32=False, n_ctx=1600)
    whole = s.feed(0, toks, [])                                            # one portion of 450
    small = s.feed(1, toks, range(100, 450, 100))                          # portions of 100: the per-token kernels
    cut = s.feed(2, toks, [130, 131, 300, 449])                            # 130 (matmul) + 1 + 169 (matmul) + 149 (matmul) + 1
    assert close16(row_err(whole, ref)) and close16(row_err(small, ref)) and close16(row_err(cut, ref))
    assert close16(row_err(whole, small)) and close16(row_err(cut, small))
    for r in range(3):
        s.end(r)
    a = s.step([(3, toks[:200]), (4, other[:59])])                         # a long portion beside a short one and a decoded token in ONE batch
    b = s.step([(4, other[59:]), (3, toks[200:])])
    assert close16(row_err(np.concatenate([a[3], b[3]]), ref))
    assert close16(row_err(np.concatenate([a[4], b[4]]), ref_o))
    s.close()
    s = Served(tmp_path, cfg, W, float32=True, n_ctx=600)                  # float32 contexts never take it
    assert row_err(s.feed(0, toks, []), ref).max() < TOL32
    s.close()


@pytest.mark.parametrize("float32", [True, False])
def test_medium_model_long_prompt_cuts_and_batches(tmp_path, float32):
    cfg = CONFIGS["medium"]()
    W = O.random_weights(cfg, 33)
    toks, other = tokens(cfg, 330, 12), tokens(cfg, 140, 13)
    ref, ref_o = oracle_logits(cfg, W, toks), oracle_logits(cfg, W, other)
    close = (lambda e: e.max() < TOL32) if float32 else close16
    s = Served(tmp_path, cfg, W, float32=float32, n_ctx=1400)
    assert close(row_err(s.feed(0, toks, []), ref))
    assert close(row_err(s.feed(1, toks, [150, 151, 153, 290] + list(range(300, 330))), ref))
    s.end(0)
    s.end(1)
    a = s.step([(2, toks[:129]), (3, other[:7])])
    b = s.step([(3, other[7:139]), (2, toks[129:131])])
    c = s.step([(2, toks[131:]), (3, other[139:])])
    assert close(row_err(np.concatenate([a[2], b[2], c[2]]), ref))
    assert close(row_err(np.concatenate([a[3], b[3], c[3]]), ref_o))
    s.close()


def test_decode_steps_around_growing_prompts(tmp_path):
    """single-token steps are replayed from captured graphs; a later, longer prompt makes the context grow its buffers, and the steps
    after it must not run on the old ones"""
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 22)
    s = Served(tmp_path, cfg, W, n_ctx=512)
    for r, n_prompt in enumerate([5, 40, 18, 130, 70]):
        toks = tokens(cfg, n_prompt + 9, 30 + r)
        ref = oracle_logits(cfg, W, toks)
        got = s.feed(r, toks, [n_prompt] + list(range(n_prompt + 1, n_prompt + 9)))
        s.end(r)
        assert row_err(got, ref).max() < TOL32, "request %d" % r
    s.close()


@pytest.mark.parametrize("float32", [True, False])
def test_greedy_generation_through_the_scheduler(tmp_path, float32):
    from pipeinfer_b200 import llama
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 21)
    O.write_model(str(tmp_path), cfg, W)
    prompt = tokens(cfg, 9, 9)
    ctx = llama.Context(model_dir=str(tmp_path), n_ctx=128, max_seq=4, float32=float32)
    out, res, _ = llama.plain_generate(ctx, prompt, 24)
    ctx.close()
    assert len(out) == 24
    # the oracle follows the library's tokens; wherever its own choice differs the two best logits must be a near tie
    seq = O.Sequence(cfg)
    lg = O.forward(cfg, W, seq, prompt)[-1]
    for t in out:
        best = int(np.argmax(lg))
        if best != t:
            assert lg[best] - lg[t] < (1e-3 if float32 else 0.3) * spread(lg), "token %d instead of %d" % (t, best)
        lg = O.forward(cfg, W, seq, [t])[-1]


def test_sizes_left_out_come_from_the_tensors(tmp_path):
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 37)
    toks = tokens(cfg, 20, 2)
    ref = oracle_logits(cfg, W, toks)
    short = copy.deepcopy(cfg)
    for jl in short["layers"]:
        for k in ("heads", "kv_heads", "dim", "vdim"):
            del jl["mixer"][k]
        jl["mixer"].pop("buckets", None)
        for part in (jl["mlp"] or {}, (jl["mlp"] or {}).get("expert", {}), (jl["mlp"] or {}).get("shared", {})):
            part.pop("ff", None)
    s = Served(tmp_path, short, W)
    assert row_err(s.feed(0, toks, []), ref).max() < TOL32
    s.close()


def test_bad_configurations_are_refused(tmp_path):
    from pipeinfer_b200 import llama
    from pipeinfer_b200.lib import PibError
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 38)
    for i, (il, path, val) in enumerate([(0, ("type",), "other"), (0, ("mixer", "kv_heads"), 4), (2, ("mixer", "kv_from"), 2), (2, ("mixer", "kv_from"), 1), (0, ("mlp", "kind"), "sparse"),
                                         (1, ("mlp", "router", "groups", "count"), 4), (1, ("mlp", "router", "groups", "keep"), 4), (1, ("mlp", "router", "top"), 7)]):
        c = copy.deepcopy(cfg)
        o = c["layers"][il]
        for k in path[:-1]:
            o = o[k]
        o[path[-1]] = val
        d = tmp_path / str(i)
        O.write_model(str(d), c, W)
        with pytest.raises(PibError):
            llama.Context(model_dir=str(d), n_ctx=64, max_seq=4)


def test_trace_runner_replays_steps(tmp_path):
    """bin/trace_run as a user starts it: JSON steps on standard input (portions beside single tokens, requests ending, more requests
    than state slots over time, cells for the live ones only), logits files out, one 'done' line per step"""
    cfg = CONFIGS["mixed_small"]()
    W = O.random_weights(cfg, 24)
    model = tmp_path / "model"
    O.write_model(str(model), cfg, W)
    reqs = {"a": tokens(cfg, 50, 1), "b": tokens(cfg, 21, 2), "c": tokens(cfg, 33, 3), "d": tokens(cfg, 2, 4), "e": tokens(cfg, 40, 5)}
    refs = {k: oracle_logits(cfg, W, v) for k, v in reqs.items()}
    plan = [[("a", 30), ("b", 2)], [("a", 1), ("b", 19), ("c", 7)], [("a", 19), ("c", 1)], [("c", 25), ("d", 2)], [("e", 38)], [("e", 1)], [("e", 1)]]
    at, steps, wanted = {k: 0 for k in reqs}, [], []
    for n, step in enumerate(plan):
        entries, end, rows = [], [], []
        for rid, cnt in step:
            lo, hi = at[rid], at[rid] + cnt
            want = sorted({0, cnt - 1}) if cnt > 1 else [0]
            entries.append({"id": rid, "tokens": reqs[rid][lo:hi], "want": want})
            rows += [(rid, lo + w) for w in want]
            at[rid] = hi
            if hi == len(reqs[rid]):
                end.append(rid)
        steps.append(json.dumps({"step": n, "entries": entries, "end": end}))
        wanted.append(rows)
    root = os.path.abspath(os.path.join(os.path.dirname(__file__), ".."))
    for dtype, tol in (("float32", TOL32), ("bfloat16", 4 * TOL16)):
        out = tmp_path / ("out_" + dtype)
        p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "128", "--slots", "3"], input="\n".join(steps) + "\n", capture_output=True, text=True, timeout=300)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.split("\n") if l.startswith("done")] == ["done %d" % json.loads(s)["step"] for s in steps]
        for n, rows in enumerate(wanted):
            got = np.fromfile(out / ("%d.f32" % n), "<f4").reshape(len(rows), -1)
            ref = np.stack([refs[rid][i] for rid, i in rows])
            assert got.shape == ref.shape and np.isfinite(got).all()
            assert row_err(got, ref).max() < tol, (dtype, n)
