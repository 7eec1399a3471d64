"""The Zodosun decoder in the native engine against the plain numpy restatement (tests/plain_zodosun.py): each mechanism
alone, prompts cut in every way, batches, reused pages and slots, distances on the borders of the bias table's buckets, far
keys, slow states, long decoding, odd sizes, generation.

Every test makes its own small configuration and random weights.  Errors are the largest difference of a logit over
the largest logit: float32 must stay within 1e-4.  In bfloat16 the bound is 3e-2 on the root mean square of all
differences (over the root mean square of the logits) and 8e-2 on the largest one; the faults that the pointed tests plant
in the restatement move logits by far more.
"""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import plain_zodosun as pz

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
TOL = {"float32": 1e-4, "bfloat16": 3e-2}
LARGEST = {"float32": 1e-4, "bfloat16": 8e-2}


def delta(heads=3, dim=16):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}}


def side(left=(4, 2, 16, 24), right=(3, 16, 8), scale=0.3, bias_max=50, q_temp=(0.4, 16), decay=None):
    l = {"heads": left[0], "kv_heads": left[1], "dim": left[2], "vdim": left[3], "scale": scale, "bias_max": bias_max}
    if q_temp:
        l["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    decay = decay or [round(1.0 - 0.5 ** (1 + 3 * h), 6) for h in range(right[0])]
    return {"type": "parallel", "mixer": {"left": l, "right": {"heads": right[0], "dim": right[1], "vdim": right[2], "decay": decay}}}


def model(layers, width=64, vocab=131, eps=1e-5, groups=4, logit_scale=0.7):
    """layers: (mixer entry, ff or None)"""
    cfg = {"architecture": "Zodosun", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "layers": []}
    for mixer, ff in layers:
        cfg["layers"].append({**copy.deepcopy(mixer), "mlp": {"kind": "dense", "ff": ff} if ff else None})
    if logit_scale:
        cfg["logit_scale"] = logit_scale
    return cfg


GENERAL = model([(delta(), 96), (side(), 80), (delta(2, 24), None), (side(left=(2, 1, 24, 8), right=(1, 8, 24), q_temp=None, bias_max=20), None)])
GENERAL_SIZES = {"buckets": {1: 8, 3: 5}, "rank": {0: 5, 2: 12}}
# sizes of real layers' kinds: heads of 64 and 128, key and value sizes equal
TENSOR = model([(side(left=(4, 2, 64, 64), right=(2, 64, 64), scale=0.125, bias_max=100), 96), (delta(2, 64), None),
                (side(left=(4, 1, 128, 128), right=(2, 128, 64), scale=0.09, bias_max=40), None)], width=128, groups=2)
BOTH = {"general": GENERAL, "tensor": TENSOR}
# widths that leave the decode product's alignment rule, head sizes that are no multiples of eight, an odd number of bucket rows
ODD = model([(side(left=(3, 3, 12, 10), right=(3, 10, 6), bias_max=17, q_temp=(0.9, 5)), 52), (delta(3, 10), 36), (side(left=(3, 1, 10, 6), right=(2, 6, 10)), None)],
            width=72, vocab=77, groups=3, logit_scale=None)
ODD_SIZES = {"buckets": {0: 7, 2: 2}, "rank": {1: 3}}
# values that are one or equal: one head, one key head, one norm group, an inner size of one, one bucket row, a temperature that steps at
# every position, a decay of one (a plain sum) and equal sizes throughout
ONES = model([(side(left=(1, 1, 16, 16), right=(1, 16, 16), scale=1.0, bias_max=1, q_temp=(1.0, 1), decay=[1.0]), None), (delta(1, 16), 32)], width=48, vocab=64, groups=1,
             logit_scale=1.0)
ONES_SIZES = {"buckets": 1, "rank": 1}

ALONE = {
    "delta": model([(delta(), None)]),
    "delta_8": model([(delta(4, 8), None)]),
    "delta_64": model([(delta(2, 64), None)], width=128),
    "delta_40": model([(delta(2, 40), None)]),
    "delta_128": model([(delta(1, 128), None)], width=128),
    "delta_200": model([(delta(1, 200), None)], width=128),
    "delta_odd": model([(delta(3, 13), None)], width=60, groups=5),
    "side": model([(side(), None)]),
    "side_no_temperature": model([(side(q_temp=None), None)]),
    "side_many_heads_a_key": model([(side(left=(40, 2, 16, 16)), None)]),
    "side_equal_32": model([(side(left=(6, 3, 32, 32)), None)]),
    "side_96": model([(side(left=(4, 2, 96, 96), scale=0.1), None)], width=128),
    "side_long_values": model([(side(left=(2, 1, 40, 200), right=(2, 24, 136)), None)]),
    "side_long_keys": model([(side(left=(2, 2, 264, 8), right=(2, 200, 40), scale=0.06), None)]),
    "side_wide_reach": model([(side(left=(2, 1, 16, 16), bias_max=5000), None)]),
    "side_odd": model([(side(left=(2, 1, 7, 9), right=(3, 5, 7)), None)], width=66, groups=11, vocab=53),
    "two_groups": model([(delta(2, 8), 40)], groups=2),
    "groups_of_two": model([(delta(2, 8), 24)], groups=32),
    "one_group": model([(delta(2, 8), 48), (side(), 48)], groups=1),
    "feed_forward": model([(delta(2, 8), 100)]),
}
SIZES = {"general": GENERAL_SIZES, "odd": ODD_SIZES, "ones": ONES_SIZES, "side_96": {"buckets": 16}, "side_wide_reach": {"buckets": 64}, "side_long_keys": {"buckets": 3},
         "delta_64": {"rank": 40}, "tensor": {"buckets": {0: 16, 2: 12}, "rank": 9}}


def tokens(vocab, n, seed):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name, cfg, seed=0, overrides=None):
        if name not in made:
            w = pz.random_weights(cfg, seed, overrides, **SIZES.get(name, {}))
            made[name] = (pz.write_model_dir(tmp_path_factory.mktemp(name), cfg, w), cfg, w)
        return made[name]

    return get


def runner(folder, dtype, pool_tokens=512, page_size=16, slots=4, graphs=True, most_tokens=None):
    from easy_gpt.cpp_b200.native import NativeStepRunner

    return NativeStepRunner(folder, dtype, page_size=page_size, num_pages=pool_tokens // page_size, max_slots=slots,
                            max_tokens_per_request=most_tokens or pool_tokens, use_graphs=graphs)


def close(got, want, dtype, what=""):
    diff = np.asarray(got, dtype=np.float64) - want
    largest = float(np.abs(diff).max() / np.abs(want).max())
    assert largest <= LARGEST[dtype], f"{what}: largest error {largest:.3g} over {LARGEST[dtype]:.3g}"
    spread = float(np.sqrt((diff * diff).mean()) / np.sqrt((want * want).mean()))
    assert spread <= TOL[dtype] or dtype == "float32", f"{what}: error {spread:.3g} over {TOL[dtype]:.3g}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(folders, name, dtype):
    folder, cfg, w = folders(name, ALONE[name], seed=3)
    toks = tokens(cfg["vocab"], 75, 1)
    got = runner(folder, dtype).run([("a", toks, list(range(75)))])
    close(got, pz.forward(cfg, w, toks), dtype, name)


def test_the_restatement_itself():
    """Pieces of the restatement against what their formulas say of simple cases."""
    assert [pz.distance_bucket(n, 8, 50) for n in (0, 1, 3, 4, 5, 49, 50, 1000)] == [0, 1, 3, 4, 4, 7, 7, 7]
    assert [pz.distance_bucket(n, 7, 17) for n in (2, 3, 16, 17)] == [2, 3, 6, 6] and pz.distance_bucket(5, 1, 1) == 0
    assert np.allclose(pz.query_temperature(range(6), {"coef": 1.0, "every": 3}), 1.0 + np.log([1, 1, 2, 2, 2, 3]))
    x = np.array([[3.0, 4.0, 0.0, 1.0]])
    assert np.allclose(pz.group_norm(x, np.ones(4), 0.0, 2), [[3 / math.sqrt(12.5), 4 / math.sqrt(12.5), 0.0, math.sqrt(2.0)]])
    assert np.allclose(pz.wave_positions([2], 5)[0], [math.sin(2), math.cos(2), math.sin(2 * 1e4 ** -0.4), math.cos(2 * 1e4 ** -0.4), math.sin(2 * 1e4 ** -0.8)])
    w = pz.random_weights(GENERAL, 1, **GENERAL_SIZES)
    assert w["l1.mix.left.rel"].shape == (8, 4) and w["l3.mix.left.rel"].shape == (5, 2) and w["l2.mix.w2"].shape == (48, 12)
    logits, streams = pz.forward(GENERAL, w, tokens(131, 9, 0), return_layers=True)
    assert streams.shape == (4, 9, 64) and logits.shape == (9, 131)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,cfg", [("general", GENERAL), ("tensor", TENSOR), ("odd", ODD), ("ones", ONES), ("alone_delta_64", None), ("alone_delta_200", None),
                                      ("alone_delta_odd", None), ("alone_side_96", None), ("alone_side_long_values", None), ("alone_side_long_keys", None),
                                      ("alone_side_wide_reach", None), ("alone_side_odd", None), ("alone_side_many_heads_a_key", None), ("alone_one_group", None)])
def test_prompt_whole_and_token_by_token(folders, name, cfg, dtype):
    if cfg is None:
        name = name[len("alone_"):]
        cfg = ALONE[name]
    folder, cfg, w = folders(name, cfg, seed=3 if name in ALONE else 5)
    toks = tokens(cfg["vocab"], 70, 2)
    want = pz.forward(cfg, w, toks)
    r = runner(folder, dtype)
    close(r.run([("whole", toks, list(range(70)))]), want, dtype, "whole")
    r.end("whole")
    rows = [r.run([("single", [t], [0])])[0] for t in toks]
    close(np.stack(rows), want, dtype, "token by token")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cuts", [[2] * 20, [3, 1, 2, 17, 1, 1, 30, 5, 2, 2, 16, 15, 1, 33], [16, 16, 16, 16, 1, 15, 48], [1, 2, 3, 4, 5, 6, 7, 8, 9, 10, 11, 12]])
@pytest.mark.parametrize("which", sorted(BOTH))
def test_portions(folders, cuts, dtype, which):
    """Portions down to two tokens, ending on and beside page borders, tiles of the recurrences and steps of the temperature."""
    folder, cfg, w = folders(which, BOTH[which], seed=5)
    toks = tokens(cfg["vocab"], sum(cuts), 7)
    want = pz.forward(cfg, w, toks)
    r = runner(folder, dtype, page_size=16)
    at, rows = 0, []
    for n in cuts:
        rows.append(r.run([("p", toks[at:at + n], list(range(n)))]))
        at += n
    close(np.concatenate(rows), want, dtype, f"portions {cuts}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(BOTH))
def test_batches_of_unequal_requests(folders, dtype, which):
    """Four requests of different lengths advance together, portions beside single tokens; each must come out as alone."""
    folder, cfg, w = folders(which, BOTH[which], seed=5)
    lengths = {"a": 61, "b": 9, "c": 130, "d": 33}
    toks = {k: tokens(cfg["vocab"], n, 10 + i) for i, (k, n) in enumerate(lengths.items())}
    want = {k: pz.forward(cfg, w, v) for k, v in toks.items()}
    plans = {"a": [40] + [1] * 21, "b": [1] * 9, "c": [2, 64, 31, 1, 1, 30, 1], "d": [16, 17]}
    r = runner(folder, dtype, pool_tokens=512)
    at = {k: 0 for k in toks}
    got = {k: [] for k in toks}
    step = 0
    while any(plans.values()):
        entries, names = [], []
        for k in sorted(plans):
            if plans[k] and (step % 3 != 2 or k != "b"):            # b sits out every third step
                n = plans[k].pop(0)
                entries.append((k, toks[k][at[k]:at[k] + n], list(range(n))))
                names.append((k, n))
                at[k] += n
        if entries:
            out = r.run(entries)
            row = 0
            for k, n in names:
                got[k].append(out[row:row + n])
                row += n
        step += 1
    for k in toks:
        close(np.concatenate(got[k]), want[k], dtype, f"request {k}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(BOTH))
def test_pages_and_slots_are_used_again(folders, dtype, which):
    """Two slots and a pool of four pages: every request takes a slot (the states of both recurrences) and pages that
    another one has left full."""
    folder, cfg, w = folders(which, BOTH[which], seed=5)
    r = runner(folder, dtype, pool_tokens=64, page_size=16, slots=2)
    for i in range(6):
        a, b = tokens(cfg["vocab"], 20 + i, 40 + i), tokens(cfg["vocab"], 31 - i, 60 + i)
        out = r.run([(f"a{i}", a[:7], []), (f"b{i}", b, [len(b) - 1])])
        close(out, pz.forward(cfg, w, b)[-1:], dtype, f"b{i}")
        r.end(f"b{i}")
        out = r.run([(f"a{i}", a[7:], list(range(len(a) - 7)))])
        close(out, pz.forward(cfg, w, a)[7:], dtype, f"a{i}")
        r.end(f"a{i}")
    assert r.info("live_requests") == 0


def aimed(cfg, seed, a, b, sharp=16.0, offset=0.0, background=-4.0, **sizes):
    """Weights under which one key stands out in the first layer's attention: the key map is the query map of its group's first
    head behind a reflection of the width that carries token b's embedding onto token a's, so that token b is the key that
    token a's first heads look for, wherever it lies.  The number per head takes the pair's score (before bias and temperature) and
    `offset` off again for those heads, so that the weight is on the sigmoid's slope and follows the bias; the other heads'
    weights make a background of about the same size (the mixer's output is normed: a lone key's weight would not show), and the
    mixer's output is what the stream then mostly holds."""
    cfg = copy.deepcopy(cfg)
    base = pz.random_weights(cfg, seed, **sizes)
    m, p = cfg["layers"][0]["mixer"]["left"], "l0.mix.left."
    m["scale"] = sharp / m["dim"]
    per = m["heads"] // m["kv_heads"]
    # embeddings a good deal larger than the waves of the position, so that a token's normed row is its own wherever it stands
    over = {"embed": base["embed"] * 6.0}
    ea, eb = base["embed"][a], base["embed"][b]
    u = ea / np.linalg.norm(ea) - eb / np.linalg.norm(eb)
    u /= np.linalg.norm(u)
    q = base[p + "q"].reshape(m["heads"], m["dim"], -1)[::per]
    k = q - 2.0 * np.einsum("gdw,w,v->gdv", q, u, u)
    over[p + "k"] = k.reshape(base[p + "k"].shape)
    for name in ("q.b", "k.b"):
        over[p + name] = np.zeros_like(base[p + name])
    for name in ("q.norm", "k.norm"):
        over[p + name] = np.ones_like(base[p + name])
    over[p + "g"] = np.zeros_like(base[p + "g"])
    over[p + "out"] = base[p + "out"] * 40.0
    over["l0.norm1"] = np.ones_like(base["l0.norm1"])
    ha, hb = pz.group_norm(np.stack([ea, eb]), np.ones(len(ea)), 0.0, cfg["norm"]["groups"])
    qa = pz.rms_unit(base[p + "q"] @ ha, 0.0).reshape(m["heads"], m["dim"])
    kb = pz.rms_unit(over[p + "k"] @ hb, 0.0).reshape(m["kv_heads"], m["dim"])
    scores = np.einsum("hd,hd->h", qa, np.repeat(kb, per, axis=0)) * m["scale"]
    over[p + "pb"] = np.where(np.arange(m["heads"]) % per == 0, -scores - offset, background - 2.4 * sharp / math.sqrt(m["dim"]))
    return cfg, over


BORDERS = {"narrow": dict(bias_max=56, buckets=9), "long": dict(bias_max=300, buckets=12), "odd": dict(bias_max=60, buckets=7)}


def first_distances(buckets, most):
    """The first distance of every bucket beyond the half, in integer arithmetic: n belongs to step e or a later one when
    (n / half)^rest >= (most / half)^e."""
    half = buckets // 2
    rest = buckets - half
    return [next(n for n in range(half, most + 1) if n ** rest * half ** e >= most ** e * half ** rest) for e in range(1, rest)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["prompt", "decoded"])
@pytest.mark.parametrize("dim", [60, 64])
@pytest.mark.parametrize("border", sorted(BORDERS))
def test_distance_buckets(folders, dtype, how, border, dim):
    """The one key that the last token looks for lies on the last distance of a bucket or on the first of the next, where the
    table's neighbouring rows differ by 4: with the restatement's buckets moved by one distance the logits there are elsewhere
    (checked), so a bias that is one distance off shows."""
    b = BORDERS[border]
    shape = model([(side(left=(2, 1, dim, dim), right=(1, 8, 8), bias_max=b["bias_max"], q_temp=None), None)], vocab=90, width=128, groups=2)
    cfg, over = aimed(shape, 4, 88, 89, buckets=b["buckets"])
    over["l0.mix.left.rel"] = np.where(np.arange(b["buckets"])[:, None] % 2, 2.0, -2.0) * np.ones((1, 2))
    name = f"border_{border}_{dim}"
    SIZES[name] = {"buckets": b["buckets"]}
    folder, cfg, w = folders(name, cfg, seed=4, overrides=over)
    starts = first_distances(b["buckets"], b["bias_max"])
    assert [pz.distance_bucket(n, b["buckets"], b["bias_max"]) for n in starts] == list(range(b["buckets"] // 2 + 1, b["buckets"]))
    for first in starts[:1] + starts[-2:]:
        for distance in (first - 1, first):
            end = first + 21
            toks = tokens(80, end + 1, 100 + end)                  # ids 80.. are kept for the two tokens
            toks[end], toks[end - distance] = 88, 89
            want = pz.forward(cfg, w, toks)[end:]
            plain = pz.distance_bucket
            pz.distance_bucket = lambda n, rows, most: plain(n + (1 if distance == first - 1 else -1) if n else 0, rows, most)
            try:
                moved = pz.forward(cfg, w, toks)[end:]
            finally:
                pz.distance_bucket = plain
            assert np.abs(moved - want).max() / np.abs(want).max() > 4 * TOL[dtype], "the test's weights do not show the border"
            r = runner(folder, dtype)
            if how == "prompt":
                got = r.run([("e", toks, [end])])
            else:
                r.run([("e", toks[:end - 2], [])])
                got = np.concatenate([r.run([("e", [t], [0])]) for t in toks[end - 2:]])[-1:]
            close(got, want, dtype, f"{border} distance {distance} {how}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim", [(60, 24), (64, 40), (64, 64), (128, 128), (96, 96)])
def test_far_keys(folders, dtype, dim, vdim):
    """A key many pages back is the one that tokens look for, in a long prompt's tail (cut in two portions) and while two requests
    decode side by side (a single token's keys are then dealt to several CTAs); a replaced key, a query without its temperature
    and a table without its last row give other logits there (checked)."""
    shape = model([(side(left=(4, 2, dim, vdim), right=(2, 16, 16), bias_max=64, q_temp=(0.2, 256)), 64), (delta(2, 16), None)], vocab=140, width=128, groups=4)
    cfg, over = aimed(shape, 9, 138, 139, offset=4.0, background=-5.5, buckets=10)
    over["l0.mix.left.rel"] = np.linspace(-1.0, 1.0, 10)[:, None] * np.ones((1, 4))
    name = f"far{dim}_{vdim}"
    SIZES[name] = {"buckets": 10}
    folder, cfg, w = folders(name, cfg, seed=9, overrides=over)
    n = 1160
    toks = tokens(130, n, 21)
    toks[47] = 139                                                # the last position of a page
    asks = (1000, 1111, n - 1)
    for place in asks:
        toks[place] = 138
    want = pz.forward(cfg, w, toks)
    changed = list(toks)
    changed[47] = 1
    cool = copy.deepcopy(cfg)
    cool["layers"][0]["mixer"]["left"].pop("q_temp")
    flat = dict(w)
    flat["l0.mix.left.rel"] = w["l0.mix.left.rel"].copy()
    flat["l0.mix.left.rel"][9] = -3.0
    for what, other in (("key", pz.forward(cfg, w, changed)), ("temperature", pz.forward(cool, w, toks)), ("last row", pz.forward(cfg, flat, toks))):
        for place in asks:
            assert np.abs(other[place] - want[place]).max() > 4 * TOL[dtype] * np.abs(want).max(), (what, place)
    r = runner(folder, dtype, pool_tokens=4096, most_tokens=2048)
    ask = [0, 1, 46, 47, 48, 255, 256, 599]
    rows = [r.run([("f", toks[:600], ask)]), r.run([("f", toks[600:1100], [400, 499])])]
    r.run([("g", toks[:1100], [])])                              # a second request with the same tokens decodes beside the first
    for t in toks[1100:]:
        out = r.run([("f", [t], [0]), ("g", [t], [0])])
        close(out[1:], out[:1], dtype, "two requests with the same tokens")
        rows.append(out[:1])
    close(np.concatenate(rows), np.concatenate([want[ask], want[[1000, 1099]], want[1100:]]), dtype, "far keys")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [16, 64])
def test_slow_states(folders, dtype, dim):
    """States that hardly fade (decays within 1e-3 of one) over 700 tokens, then decoding: what the first token wrote is still
    read at the end (checked: another first token gives other logits), and so is what a removal takes off (checked)."""
    cfg = model([(side(left=(2, 1, 16, 16), right=(2, dim, dim), decay=[0.9995, 0.999]), None), (delta(2, dim), None)], width=128, groups=2, vocab=150)
    base = pz.random_weights(cfg, 12)
    over = {"l1.mix.w0": np.full_like(base["l1.mix.w0"], -8.0), "l1.mix.a.b": np.full_like(base["l1.mix.a.b"], -3.0), "embed": base["embed"].copy(),
            "l0.mix.right.out": base["l0.mix.right.out"] * 6.0, "l1.mix.norm": base["l1.mix.norm"] * 6.0}
    # one token whose keys and values stand out: a channel (that of the slowest sine) which no other token uses, with large weights
    over["embed"][:, 126] = 0.0
    over["embed"][149, 126] = 9.0
    for name in ("l0.mix.right.k", "l0.mix.right.v", "l1.mix.k", "l1.mix.v"):
        over[name] = base[name].copy()
        over[name][:, 126] *= 10.0 if dim < 64 else 25.0
    name = f"slow{dim}"
    folder, cfg, w = folders(name, cfg, seed=12, overrides=over)
    toks = tokens(140, 700, 5)
    want = pz.forward(cfg, w, toks)
    other = [149] + toks[1:]
    moved = pz.forward(cfg, w, other)
    assert np.abs(moved[-1] - want[-1]).max() > 4 * TOL[dtype] * np.abs(want).max(), "the first token does not show"
    kept = dict(w)
    kept["l1.mix.a.b"] = np.full_like(base["l1.mix.a.b"], -30.0)
    assert np.abs(pz.forward(cfg, kept, toks)[-1] - want[-1]).max() > 4 * TOL[dtype] * np.abs(want).max(), "the removal does not show"
    for seq, ref in ((toks, want), (other, moved)):
        r = runner(folder, dtype, pool_tokens=1024)
        rows = [r.run([("s", seq[:333], [0, 1, 332])]), r.run([("s", seq[333:650], [316])])] + [r.run([("s", [t], [0])]) for t in seq[650:]]
        close(np.concatenate(rows), np.concatenate([ref[[0, 1, 332, 649]], ref[650:]]), dtype, "slow states")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["odd", "tensor"])
def test_long_decoding_through_captured_steps(folders, dtype, which):
    folder, cfg, w = folders(which, ODD if which == "odd" else TENSOR, seed=5)
    toks = tokens(cfg["vocab"], 240, 31)
    want = pz.forward(cfg, w, toks)
    r = runner(folder, dtype, pool_tokens=512)
    rows = [r.run([("x", toks[:5], [4]), ("y", toks[:3], [])])]
    rows += [r.run([("x", [t], [0]), ("y", [u], [0])])[:1] for t, u in zip(toks[5:], toks[3:])]
    close(np.concatenate(rows), want[4:], dtype, "decoding")
    assert r.info("graph_replays") > 200


def test_first_tokens_of_a_sequence(folders):
    """Position 0 alone, then position 1: empty states, one key, also in a slot that another request has used."""
    folder, cfg, w = folders("general", GENERAL, seed=5)
    r = runner(folder, "float32", slots=1)
    for seed in range(3):
        toks = tokens(cfg["vocab"], 2, 80 + seed)
        want = pz.forward(cfg, w, toks)
        close(r.run([(seed, toks[:1], [0])]), want[:1], "float32", "first token")
        close(r.run([(seed, toks[1:], [0])]), want[1:], "float32", "second token")
        r.end(seed)


def test_many_requests_at_once(folders):
    """A batch of 24 single tokens (the library's products instead of the decode product) and portions of more than the decode
    product's rows, against each request alone."""
    folder, cfg, w = folders("tensor", TENSOR, seed=5)
    r = runner(folder, "bfloat16", pool_tokens=2048, slots=24, most_tokens=128)
    toks = {i: tokens(cfg["vocab"], 20 + i, 300 + i) for i in range(24)}
    r.run([(i, t[:-3], []) for i, t in toks.items()])
    got = [r.run([(i, [t[len(t) - 3 + s]], [0]) for i, t in toks.items()]) for s in range(3)]
    for i, t in toks.items():
        close(np.stack([g[i] for g in got]), pz.forward(cfg, w, t)[-3:], "bfloat16", f"request {i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(folders, dtype):
    """The scheduler's own entry point: prompts in portions beside decoding requests, greedy; each generated token must be
    (within the tolerance) the plain implementation's best token after the same prefix."""
    from easy_gpt.cpp_b200.native import NativeEngine

    folder, cfg, w = folders("general", GENERAL, seed=5)
    prompts = [tokens(cfg["vocab"], n, 90 + n) for n in (3, 41, 18, 70, 9, 26)]
    engine = NativeEngine(folder, dtype=dtype, page_size=16, cache_tokens=512, max_active=4, chunk_size=16, max_batch_tokens=48)
    outputs = engine.generate(prompts, max_new_tokens=12, greedy=True)
    for prompt, out in zip(prompts, outputs):
        assert len(out) == 12
        logits = pz.forward(cfg, w, prompt + out)
        for i, tok in enumerate(out):
            row = logits[len(prompt) + i - 1]
            assert float(row.max() - row[tok]) <= 4 * TOL[dtype] * np.abs(row).max(), (dtype, i, tok, int(row.argmax()))


def test_trace_replay_program(folders, tmp_path):
    """bin/trace_run on a model folder of this design: steps in, logits files out."""
    folder, cfg, w = folders("odd", ODD, seed=5)
    toks = tokens(cfg["vocab"], 40, 55)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": toks[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": toks[30:], "want": [9]}, {"id": "z", "tokens": toks[:2], "want": []}], "end": ["q", "z"]}]
    out = tmp_path / "out"
    run = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1"]
    want = pz.forward(cfg, w, toks)
    close(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1), want[[0, 29]], "float32", "step 0")
    close(np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1), want[[39]], "float32", "step 1")


def test_command_line_with_random_weights(tmp_path):
    """The engine's own program on this design: random-weights mode writes a folder from a config.json, then prompts of token ids
    are decoded greedily; the tokens must be the plain implementation's for the weights that were written."""
    cfg = model([(delta(2, 16), None), (side(left=(2, 1, 16, 8), right=(2, 16, 8)), 40)], width=64, vocab=97)
    cfg["layers"][0]["mixer"]["rank"] = 6
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    prompts = tmp_path / "prompts.txt"
    prompts.write_text("5 17 3\n9,8,7,6\n")
    folder = tmp_path / "model"
    folder.mkdir()
    cmd = [sys.executable, str(ROOT / "bin" / "easy_llm"), "--model", str(folder), "--random-weights", "7", "--config", str(tmp_path / "config.json"),
           "--token-ids", "--greedy", "--max-steps", "10", "--dtype", "float32", "-f", str(prompts)]
    r = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    outs = [[int(t) for t in line.split()] for line in (tmp_path / "prompts_output.txt").read_text().splitlines()]
    assert len(outs) == 2 and len(outs[0]) == 8 and len(outs[1]) == 7
    cfg_read, w = pz.read_model_dir(folder)
    assert np.all(w["l0.norm1"] == 1.0) and np.all(w["l1.mix.left.out"] == 1.0) and w["l0.mix.w1"].shape == (6, 64)
    for prompt, out in zip([[5, 17, 3], [9, 8, 7, 6]], outs):
        logits = pz.forward(cfg_read, w, prompt + out)
        for i, tok in enumerate(out):
            row = logits[len(prompt) + i - 1]
            assert float(row.max() - row[tok]) <= 4e-4 * np.abs(row).max(), (i, tok, int(row.argmax()))
