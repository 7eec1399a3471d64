"""The Mipurax decoder in the native engine against the plain numpy restatement (tests/plain_mipurax.py): each mechanism
alone, prompts cut in every way, batches, reused pages and slots, the edges of every chunk, far keys, long decoding, odd
sizes, generation.

Every test makes its own small configuration and random weights.  Errors are the largest difference of a logit over
the largest logit: float32 must stay within 1e-4.  In bfloat16 every branch's input and output is rounded to eight bits
of mantissa before it joins the stream: there the bound is 3e-2 on the root mean square of all differences (over the root
mean square of the logits) and 8e-2 on the largest one; the faults that the pointed tests plant move logits by far more.
Routers get weights under which no choice is close (see steady_routers), so that rounding never picks another expert.
"""
import copy
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import plain_mipurax as pm

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
TOL = {"float32": 1e-4, "bfloat16": 3e-2}
LARGEST = {"float32": 1e-4, "bfloat16": 8e-2}


def latent(form=1, heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, q_rank=32, scale=0.2, base=10000.0):
    return {"type": "latent_attention" if form == 1 else "latent_attention_2",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def chunked(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.3, size=20, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def moe(experts=8, top=2, ff=48, groups=(4, 2), shared=40):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def model(layers, width=64, vocab=131, eps=1e-5):
    """layers: (mixer entry, a dense feed-forward's size, a moe entry or None)."""
    cfg = {"architecture": "Mipurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": []}
    for mixer, ff in layers:
        cfg["layers"].append({**copy.deepcopy(mixer), "mlp": {"kind": "dense", "ff": ff} if isinstance(ff, int) else copy.deepcopy(ff)})
    return cfg


GENERAL = model([(chunked(), 96), (latent(), moe()), (latent(2, heads=5, dim=8, rot_dim=4, vdim=8, kv_rank=24, q_rank=16, scale=0.35, base=300.0), None),
                 (chunked(size=33, kv_from=0), moe(experts=6, top=3, ff=32, groups=(2, 1), shared=None)), (latent(2), 80),
                 (chunked(heads=2, kv_heads=2, dim=12, vdim=8, size=9), moe(experts=5, top=2, groups=None, ff=24))])
# sizes that the tensor-core kernels take: keys and values of one size (32, 64, 128), latents and heads in multiples of eight; a width and
# experts that the grouped product takes
TENSOR = model([(latent(1, heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, q_rank=48, scale=0.14), moe(experts=6, top=2, ff=128, groups=(3, 2), shared=128)),
                (chunked(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.12, size=40), 128),
                (latent(2, heads=20, dim=16, rot_dim=8, vdim=16, kv_rank=136, q_rank=32, scale=0.2), None),
                (chunked(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.15, size=24, kv_from=1), moe(experts=4, top=1, ff=128, groups=(2, 1), shared=None)),
                (chunked(heads=6, kv_heads=1, dim=128, vdim=128, scale=0.09, size=33), 64)], width=128)
BOTH = {"general": GENERAL, "tensor": TENSOR}
# a width that leaves the decode product's alignment rule, sizes that are no powers of two
ODD = model([(latent(heads=3, dim=10, rot_dim=6, vdim=14, kv_rank=20, q_rank=28, scale=0.3, base=77.0), moe(experts=6, top=2, ff=20, groups=(3, 2), shared=12)),
             (chunked(heads=3, kv_heads=3, dim=12, vdim=10, scale=0.4, size=7), 36), (chunked(heads=3, kv_heads=3, dim=12, vdim=10, scale=0.25, size=5, kv_from=1), None),
             (latent(2, heads=1, dim=6, rot_dim=10, vdim=9, kv_rank=7, q_rank=11, scale=0.4), 52)], width=72, vocab=77)
# values that are one or equal: one head, one pair turned, one expert, one group, chunks of one position (a token sees itself alone), equal sizes everywhere
ONES = model([(latent(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, q_rank=8, scale=0.3, base=2.0), moe(experts=1, top=1, ff=16, groups=(1, 1), shared=16)),
              (chunked(heads=1, kv_heads=1, dim=16, vdim=16, scale=1.0, size=1), 32), (latent(2, heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, q_rank=8, scale=0.3), None),
              (chunked(heads=1, kv_heads=1, dim=16, vdim=16, scale=0.15, size=16, kv_from=1), moe(experts=4, top=4, ff=16, groups=(4, 4), shared=None))], width=48, vocab=64)

ALONE = {
    "latent": model([(latent(), None)]),
    "latent_2": model([(latent(2), None)]),
    "latent_tensor": model([(latent(1, heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128, q_rank=96, scale=0.1), None)], width=128),
    "latent_2_tensor": model([(latent(2, heads=18, dim=32, rot_dim=16, vdim=40, kv_rank=72, q_rank=40, scale=0.14), None)], width=128),
    "latent_large": model([(latent(1, heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=64, scale=0.07), None)]),
    "latent_2_large": model([(latent(2, heads=17, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=64, scale=0.07), None)]),
    "latent_one_head": model([(latent(1, heads=1, dim=16, rot_dim=8, vdim=16, kv_rank=32, q_rank=24, scale=0.2), None),
                              (latent(2, heads=1, dim=8, rot_dim=16, vdim=8, kv_rank=24, q_rank=16, scale=0.2), None)]),
    "latent_uneven": model([(latent(1, heads=3, dim=5, rot_dim=6, vdim=7, kv_rank=9, q_rank=11, scale=0.4), None)]),
    "chunked": model([(chunked(), None)]),
    "chunked_all_keys": model([(chunked(size=None), None)]),
    "chunked_one_key_head": model([(chunked(heads=12, kv_heads=1, dim=8, vdim=8, size=30), None)]),
    "chunked_planes_32": model([(chunked(heads=6, kv_heads=3, dim=32, vdim=32, scale=0.2, size=33), None)]),
    "chunked_planes_64": model([(chunked(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.125, size=48), None)], width=128),
    "chunked_planes_128": model([(chunked(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.09, size=70), None)], width=128),
    "chunked_planes_all_keys": model([(chunked(heads=4, kv_heads=1, dim=64, vdim=64, scale=0.125, size=None), None)], width=128),
    "chunked_large_values": model([(chunked(heads=2, kv_heads=1, dim=24, vdim=136, scale=0.25, size=50), None)]),
    "another_layers_keys": model([(chunked(size=20), None), (chunked(size=50, kv_from=0), None), (chunked(size=8, kv_from=0), 32)]),
    "another_layers_keys_planes": model([(chunked(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.12, size=50), None),
                                         (chunked(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.2, size=20, kv_from=0), None),
                                         (chunked(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.1, size=None, kv_from=0), None)], width=128),
    # a width that is no multiple of four, sizes that are no multiples of four either
    "odd_width": model([(latent(heads=3, dim=10, rot_dim=2, vdim=6, kv_rank=14, q_rank=18, scale=0.3), moe(experts=6, top=2, ff=22, groups=(2, 1), shared=18)),
                        (chunked(heads=3, kv_heads=1, dim=10, vdim=6, scale=0.4, size=9), 27), (latent(2, heads=2, dim=6, rot_dim=6, vdim=10, kv_rank=10, q_rank=6, scale=0.3), None)],
                       width=90, vocab=53),
    "dense": model([(chunked(heads=2, kv_heads=2, dim=8, vdim=8), 100)]),
    "routed": model([(chunked(heads=2, kv_heads=1, dim=8, vdim=8), moe())]),
    "routed_no_groups": model([(chunked(heads=2, kv_heads=1, dim=8, vdim=8), moe(experts=7, top=3, groups=None, shared=None))]),
    "routed_single_members": model([(chunked(heads=2, kv_heads=1, dim=8, vdim=8), moe(experts=6, top=2, groups=(6, 3)))]),
    "routed_large_groups": model([(chunked(heads=2, kv_heads=1, dim=8, vdim=8), moe(experts=12, top=5, groups=(2, 1), ff=32))]),
    "routed_grouped_product": model([(chunked(heads=2, kv_heads=1, dim=32, vdim=32), moe(experts=6, top=3, groups=(3, 2), ff=128, shared=256))], width=128),
}


def steady_routers(cfg, seed):
    """Overrides under which no router's choice is close: one channel of the stream per expert carries a level of the token's own
    (a permutation of evenly spaced levels), no branch writes into these channels, and a router reads nothing but them.  A token's
    levels are drawn again until the last choice leads the first that is left out, in experts and in groups, at every scale the
    stream's norm may bring."""
    routers = [l["mlp"]["router"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"]
    if not routers:
        return {}
    rng = np.random.default_rng(seed)
    shapes = pm.tensor_shapes(cfg)
    base = pm.random_weights(cfg, seed)
    E = max(r["experts"] for r in routers)
    ladder = np.linspace(-2.2, 2.2, E)

    def steady(levels):
        for r in routers:
            for gain in (0.4, 0.8, 1.4):
                s = pm.sigmoid(gain * levels[:r["experts"]])
                allowed = np.ones(len(s), dtype=bool)
                if r.get("groups") and r["groups"]["keep"] < r["groups"]["count"]:
                    per = len(s) // r["groups"]["count"]
                    sums = np.array([np.sort(s[i:i + per])[-2:].sum() for i in range(0, len(s), per)])
                    order = np.argsort(-sums)
                    if sums[order[r["groups"]["keep"] - 1]] - sums[order[r["groups"]["keep"]]] < 0.02:
                        return False
                    for g in order[r["groups"]["keep"]:]:
                        allowed[g * per:(g + 1) * per] = False
                left = np.sort(s[allowed])[::-1]
                if len(left) > r["top"] and left[r["top"] - 1] - left[r["top"]] < 0.02:
                    return False
        return True

    over = {"embed": base["embed"].copy(), "embed.norm": base["embed.norm"].copy()}
    over["embed.norm"][:E] = 0.0
    for t in range(cfg["vocab"]):
        for _ in range(1000):
            levels = rng.permutation(ladder)
            if steady(levels):
                break
        else:
            raise AssertionError("no steady levels for this router")
        over["embed"][t, :E] = levels
    for name in shapes:
        if name.endswith((".o", ".down")):
            over[name] = base[name].copy()
            over[name][:E] = 0.0
        elif name.endswith(".norm2"):
            over[name] = base[name].copy()
            over[name][:E] = 0.0
        elif name.endswith(".router"):
            over[name] = np.eye(*shapes[name])
    return over


def tokens(vocab, n, seed):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name, cfg, seed=0, overrides=None):
        if name not in made:
            w = pm.random_weights(cfg, seed, {**steady_routers(cfg, seed), **(overrides or {})})
            made[name] = (pm.write_model_dir(tmp_path_factory.mktemp(name), cfg, w), cfg, w)
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
    close(got, pm.forward(cfg, w, toks), dtype, name)


def test_routers_with_plain_random_weights(tmp_path):
    """The choice itself in 32-bit, from router weights without any order in them: several group layouts."""
    for i, (experts, top, groups) in enumerate([(12, 3, (4, 2)), (40, 6, (8, 3)), (9, 2, (3, 1)), (66, 4, None), (64, 5, (32, 9)), (70, 7, (70, 20)), (32, 4, (8, 3)), (48, 6, (6, 3)),
                                               (80, 34, (5, 4)), (64, 6, (2, 1))]):
        cfg = model([(chunked(heads=2, kv_heads=1, dim=8, vdim=8), moe(experts=experts, top=top, groups=groups, ff=16, shared=None))])
        w = pm.random_weights(cfg, 30 + i)
        folder = pm.write_model_dir(tmp_path / str(i), cfg, w)
        toks = tokens(cfg["vocab"], 60, i)
        close(runner(folder, "float32").run([("a", toks, list(range(60)))]), pm.forward(cfg, w, toks), "float32", f"{experts} experts, {groups}")


def test_the_restatements_own_pieces():
    """The restatement's pieces against themselves written out another way."""
    w = pm.random_weights(GENERAL, 1)
    assert "l3.mix.k" not in w and "l3.mix.v" not in w and w["l1.mix.g"].shape == (3 * 24, 64) and w["l2.mix.g"].shape == (5, 64) and "l1.mix.sink" not in w
    logits, streams = pm.forward(GENERAL, w, tokens(131, 9, 0), return_layers=True)
    assert streams.shape == (6, 9, 64) and logits.shape == (9, 131)
    assert pm.seen_chunk(7, 3).astype(int).tolist()[4] == [0, 0, 0, 1, 1, 0, 0] and pm.seen_chunk(7, 3).astype(int).tolist()[6] == [0, 0, 0, 0, 0, 0, 1]
    assert np.allclose(pm.slopes(4), [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8])
    s = np.array([0.9, 0.1, 0.6, 0.55, 0.5, 0.5, 0.2, 0.95])                      # groups of two: 1.0, 1.15, 1.0, 1.15
    assert sorted(pm.choose_experts(s, {"top": 2, "groups": {"count": 4, "keep": 2}})) == [2, 7]
    assert sorted(pm.choose_experts(s, {"top": 2})) == [0, 7]
    v = np.arange(12.0).reshape(1, 2, 6)
    for interleaved, pairs in ((True, [(0, 1), (2, 3)]), (False, [(0, 2), (1, 3)])):
        out = pm.rotate(v, [3], {"base": 100.0, "dims": 4}, interleaved)
        for i, (a, b) in enumerate(pairs):
            turned = (v[0, :, a] + 1j * v[0, :, b]) * np.exp(1j * 3 * 100.0 ** (-2 * i / 4))
            assert np.allclose(out[0, :, a], turned.real) and np.allclose(out[0, :, b], turned.imag)
        assert np.array_equal(out[..., 4:], v[..., 4:])
    assert abs(pm.gelu(np.array([1.3]))[0] - 1.3 * 0.9031995154143897) < 1e-12


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["general", "tensor", "odd", "ones", "latent_tensor", "latent_2_tensor", "latent_large", "latent_2_large", "latent_uneven", "latent_one_head", "odd_width", "chunked_planes_32",
                                  "chunked_planes_64", "chunked_planes_128", "chunked_planes_all_keys", "chunked_large_values", "another_layers_keys",
                                  "another_layers_keys_planes", "routed_grouped_product", "routed_single_members"])
def test_prompt_whole_and_token_by_token(folders, name, dtype):
    cfg = {**BOTH, "odd": ODD, "ones": ONES, **ALONE}[name]
    folder, cfg, w = folders(name, cfg, seed=3 if name in ALONE else 5)
    toks = tokens(cfg["vocab"], 70, 2)
    want = pm.forward(cfg, w, toks)
    r = runner(folder, dtype)
    close(r.run([("whole", toks, list(range(70)))]), want, dtype, "whole")
    r.end("whole")
    rows = [r.run([("single", [t], [0])])[0] for t in toks]
    close(np.stack(rows), want, dtype, "token by token")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cuts", [[2] * 20, [3, 1, 2, 17, 1, 1, 30, 5, 2, 2, 16, 15, 1, 33], [16, 16, 16, 16, 1, 15, 48], [1, 2, 3, 4, 5, 6, 7, 8, 9, 10, 11, 12]])
@pytest.mark.parametrize("which", sorted(BOTH))
def test_portions(folders, cuts, dtype, which):
    """Portions down to two tokens, ending on and beside page and chunk borders."""
    folder, cfg, w = folders(which, BOTH[which], seed=5)
    toks = tokens(cfg["vocab"], sum(cuts), 7)
    want = pm.forward(cfg, w, toks)
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
    want = {k: pm.forward(cfg, w, v) for k, v in toks.items()}
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


@pytest.mark.parametrize("name", ["latent_tensor", "latent_2_tensor", "latent_2_large"])
def test_latent_tiles_of_every_kind(folders, name):
    """The tensor-core latent attention: a prompt over two listed tiles whose token groups are cut by the portion's end, single
    tokens beside another request's portion, entries of two to four tokens, and decoding."""
    folder, cfg, w = folders(name, ALONE[name], seed=3)
    a, b = tokens(cfg["vocab"], 216, 5), tokens(cfg["vocab"], 180, 6)
    want_a, want_b = pm.forward(cfg, w, a), pm.forward(cfg, w, b)
    r = runner(folder, "bfloat16", pool_tokens=512)
    close(r.run([("a", a[:190], list(range(190)))]), want_a[:190], "bfloat16", name + ": two tiles")
    got = r.run([("a", a[190:191], [0]), ("b", b[:137], list(range(137)))])
    close(got, np.concatenate([want_a[190:191], want_b[:137]]), "bfloat16", name + ": a token beside a portion")
    got = r.run([("a", a[191:194], [0, 1, 2]), ("b", b[137:139], [0, 1])])
    close(got, np.concatenate([want_a[191:194], want_b[137:139]]), "bfloat16", name + ": short entries")
    got = r.run([("a", a[194:201], list(range(7))), ("b", b[139:144], list(range(5)))])
    close(got, np.concatenate([want_a[194:201], want_b[139:144]]), "bfloat16", name + ": tiles of few tokens")
    for i in range(11):
        got = r.run([("a", [a[201 + i]], [0]), ("b", [b[144 + i]], [0])])
        close(got, np.stack([want_a[201 + i], want_b[144 + i]]), "bfloat16", name + f": decoding {i}")


@pytest.mark.parametrize("count", [1, 3, 7, 12, 16, 17, 30])
def test_routed_batches_of_single_tokens(folders, count):
    """Steps of single tokens of many requests: experts that several of them chose, and experts that none did."""
    folder, cfg, w = folders("routed_grouped_product", ALONE["routed_grouped_product"], seed=3)
    r = runner(folder, "bfloat16", pool_tokens=1024, slots=32, most_tokens=32)
    toks = [tokens(cfg["vocab"], 4, 300 + i % 9) for i in range(count)]          # some requests hold the same tokens
    for step in range(4):
        got = r.run([(i, [toks[i][step]], [0]) for i in range(count)])
        close(got, np.stack([pm.forward(cfg, w, t[:step + 1])[-1] for t in toks]), "bfloat16", f"{count} single tokens, step {step}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(BOTH))
def test_pages_and_slots_are_used_again(folders, dtype, which):
    """Two slots and a pool of four pages: every request takes pages that another one has left full."""
    folder, cfg, w = folders(which, BOTH[which], seed=5)
    r = runner(folder, dtype, pool_tokens=64, page_size=16, slots=2)
    for i in range(6):
        a, b = tokens(cfg["vocab"], 20 + i, 40 + i), tokens(cfg["vocab"], 31 - i, 60 + i)
        out = r.run([(f"a{i}", a[:7], []), (f"b{i}", b, [len(b) - 1])])
        close(out, pm.forward(cfg, w, b)[-1:], dtype, f"b{i}")
        r.end(f"b{i}")
        out = r.run([(f"a{i}", a[7:], list(range(len(a) - 7)))])
        close(out, pm.forward(cfg, w, a)[7:], dtype, f"a{i}")
        r.end(f"a{i}")
    assert r.info("live_requests") == 0


def test_chunked_pool_holds_long_requests(folders):
    """A request far longer than the pool: chunks give pages back while it runs, and the cache keeps what the layer of the longest
    chunk among those that share it may still see (here a reader's 50 positions, in front of a writer's 20)."""
    cfg = model([(chunked(size=20), 32), (chunked(size=50, kv_from=0), None), (chunked(heads=2, kv_heads=1, dim=8, vdim=8, size=33), None)])
    folder, cfg, w = folders("chunks_only", cfg, seed=8)
    toks = tokens(cfg["vocab"], 300, 3)
    want = pm.forward(cfg, w, toks)
    r = runner(folder, "float32", pool_tokens=112, page_size=16, slots=2, most_tokens=512)
    rows, at = [], 0
    for n in [30, 17, 2, 31] + [20] * 11:
        rows.append(r.run([("long", toks[at:at + n], list(range(n)))]))
        at += n
    close(np.concatenate(rows), want, "float32", "300 tokens through seven pages")


def aimed(cfg, seed, a, b, sharp=12.0, at=0):
    """Weights under which one score stands out in layer `at`: the key map is the query map behind a reflection of the model's width
    that carries token b's embedding onto token a's.  Token b is then the key that token a looks for, whatever lies between them;
    b's value is its own.  The score of that pair is about `sharp`, the others' a fraction of it.  What stands in front of the layer
    leaves the stream as it is.  An attention that reads another layer's keys gets that layer's key map."""
    cfg = copy.deepcopy(cfg)
    base = pm.random_weights(cfg, seed)
    over = {"embed.norm": np.zeros_like(base["embed.norm"])}
    layer = cfg["layers"][at]
    m, p = layer["mixer"], f"l{at}.mix."
    keys = m.get("kv_from", at)
    for i in range(at):
        over[f"l{i}.mix.o"] = np.zeros_like(base[f"l{i}.mix.o"])
        assert cfg["layers"][i]["mlp"] is None
    for i in {at, keys}:
        over[f"l{i}.norm1"] = np.zeros_like(base[f"l{i}.norm1"])
    ea, eb = base["embed"][a], base["embed"][b]
    u = ea / np.linalg.norm(ea) - eb / np.linalg.norm(eb)
    u /= np.linalg.norm(u)
    if layer["type"] == "attention":
        q = base[p + "q"].reshape(m["heads"], m["dim"], -1)[::m["heads"] // m["kv_heads"]]
        over[f"l{keys}.mix.k"] = (q - 2.0 * np.einsum("gdw,w,v->gdv", q, u, u)).reshape(m["kv_heads"] * m["dim"], -1)
        m["scale"] = sharp / (2.25 * m["dim"])
    else:
        assert m["q_rank"] == m["kv_rank"]
        H, dn, dr, rank = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
        dq = base[p + "dq"]
        over[p + "dkv"] = np.concatenate([dq - 2.0 * np.outer(dq @ u, u), base[p + "dkv"][rank:]])
        over[p + "dq.norm"] = over[p + "dkv.norm"] = np.ones(rank)
        uq = base[p + "uq"].reshape(H, dn + dr, rank).copy()
        over[p + "uk"] = uq[:, :dn].reshape(H * dn, rank)
        uq[:, dn:] *= 0.3                                          # the turned part stays small beside the pair's score
        over[p + "uq"] = uq.reshape(H * (dn + dr), rank)
        m["scale"] = sharp / (2.25 * dn)
    return cfg, over


def with_chunks_moved(by, cfg, w, toks):
    """The restatement's logits with every chunk starting `by` positions later."""
    saved = pm.seen_chunk

    def moved(n, size):
        i, j = np.arange(n)[:, None], np.arange(n)[None, :]
        return (j <= i) & ((i - by) // size == (j - by) // size)

    pm.seen_chunk = moved
    try:
        return pm.forward(cfg, w, toks)
    finally:
        pm.seen_chunk = saved


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("offset", ["inside", "outside"])
@pytest.mark.parametrize("how", ["prompt", "decoded"])
@pytest.mark.parametrize("dim", [16, 64])
@pytest.mark.parametrize("reader", [False, True])
def test_chunk_edges(folders, dtype, offset, how, dim, reader):
    """The one key that the last token looks for lies on its chunk's first position, or on the one before it, in a layer with keys of
    its own and in one that reads another layer's under a mask of another size.  The restatement with the chunks moved by one
    gives other logits at that place (checked), so a mask that is one off shows."""
    own = (chunked(heads=2, kv_heads=1, dim=dim, vdim=dim, size=31 if reader else 20), None)
    layers = [own, (chunked(heads=2, kv_heads=1, dim=dim, vdim=dim, size=20, kv_from=0), None)] if reader else [own]
    cfg, over = aimed(model(layers, vocab=90), 4, 88, 89, at=1 if reader else 0)
    folder, cfg, w = folders(f"edge{dim}{reader}", cfg, seed=4, overrides=over)
    n = 70                                                        # the key lies on and beside a page border in turn
    for end in (n - 1, n - 2, n - 6):
        toks = tokens(80, n, 100 + end)                           # ids 80.. are kept for the two tokens
        toks[end] = 88
        toks[end // 20 * 20 - (offset == "outside")] = 89
        want = pm.forward(cfg, w, toks)
        other_row = with_chunks_moved(1 if offset == "inside" else -1, cfg, w, toks)[end]
        moved = np.abs(other_row - want[end]).max() / np.abs(want).max()
        assert moved > 4 * TOL[dtype], f"the test's weights do not show the edge ({moved:.3g})"
        r = runner(folder, dtype, pool_tokens=128)
        if how == "prompt":
            got = r.run([("e", toks, [end])])
        else:
            r.run([("e", toks[:end - 3], [])])
            got = np.concatenate([r.run([("e", [t], [0])]) for t in toks[end - 3:end + 1]])[-1:]
        close(got, want[end:end + 1], dtype, f"{offset} {how} end {end}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("form", [1, 2])
@pytest.mark.parametrize("large", [False, True])
def test_far_latent_keys(folders, dtype, form, large):
    """Sharp latent attention: the keys that the last tokens look for lie hundreds of positions back (the first position, a page's last
    and first, the first of a tile of 64), in a prompt's tail and while decoding; with the key replaced the logits are elsewhere."""
    sizes = dict(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128, q_rank=128) if large else dict(heads=2, dim=24, rot_dim=6, vdim=10, kv_rank=24, q_rank=24)
    cfg, over = aimed(model([(latent(form, **sizes), 64)], vocab=140, width=128), 9, 138, 139)
    folder, cfg, w = folders(f"far{form}{large}", cfg, seed=9, overrides=over)
    for key in (0, 15, 16, 64):
        toks = tokens(130, 400, 21 + key)
        toks[key] = 139
        toks[350] = toks[395] = 138
        want = pm.forward(cfg, w, toks)
        changed = list(toks)
        changed[key] = 1
        for place in (350, 395):
            assert np.abs(pm.forward(cfg, w, changed)[place] - want[place]).max() > 4 * TOL[dtype] * np.abs(want).max()
        r = runner(folder, dtype, pool_tokens=448, page_size=16)
        ask = [0, 1, 15, 16, 17, 64, 330, 350, 369]
        rows = [r.run([("f", toks[:370], ask)])] + [r.run([("f", [t], [0])]) for t in toks[370:]]
        close(np.concatenate(rows), np.concatenate([want[ask], want[370:]]), dtype, f"key {key}")


def test_every_mechanism_matters():
    """The small models are made so that a mechanism that is left out shows: the restatement without the sinks, the gates, the slopes,
    the groups, the embedding's norm or another layer's keys gives other logits."""
    cfg = GENERAL
    w = pm.random_weights(cfg, 5, steady_routers(cfg, 5))
    toks = tokens(cfg["vocab"], 64, 12)
    want = pm.forward(cfg, w, toks)
    far = 2 * TOL["bfloat16"] * np.sqrt((want * want).mean())

    def differs(what, cfg2=cfg, w2=w):
        d = pm.forward(cfg2, w2, toks) - want
        assert np.sqrt((d * d).mean()) > far, what

    differs("sinks", w2={**w, "l2.mix.sink": w["l2.mix.sink"] * 0 - 60.0, "l4.mix.sink": w["l4.mix.sink"] * 0 - 60.0})
    for name in ("l1.mix.g", "l4.mix.g"):
        differs(name, w2={**w, name: w[name] * 0.0})
    differs("embedding's norm", w2={**w, "embed.norm": w["embed.norm"] * 0.0})
    other = copy.deepcopy(cfg)
    other["layers"][1]["mlp"]["router"].pop("groups")
    differs("groups", cfg2=other)
    other = copy.deepcopy(cfg)
    other["layers"][3]["mixer"]["mask"]["size"] = 20
    differs("the reader's own mask", cfg2=other)
    saved = pm.slopes
    pm.slopes = lambda heads: np.zeros(heads)
    try:
        differs("slopes")
    finally:
        pm.slopes = saved
    saved = pm.rotate
    pm.rotate = lambda v, positions, rot, interleaved: saved(v, positions, rot, not interleaved)
    try:
        differs("rotation layouts")
    finally:
        pm.rotate = saved


def test_long_chunks_over_several_ctas(folders):
    """Chunks of hundreds of positions on the tensor-core path: a single token's keys are then dealt to several CTAs, a prompt tile's
    keys to several units.  One key far back is the one that the last tokens look for, in a portion's tail and while two requests
    decode side by side, in the layer that has the keys and in one that reads them."""
    cfg, over = aimed(model([(chunked(heads=4, kv_heads=2, dim=64, vdim=64, size=1300), None), (chunked(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.1, size=900, kv_from=0), None),
                             (chunked(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.09, size=700), None),
                             (latent(2, heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64, q_rank=48, scale=0.14), None)], vocab=140, width=128), 9, 138, 139, sharp=20.0)
    folder, cfg, w = folders("long_chunks", cfg, seed=9, overrides=over)
    n = 1440
    toks = tokens(130, n, 77)
    toks[1301] = 139
    for place in (1310, 1399, 1439):
        toks[place] = 138
    toks[2], toks[1290] = 139, 138                                # the first chunk's, 1,288 positions back
    want = pm.forward(cfg, w, toks)
    changed = list(toks)
    changed[1301] = 1
    assert np.abs(pm.forward(cfg, w, changed)[1439] - want[1439]).max() > 4 * TOL["bfloat16"] * np.abs(want).max()
    r = runner(folder, "bfloat16", pool_tokens=4096, most_tokens=2048)
    ask = [0, 69, 70, 639, 640, 699, 700, 701, 899]
    rows = [r.run([("a", toks[:900], ask)]), r.run([("a", toks[900:1300], [0, 389, 390, 399])])]
    r.run([("b", toks[:1300], [])])                              # a second request with the same tokens decodes beside the first
    for t in toks[1300:]:
        out = r.run([("a", [t], [0]), ("b", [t], [0])])
        close(out[1:], out[:1], "bfloat16", "two requests with the same tokens")
        rows.append(out[:1])
    close(np.concatenate(rows), np.concatenate([want[ask], want[[900, 1289, 1290, 1299]], want[1300:]]), "bfloat16", "long chunks")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["odd", "tensor"])
def test_long_decoding_through_captured_steps(folders, dtype, which):
    folder, cfg, w = folders(which, ODD if which == "odd" else TENSOR, seed=5)
    toks = tokens(cfg["vocab"], 240, 31)
    want = pm.forward(cfg, w, toks)
    r = runner(folder, dtype, pool_tokens=512)
    rows = [r.run([("x", toks[:5], [4]), ("y", toks[:3], [])])]
    rows += [r.run([("x", [t], [0]), ("y", [u], [0])])[:1] for t, u in zip(toks[5:], toks[3:])]
    close(np.concatenate(rows), want[4:], dtype, "decoding")
    assert r.info("graph_replays") > 200


def test_first_tokens_of_a_sequence(folders):
    """Position 0 alone, then position 1: nothing before the sequence leaks in (a softmax over one key, with and without a sink), also
    in a slot that another request has used."""
    folder, cfg, w = folders("general", GENERAL, seed=5)
    r = runner(folder, "float32", slots=1)
    for seed in range(3):
        toks = tokens(cfg["vocab"], 2, 80 + seed)
        want = pm.forward(cfg, w, toks)
        close(r.run([(seed, toks[:1], [0])]), want[:1], "float32", "first token")
        close(r.run([(seed, toks[1:], [0])]), want[1:], "float32", "second token")
        r.end(seed)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(BOTH))
def test_greedy_generation_through_the_engine(folders, dtype, which):
    """The scheduler's own entry point: prompts in portions beside decoding requests, greedy; each generated token must be
    (within the tolerance) the plain implementation's best token after the same prefix."""
    from easy_gpt.cpp_b200.native import NativeEngine

    folder, cfg, w = folders(which, BOTH[which], seed=5)
    prompts = [tokens(cfg["vocab"], n, 90 + n) for n in (3, 41, 18, 70, 9, 26)]
    engine = NativeEngine(folder, dtype=dtype, page_size=16, cache_tokens=512, max_active=4, chunk_size=16, max_batch_tokens=48)
    outputs = engine.generate(prompts, max_new_tokens=12, greedy=True)
    for prompt, out in zip(prompts, outputs):
        assert len(out) == 12
        logits = pm.forward(cfg, w, prompt + out)
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
    want = pm.forward(cfg, w, toks)
    close(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1), want[[0, 29]], "float32", "step 0")
    close(np.fromfile(out / "1.f32", dtype="<f4").reshape(1, -1), want[[39]], "float32", "step 1")


def test_command_line_with_random_weights(tmp_path):
    """The engine's own program on this design: random-weights mode writes a folder from a config.json (with the per-tensor hints that
    keep norms and sinks sane), then prompts of token ids are decoded greedily; the tokens must be the plain implementation's for the
    weights that were written."""
    cfg = model([(latent(heads=2, dim=16, rot_dim=4, vdim=8, kv_rank=16, q_rank=24), moe(experts=4, top=2, ff=24, groups=(2, 1), shared=16)),
                 (chunked(heads=2, kv_heads=1, dim=16, vdim=8, size=12), None), (latent(2, heads=2, dim=8, rot_dim=4, vdim=16, kv_rank=24, q_rank=16), 24),
                 (chunked(heads=2, kv_heads=1, dim=16, vdim=8, size=6, kv_from=1), 40)], width=64, vocab=97)
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
    cfg_read, w = pm.read_model_dir(folder)
    assert set(w) == set(pm.tensor_shapes(cfg)) and np.all(w["l0.norm1"] == 0.0) and np.all(w["embed.norm"] == 0.0) and np.all(w["l0.mix.dkv.norm"] == 1.0)
    assert np.all(w["l2.mix.sink"] == 0.0) and "l3.mix.k" not in w
    for prompt, out in zip([[5, 17, 3], [9, 8, 7, 6]], outs):
        logits = pm.forward(cfg_read, w, prompt + out)
        for i, tok in enumerate(out):
            row = logits[len(prompt) + i - 1]
            assert float(row.max() - row[tok]) <= 4e-4 * np.abs(row).max(), (i, tok, int(row.argmax()))
