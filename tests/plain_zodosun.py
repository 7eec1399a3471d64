"""Plain, slow restatement of the Zodosun decoder in numpy float64: whole sequences, no cache, no batching, one
function per mechanism.  It shares nothing with the engine and is what the engine's results are held against.

A model is (config, weights): ``config`` the parsed config.json, ``weights`` a dict name -> float64 array.

Notation: n tokens, d the model width; a linear map stored [out, in] is applied as ``x @ W.T``; positions count from 0.
A layer is  x += mixer(N1(x)); x += ff(N2(x))  with N an RMS norm over consecutive groups of channels.
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np


# ---- elementwise pieces -------------------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_unit(x, eps):
    """x over its root mean square along the last axis, eps under the root."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def group_norm(x, gain, eps, groups):
    """Every one of `groups` equal runs of channels over its own root mean square; one gain per channel."""
    n, d = x.shape
    return rms_unit(x.reshape(n, groups, d // groups), eps).reshape(n, d) * gain


def wave_positions(positions, width):
    """Entry 2i: sine, entry 2i + 1: cosine of position * 10000^(-2i / width)."""
    channel = np.arange(width)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * 10000.0 ** (-2.0 * (channel // 2) / width)
    return np.where(channel % 2 == 0, np.sin(angle), np.cos(angle))


# ---- attention with sigmoid weights ------------------------------------------------------------------------------
def distance_bucket(n, buckets, most):
    """Which row of a bias table a distance n >= 0 reads: one row per distance below half the rows, then rows whose reach
    grows geometrically up to `most`; the last row serves everything beyond."""
    half = buckets // 2
    if n < half:
        return n
    if half == 0:
        return buckets - 1
    grown = math.log(n / half) / math.log(most / half) * (buckets - half)
    return min(buckets - 1, half + math.floor(grown))


def query_temperature(positions, temp):
    """The factor on a query: one plus coef times the logarithm of how many runs of `every` positions have begun."""
    if not temp:
        return np.ones(len(positions))
    return np.array([1.0 + temp["coef"] * math.log((p + 1) // temp["every"] + 1) for p in positions])


def sigmoid_attention(h, w, p, m, eps):
    """Grouped heads without rotation; q and k normed over the whole projection, q scaled by position; a learned bias by
    distance and head on every score; each key's weight is the sigmoid of its own score; a gate per head."""
    n = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_unit(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]
    k = rms_unit(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(n, G, dv)
    q = (q * query_temperature(range(n), m.get("q_temp"))[:, None]).reshape(n, H, dk)
    k = k.reshape(n, G, dk)
    gate = sigmoid(h @ w[p + "g"].T)
    table = w[p + "rel"]
    by_distance = table[[distance_bucket(d, table.shape[0], m["bias_max"]) for d in range(n)]]         # [distance, head]
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen, distance = j <= i, np.maximum(i - j, 0)
    out = np.zeros((n, H, dv))
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T) * m["scale"] + by_distance[distance, head] + w[p + "pb"][head]
        out[:, head] = np.where(seen, sigmoid(s), 0.0) @ v[:, g] * gate[:, head][:, None]
    return out.reshape(n, H * dv) @ w[p + "o"].T


# ---- recurrences ---------------------------------------------------------------------------------------------------
def lightning_attention(h, w, p, m, eps):
    """A state [dim, vdim] per head that fades by a constant of the head and takes in k v^T, read with q."""
    n = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(n, H, dk)
    k = silu(h @ w[p + "k"].T).reshape(n, H, dk)
    v = silu(h @ w[p + "v"].T).reshape(n, H, dv)
    out = np.zeros((n, H, dv))
    for head in range(H):
        S = np.zeros((dk, dv))
        for t in range(n):
            S = m["decay"][head] * S + np.outer(k[t, head], v[t, head])
            out[t, head] = S.T @ q[t, head]
    y = rms_unit(out.reshape(n, H * dv), eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


def general_delta(h, w, p, m, eps):
    """The delta rule with a decay and a removal rate per head and key channel: the state's rows decay, what it holds along
    the unit key is taken off at the channel's rate, and the (unnormed) key writes the value; both read the old state."""
    n = h.shape[0]
    H, dk = m["heads"], m["dim"]
    r = (h @ w[p + "r"].T).reshape(n, H, dk)
    k = (h @ w[p + "k"].T).reshape(n, H, dk)
    v = (h @ w[p + "v"].T).reshape(n, H, dk)
    decay = np.exp(-math.exp(-0.5) * sigmoid(np.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).reshape(n, H, dk)
    rate = sigmoid(h @ w[p + "a"].T + w[p + "a.b"]).reshape(n, H, dk)
    u = k / np.sqrt((k * k).sum(axis=-1, keepdims=True) + 1e-6)
    out = np.zeros((n, H, dk))
    for head in range(H):
        S = np.zeros((dk, dk))
        for t in range(n):
            held = S.T @ u[t, head]
            S = decay[t, head][:, None] * S - np.outer(rate[t, head] * u[t, head], held) + np.outer(k[t, head], v[t, head])
            out[t, head] = S.T @ r[t, head]
    y = rms_unit(out, eps).reshape(n, H * dk) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    """Two mixers read the same rows; each output is normed over the width with a gain, and the mean of the two goes on."""
    left = rms_unit(sigmoid_attention(h, w, p + "left.", m["left"], eps), eps) * w[p + "left.out"]
    right = rms_unit(lightning_attention(h, w, p + "right.", m["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (left + right)


MIXERS = {"parallel": side_by_side, "general_delta": general_delta}


# ---- feed-forward ---------------------------------------------------------------------------------------------------------
def gated_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# ---- the model --------------------------------------------------------------------------------------------------------------
def forward(config, w, tokens, return_layers=False):
    """Logits [n, vocab] of a whole sequence (and the stream after every layer)."""
    eps, groups = config["norm"]["eps"], config["norm"]["groups"]
    x = w["embed"][np.asarray(tokens)] + wave_positions(range(len(tokens)), config["width"])
    streams = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](group_norm(x, w[p + "norm1"], eps, groups), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + gated_ff(group_norm(x, w[p + "norm2"], eps, groups), w, p + "mlp.")
        streams.append(x.copy())
    logits = group_norm(x, w["final.norm"], eps, groups) @ w["head"].T * config.get("logit_scale", 1.0)
    return (logits, np.stack(streams)) if return_layers else logits


# ---- model folders ------------------------------------------------------------------------------------------------------
def tensor_shapes(config, buckets=8, rank=8):
    """name -> shape of every tensor a model of this configuration has.  The rows of the bias tables and the inner size of
    the decay maps are no keys of the configuration (the tensors' shapes give them): one number for all layers, or a dict
    layer index -> number."""
    of = lambda value, i: value.get(i, 8) if isinstance(value, dict) else value
    d, V = config["width"], config["vocab"]
    shapes = {"embed": (V, d), "final.norm": (d,), "head": (V, d)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        shapes[p + "norm1"] = (d,)
        if layer["type"] == "general_delta":
            n = m["heads"] * m["dim"]
            shapes.update({p + "mix." + name: (n, d) for name in ("r", "k", "v", "g", "a")})
            shapes.update({p + "mix.a.b": (n,), p + "mix.w1": (of(rank, i), d), p + "mix.w2": (n, of(rank, i)), p + "mix.w0": (n,), p + "mix.norm": (n,),
                           p + "mix.o": (d, n)})
        else:
            l, r = m["left"], m["right"]
            nq, nk, nv = l["heads"] * l["dim"], l["kv_heads"] * l["dim"], l["kv_heads"] * l["vdim"]
            a = p + "mix.left."
            shapes.update({a + "q": (nq, d), a + "q.b": (nq,), a + "k": (nk, d), a + "k.b": (nk,), a + "v": (nv, d), a + "v.b": (nv,), a + "q.norm": (nq,),
                           a + "k.norm": (nk,), a + "rel": (of(buckets, i), l["heads"]), a + "pb": (l["heads"],), a + "g": (l["heads"], d),
                           a + "o": (d, l["heads"] * l["vdim"]), a + "out": (d,)})
            a, nk, nv = p + "mix.right.", r["heads"] * r["dim"], r["heads"] * r["vdim"]
            shapes.update({a + "q": (nk, d), a + "k": (nk, d), a + "v": (nv, d), a + "g": (nv, d), a + "norm": (nv,), a + "o": (d, nv), a + "out": (d,)})
        mlp = layer.get("mlp")
        if mlp:
            shapes.update({p + "norm2": (d,), p + "mlp.gate": (mlp["ff"], d), p + "mlp.up": (mlp["ff"], d), p + "mlp.down": (d, mlp["ff"])})
    return shapes


def to_bf16_bits(a):
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16_bits(b):
    return (b.astype(np.uint32) << 16).view(np.float32)


def random_weights(config, seed, overrides=None, buckets=8, rank=8):
    """Random weights (rounded to bfloat16, as a model file stores them) of sizes that keep activations of order one."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(config, buckets, rank).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm", "norm1", "norm2", "out"):
            v = 1.0 + 0.2 * rng.standard_normal(shape)
        elif leaf == "b":
            v = 0.3 * rng.standard_normal(shape)
        elif leaf == "rel":
            v = rng.standard_normal(shape)
        elif leaf == "pb":
            v = -3.0 + rng.standard_normal(shape)                # with order ten to a hundred keys a sum of weights of order one
        elif leaf == "w0":
            v = -2.0 + 1.5 * rng.standard_normal(shape)
        elif leaf == "embed":
            v = rng.standard_normal(shape)
        else:
            v = rng.standard_normal(shape) * (1.5 / math.sqrt(shape[-1]))
        w[name] = from_bf16_bits(to_bf16_bits(v)).astype(np.float64)
    for name, v in (overrides or {}).items():
        w[name] = from_bf16_bits(to_bf16_bits(v)).astype(np.float64)
    return w


def write_model_dir(folder, config, w):
    """config.json and model.safetensors (bfloat16) as the engine reads them."""
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    header, blobs, at = {}, [], 0
    for name in sorted(w):
        raw = to_bf16_bits(w[name]).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(w[name].shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    return folder


def read_model_dir(folder):
    folder = Path(folder)
    config = json.loads((folder / "config.json").read_text())
    raw = (folder / "model.safetensors").read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    w = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        buf = raw[8 + n + lo:8 + n + hi]
        if meta["dtype"] == "BF16":
            a = from_bf16_bits(np.frombuffer(buf, dtype=np.uint16))
        elif meta["dtype"] == "F32":
            a = np.frombuffer(buf, dtype=np.float32)
        else:
            a = np.frombuffer(buf, dtype=np.int32)
        w[name] = a.reshape(meta["shape"]).astype(np.float64)
    return config, w
