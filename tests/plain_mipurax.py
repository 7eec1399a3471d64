"""Plain, slow restatement of the Mipurax decoder in numpy float64: whole sequences, no cache, no batching, one
function per mechanism.  It shares nothing with the engine and is what the engine's results are held against.

A model is (config, weights): ``config`` the parsed config.json, ``weights`` a dict name -> float64 array.

Notation: n tokens, d the model width; a linear map stored [out, in] is applied as ``x @ W.T``; positions count from 0.
The stream starts as N(embed[token]); a layer is  x += mixer(N1(x)); x += ff(N2(x))  with N(y) = y / rms(y) * (1 + w);
the logits are embed N(x).
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np

_erf = np.frompyfunc(math.erf, 1, 1)


# ---- elementwise pieces -------------------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu(z):
    """z times the normal distribution's integral up to z."""
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)).astype(np.float64))


def rms_unit(x, eps):
    """x over its root mean square along the last axis, eps under the root."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def offset_norm(y, gain, eps):
    """The model's norm: the tensor holds the gain's distance from one."""
    return rms_unit(y, eps) * (1.0 + gain)


# ---- rotation -------------------------------------------------------------------------------------------------------------
def rotate(v, positions, rot, interleaved):
    """v [n, heads, dim]: of the first dims values, pairs (2i, 2i+1) (interleaved) or (i, i + dims/2) are turned by the angle
    position * base^(-2 i / dims); the rest pass."""
    dims, base = rot["dims"], rot["base"]
    if not dims:
        return v
    half = dims // 2
    f = base ** (-2.0 * np.arange(half, dtype=np.float64) / dims)
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    first = slice(0, dims, 2) if interleaved else slice(0, half)
    second = slice(1, dims, 2) if interleaved else slice(half, dims)
    out = v.copy()
    out[..., first] = v[..., first] * c - v[..., second] * s
    out[..., second] = v[..., second] * c + v[..., first] * s
    return out


# ---- which keys a query sees, and how they weigh ----------------------------------------------------------------------------
def seen_all(n):
    return np.arange(n)[None, :] <= np.arange(n)[:, None]


def seen_chunk(n, size):
    """Keys of the query's own block of `size` positions, blocks counted from position 0."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & (i // size == j // size)


def slopes(heads):
    """What a step of distance takes off a head's scores: powers of 2^(-8/heads)."""
    return 2.0 ** (-8.0 * np.arange(1, heads + 1) / heads)


def softmax_rows(s, seen, sink=None):
    """Weights over the seen keys of every row; a sink is one more term of the sum, with no key and no value."""
    s = np.where(seen, s, -np.inf)
    top = s.max(axis=1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(s - top)
    total = e.sum(axis=1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - top)
    return e / total


# ---- the mixers -----------------------------------------------------------------------------------------------------------
def latent_attention(h, w, p, m, eps, interleaved, sinks, gate_per_head):
    """Queries, keys and values expanded from normed latents; one rotated key part for all heads; a gate on the heads'
    outputs, a number per value or per head."""
    n = h.shape[0]
    H, dn, dr, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(n)
    cq = rms_unit(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(n, H, dn + dr)
    down = h @ w[p + "dkv"].T
    c = rms_unit(down[:, :rank], eps) * w[p + "dkv.norm"]
    k_rot = rotate(down[:, None, rank:], pos, m["rot"], interleaved)[:, 0]
    q_rot = rotate(q[..., dn:], pos, m["rot"], interleaved)
    k = (c @ w[p + "uk"].T).reshape(n, H, dn)
    v = (c @ w[p + "uv"].T).reshape(n, H, dv)
    gate = sigmoid(h @ w[p + "g"].T)
    seen = seen_all(n)
    out = np.zeros((n, H, dv))
    for head in range(H):
        s = (q[:, head, :dn] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * m["scale"]
        out[:, head] = softmax_rows(s, seen, sink=w[p + "sink"][head] if sinks else None) @ v[:, head]
    if gate_per_head:
        return (out * gate[:, :, None]).reshape(n, H * dv) @ w[p + "o"].T
    return (out.reshape(n, H * dv) * gate) @ w[p + "o"].T


def project_keys(h, w, p, m):
    n = h.shape[0]
    return (h @ w[p + "k"].T).reshape(n, m["kv_heads"], m["dim"]), (h @ w[p + "v"].T).reshape(n, m["kv_heads"], m["vdim"])


def sloped_attention(h, w, p, m, k, v):
    """Grouped heads without rotation; the scores lose slope * distance; keys of the query's own block of positions."""
    n = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].T).reshape(n, H, m["dim"])
    seen = seen_chunk(n, m["mask"]["size"]) if m.get("mask") else seen_all(n)
    distance = np.arange(n)[:, None] - np.arange(n)[None, :]
    out = np.zeros((n, H, m["vdim"]))
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].T) * m["scale"] - slopes(H)[head] * distance
        out[:, head] = softmax_rows(s, seen) @ v[:, g]
    return out.reshape(n, H * m["vdim"]) @ w[p + "o"].T


# ---- the feed-forwards ------------------------------------------------------------------------------------------------------
def gelu_ff(h, w, p):
    return gelu(h @ w[p + "up"].T) @ w[p + "down"].T


def choose_experts(s, router):
    """The indices of the chosen experts of one token from its scores s: the `top` largest within the best groups, a group
    counting the sum of its two largest scores."""
    allowed = np.ones(len(s), dtype=bool)
    groups = router.get("groups")
    if groups:
        per = len(s) // groups["count"]
        value = [np.sort(s[g * per:(g + 1) * per])[::-1][:2].sum() for g in range(groups["count"])]
        best = np.argsort(-np.asarray(value), kind="stable")[:groups["keep"]]
        allowed[:] = False
        for g in best:
            allowed[g * per:(g + 1) * per] = True
    return np.argsort(-np.where(allowed, s, -np.inf), kind="stable")[:router["top"]]


def moe(h, w, p, mlp):
    """Sigmoid scores, the chosen ones' shares of their sum as weights, a shared expert beside them."""
    s = sigmoid(h @ w[p + "router"].T)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose_experts(s[t], mlp["router"])
        share = s[t][ids] / (s[t][ids].sum() + 1e-20)
        for e, a in zip(ids, share):
            out[t] += a * gelu_ff(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out += gelu_ff(h, w, p + "shared.")
    return out


# ---- the model ----------------------------------------------------------------------------------------------------------------
def forward(config, w, tokens, return_layers=False):
    """Logits [n, vocab] for one whole sequence (and, if asked, the stream after every layer)."""
    eps = config["norm"]["eps"]
    x = offset_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    streams, kept = [], {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = offset_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            x = x + latent_attention(h, w, p + "mix.", m, eps, interleaved=True, sinks=False, gate_per_head=False)
        elif layer["type"] == "latent_attention_2":
            x = x + latent_attention(h, w, p + "mix.", m, eps, interleaved=False, sinks=True, gate_per_head=True)
        elif layer["type"] == "attention":
            if m.get("kv_from") is None:
                kept[i] = project_keys(h, w, p + "mix.", m)
            k, v = kept[i if m.get("kv_from") is None else m["kv_from"]]
            x = x + sloped_attention(h, w, p + "mix.", m, k, v)
        else:
            raise ValueError(layer["type"])
        mlp = layer.get("mlp")
        if mlp:
            h = offset_norm(x, w[p + "norm2"], eps)
            x = x + (gelu_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else moe(h, w, p + "mlp.", mlp))
        streams.append(x.copy())
    y = offset_norm(x, w["final.norm"], eps) @ w["embed"].T
    return (y, np.stack(streams)) if return_layers else y


# ---- model folders ------------------------------------------------------------------------------------------------------
def tensor_shapes(config):
    """name -> shape of every tensor a model of this configuration has."""
    d, V = config["width"], config["vocab"]
    shapes = {"embed": (V, d), "embed.norm": (d,), "final.norm": (d,)}
    for i, layer in enumerate(config["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        shapes[p + "norm1"] = (d,)
        if layer["type"] == "attention":
            shapes.update({q + "q": (H * dk, d), q + "o": (d, H * dv)})
            if m.get("kv_from") is None:
                shapes.update({q + "k": (m["kv_heads"] * dk, d), q + "v": (m["kv_heads"] * dv, d)})
        else:
            second, dr, rank, q_rank = layer["type"] == "latent_attention_2", m["rot_dim"], m["kv_rank"], m["q_rank"]
            shapes.update({q + "dq": (q_rank, d), q + "dq.norm": (q_rank,), q + "uq": (H * (dk + dr), q_rank), q + "dkv": (rank + dr, d),
                           q + "dkv.norm": (rank,), q + "uk": (H * dk, rank), q + "uv": (H * dv, rank), q + "o": (d, H * dv),
                           q + "g": (H if second else H * dv, d)})
            if second:
                shapes[q + "sink"] = (H,)
        mlp = layer.get("mlp")
        if mlp:
            shapes[p + "norm2"] = (d,)
            forms = {"mlp.": mlp["ff"]} if mlp["kind"] == "dense" else {f"mlp.e{e}.": mlp["expert"]["ff"] for e in range(mlp["router"]["experts"])}
            if mlp.get("shared"):
                forms["mlp.shared."] = mlp["shared"]["ff"]
            for form, ff in forms.items():
                shapes.update({p + form + "up": (ff, d), p + form + "down": (d, ff)})
            if mlp["kind"] == "moe":
                shapes[p + "mlp.router"] = (mlp["router"]["experts"], d)
    return shapes


def to_bf16_bits(a):
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16_bits(b):
    return (b.astype(np.uint32) << 16).view(np.float32)


def random_weights(config, seed, overrides=None):
    """Random weights (rounded to bfloat16, as a model file stores them) of sizes that keep activations of order one."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        if name.endswith(("dq.norm", "dkv.norm")):
            v = 1.0 + 0.2 * rng.standard_normal(shape)
        elif leaf in ("norm1", "norm2", "norm"):
            v = 0.2 * rng.standard_normal(shape)                 # the gain is one plus this
        elif leaf == "sink":
            v = 2.0 + rng.standard_normal(shape)                 # as much as several keys: a sink that is left out shows
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
