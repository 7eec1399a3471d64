"""Random-weights mode for the Zodosun decoder: the names and shapes of the tensors a configuration asks for, and a
writer of a model folder (config.json, model.safetensors in bfloat16) from a configuration and a seed.

Made for models of several gigabytes: matrices are cut out of one pool of random bfloat16 values at offsets drawn
per tensor, so a folder is written at the speed of the disk.  Constants that must be sane for the model to run
(norm gains, the number added to every score, the decays' biases) get values of their own.  The rows of a distance-bias
table and the inner size of a decay map are no keys of the configuration: `buckets` (default 32) and a delta mixer's
"rank" (default 64).  numpy only.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np


def tensor_shapes(config: dict, buckets: int = 32) -> dict:
    d, vocab = config["width"], config["vocab"]
    shapes = {"embed": (vocab, d), "final.norm": (d,), "head": (vocab, d)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        shapes[p + "norm1"] = (d,)
        if layer["type"] == "general_delta":
            n, rank, q = m["heads"] * m["dim"], m.get("rank", 64), p + "mix."
            shapes.update({q + name: (n, d) for name in ("r", "k", "v", "g", "a")})
            shapes.update({q + "a.b": (n,), q + "w1": (rank, d), q + "w2": (n, rank), q + "w0": (n,), q + "norm": (n,), q + "o": (d, n)})
        elif layer["type"] == "parallel":
            left, right = m["left"], m["right"]
            q, heads = p + "mix.left.", left["heads"]
            nq, nk, nv = heads * left["dim"], left["kv_heads"] * left["dim"], left["kv_heads"] * left["vdim"]
            shapes.update({q + "q": (nq, d), q + "q.b": (nq,), q + "k": (nk, d), q + "k.b": (nk,), q + "v": (nv, d), q + "v.b": (nv,), q + "q.norm": (nq,),
                           q + "k.norm": (nk,), q + "rel": (buckets, heads), q + "pb": (heads,), q + "g": (heads, d), q + "o": (d, heads * left["vdim"]),
                           q + "out": (d,)})
            q, nk, nv = p + "mix.right.", right["heads"] * right["dim"], right["heads"] * right["vdim"]
            shapes.update({q + "q": (nk, d), q + "k": (nk, d), q + "v": (nv, d), q + "g": (nv, d), q + "norm": (nv,), q + "o": (d, nv), q + "out": (d,)})
        else:
            raise ValueError(f"layers[{i}].type '{layer['type']}' is no mixer of this design")
        mlp = layer.get("mlp")
        if mlp:
            shapes.update({p + "norm2": (d,), p + "mlp.gate": (mlp["ff"], d), p + "mlp.up": (mlp["ff"], d), p + "mlp.down": (d, mlp["ff"])})
    return shapes


def _bf16_bits(a: np.ndarray) -> np.ndarray:
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def write_random_model(folder, config: dict, seed: int, std: float = 0.02) -> Path:
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    shapes = tensor_shapes(config)
    rng = np.random.default_rng(seed)
    pool = _bf16_bits(rng.standard_normal(1 << 24) * std)
    (folder / "config.json").write_text(json.dumps(config, indent=1))

    def values(name, shape):
        n = int(np.prod(shape))
        leaf = name.split(".")[-1]
        if leaf in ("norm", "norm1", "norm2", "out"):
            return _bf16_bits(np.ones(n))
        if leaf == "pb":
            return _bf16_bits(np.full(n, -6.0))                                  # a few hundred keys then weigh about one together
        if leaf == "w0":
            return _bf16_bits(rng.uniform(-8.0, -1.0, n))                        # decays between 0.85 and 0.9998
        if leaf == "rel":
            return _bf16_bits(rng.standard_normal(n))
        out = np.empty(n, dtype=np.uint16)
        at = 0
        while at < n:
            take = min(n - at, len(pool) // 2)
            start = int(rng.integers(0, len(pool) - take))
            out[at:at + take] = pool[start:start + take]
            at += take
        return out

    header, at = {}, 0
    for name, shape in shapes.items():
        size = int(np.prod(shape)) * 2
        header[name] = {"dtype": "BF16", "shape": list(shape), "data_offsets": [at, at + size]}
        at += size
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head)
        for name, shape in shapes.items():
            f.write(values(name, shape).tobytes())
    return folder
