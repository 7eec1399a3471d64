"""Random-weights mode for the Mipurax decoder: the names and shapes of the tensors a configuration asks for, and a
writer of a model folder (config.json, model.safetensors in bfloat16) from a configuration and a seed.

Made for models of several gigabytes: matrices are cut out of one pool of random bfloat16 values at offsets drawn
per tensor, so a folder is written at the speed of the disk.  The norms' tensors (gains minus one, and the latents' plain
gains) and the sinks get values of their own.  An attention layer with "kv_from" has no tensors of keys and values.
numpy only.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np


def tensor_shapes(config: dict) -> dict:
    d, vocab = config["width"], config["vocab"]
    shapes = {"embed": (vocab, d), "embed.norm": (d,), "final.norm": (d,)}
    for i, layer in enumerate(config["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        heads, dk, dv = m["heads"], m["dim"], m["vdim"]
        shapes[p + "norm1"] = (d,)
        if layer["type"] == "attention":
            shapes.update({q + "q": (heads * dk, d), q + "o": (d, heads * dv)})
            if m.get("kv_from") is None:
                shapes.update({q + "k": (m["kv_heads"] * dk, d), q + "v": (m["kv_heads"] * dv, d)})
        elif layer["type"] in ("latent_attention", "latent_attention_2"):
            per_head = layer["type"] == "latent_attention_2"
            shapes.update({q + "dq": (m["q_rank"], d), q + "dq.norm": (m["q_rank"],), q + "uq": (heads * (dk + m["rot_dim"]), m["q_rank"]),
                           q + "dkv": (m["kv_rank"] + m["rot_dim"], d), q + "dkv.norm": (m["kv_rank"],), q + "uk": (heads * dk, m["kv_rank"]),
                           q + "uv": (heads * dv, m["kv_rank"]), q + "g": (heads if per_head else heads * dv, d), q + "o": (d, heads * dv)})
            if per_head:
                shapes[q + "sink"] = (heads,)
        else:
            raise ValueError(f"layers[{i}].type '{layer['type']}' is no mixer of this design")
        mlp = layer.get("mlp")
        if not mlp:
            continue
        shapes[p + "norm2"] = (d,)
        if mlp["kind"] == "dense":
            forms = {"mlp.": mlp["ff"]}
        else:
            forms = {f"mlp.e{e}.": mlp["expert"]["ff"] for e in range(mlp["router"]["experts"])}
            shapes[p + "mlp.router"] = (mlp["router"]["experts"], d)
            if mlp.get("shared"):
                forms["mlp.shared."] = mlp["shared"]["ff"]
        for form, ff in forms.items():
            shapes.update({p + form + "up": (ff, d), p + form + "down": (d, ff)})
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
        if name.endswith(("dq.norm", "dkv.norm")):
            return _bf16_bits(np.ones(n))
        if name.endswith(("norm", "norm1", "norm2", "sink")):
            return _bf16_bits(np.zeros(n))                                       # the gain is one plus the tensor; a sink of exp(0)
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
