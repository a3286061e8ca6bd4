"""Folders with config.json and model.safetensors, written and read without the product's loader."""
import json
import os
import struct

import numpy as np
import torch


def write_model(folder, config, weights):
    """config.json and model.safetensors."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    head, off, blobs = {}, 0, []
    for n in sorted(weights):
        b = weights[n].contiguous().view(torch.int16).numpy().tobytes()
        head[n] = {"dtype": "BF16", "shape": list(weights[n].shape), "data_offsets": [off, off + len(b)]}
        off += len(b)
        blobs.append(b)
    j = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(j)) + j + b"".join(blobs))


def read_model(folder):
    with open(os.path.join(folder, "config.json")) as f:
        c = json.load(f)
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head, raw = json.loads(f.read(n)), f.read()
    w = {}
    for k, e in head.items():
        if k != "__metadata__":
            a, b = e["data_offsets"]
            w[k] = torch.from_numpy(np.frombuffer(raw[a:b], np.int16).copy()).view(torch.bfloat16).reshape(e["shape"])
    return c, w
