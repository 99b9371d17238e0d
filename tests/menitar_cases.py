"""Small Menitar configurations for the tests and their model folders."""

from __future__ import annotations

import os

import torch


def attention(heads, kv_heads, dim, vdim, scale=None, chunk=None, rot=None, mlp=None):
    m = {"heads": heads, "dim": dim}
    if kv_heads is not None:
        m["kv_heads"] = kv_heads
    if vdim is not None:
        m["vdim"] = vdim
    if scale is not None:
        m["scale"] = scale
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def dense(ff, limit=None):
    m = {"kind": "dense", "ff": ff}
    if limit is not None:
        m["limit"] = limit
    return m


# Sizes without a tensor-core variant beside ones with it; values narrower and wider than keys; one head,
# one key/value head, as many key/value heads as heads; runs of positions of several lengths and none;
# rotation of a part, of all, of nothing; a layer without a feed-forward; a loop behind the first layer.
CASE_A = {
    "architecture": "Menitar", "vocab": 211, "width": 96, "logit_scale": 1.5, "norm": {"eps": 1e-5},
    "embedding": {"scale": 4.0}, "loop": {"start": 1, "stop": 3, "times": 3},
    "layers": [attention(4, 2, 16, 24, 0.3, 21, (8, 10000.0), dense(176, 0.8)),
               attention(6, 3, 12, 12, 0.25, 13, (12, 500.0), dense(64, 1.25)),
               attention(1, 1, 20, 16, 0.2, None, None, None),
               attention(8, 8, 8, 32, 0.35, 64, (4, 100.0), dense(40, 3.0))]}
# What may be left out is left out; no loop; widths that are no multiple of 8 (two products end a layer).
CASE_B = {
    "architecture": "Menitar", "vocab": 133, "width": 100, "norm": {"eps": 1e-6},
    "layers": [attention(3, 1, 10, 6, None, 7, (4, 1000.0), dense(100)),
               attention(2, None, 14, None, None, None, (14, 10000.0), dense(36, 2.0)),
               attention(5, 5, 6, 10, 0.4, 1, None, dense(50, 0.5))]}
# Sizes the tensor-core kernel takes, heads that do and do not fill its pieces; every layer in the loop.
CASE_C = {
    "architecture": "Menitar", "vocab": 301, "width": 128, "logit_scale": 0.5, "norm": {"eps": 2e-6},
    "embedding": {"scale": 2.5}, "loop": {"start": 0, "stop": 3, "times": 2},
    "layers": [attention(8, 2, 32, 48, 0.2, 50, (16, 10000.0), dense(192, 1.0)),
               attention(12, 4, 16, 32, 0.3, 17, (16, 2000.0), dense(128, 0.7)),
               attention(5, 5, 64, 16, 0.15, 33, (32, 10000.0), dense(96, 1.5))]}
# Larger head counts; runs longer than most requests, none at all; a loop of one pass.
CASE_D = {
    "architecture": "Menitar", "vocab": 280, "width": 192, "logit_scale": 3.0, "norm": {"eps": 1e-5},
    "embedding": {"scale": 1.0}, "loop": {"start": 1, "stop": 2, "times": 1},
    "layers": [attention(16, 4, 64, 64, 0.12, 128, (64, 50000.0), dense(256, 0.9)),
               attention(32, 8, 32, 32, 0.2, None, (8, 10000.0), dense(320, 1.1)),
               attention(10, 1, 16, 80, 0.25, 40, (16, 100.0), None)]}
CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C, "D": CASE_D}
PAGE_SIZES = {"A": 4, "B": 8, "C": 16, "D": 16}


def random_case(seed: int) -> dict:
    """A configuration drawn at random from sizes a small model might have."""
    import random
    rng = random.Random(seed)
    width = rng.choice([128, 192, 224, 256, 352, 384])
    layers = []
    for _ in range(rng.randint(2, 5)):
        heads = rng.choice([2, 4, 6, 8, 10, 12, 16])
        kv = rng.choice([h for h in (1, 2, 3, 4, 5, 6, 8) if heads % h == 0])
        dim = rng.choice([16, 24, 32, 48, 64, 80])
        rd = rng.choice([0, dim // 4 * 2, dim])
        mlp = dense(rng.choice([96, 128, 200, 320]), rng.choice([None, 0.5, 1.0, 2.0, 7.0])) if rng.random() < 0.85 else None
        layers.append(attention(heads, kv, dim, rng.choice([dim, 16, 32, 48, 64, 96, 128]), rng.choice([dim ** -0.5, 0.1, 0.3]),
                                rng.choice([None, 16, 23, 32, 48, 96, 100]),
                                (rd, rng.choice([100.0, 10000.0, 250000.0])) if rd else None, mlp))
    cfg = {"architecture": "Menitar", "vocab": rng.choice([300, 512, 777, 1000]), "width": width,
           "logit_scale": rng.choice([0.5, 1.0, 4.0]), "norm": {"eps": rng.choice([1e-5, 1e-6])},
           "embedding": {"scale": rng.choice([1.0, 2.0, 6.0])}, "layers": layers}
    if rng.random() < 0.8:
        start = rng.randint(0, len(layers) - 1)
        cfg["loop"] = {"start": start, "stop": rng.randint(start + 1, len(layers)), "times": rng.randint(1, 3)}
    return cfg


def make_folder(folder: str, config: dict, seed: int, sharpen: float = 0.0, drop=None, add=None) -> str:
    """A random model through the package's writer, reshaped so that faults show: values and gates large
    enough to matter, gate and up projections that reach their limits, an exchange that is far from the
    identity.  ``sharpen`` multiplies the mixers' ``scale`` so that the softmax is peaked and one wrong key
    shows in the logits.  ``drop`` / ``add``: tensors taken out of the file, or put in (name -> shape)."""
    import json

    from infernum_b200.weights.random_init import write_random_model
    from safetensors.torch import load_file, save_file

    if sharpen:
        config = json.loads(json.dumps(config))
        for layer in config["layers"]:
            m = layer["mixer"]
            m["scale"] = (m["scale"] if m.get("scale") is not None else m["dim"] ** -0.5) * sharpen
    write_random_model(folder, config, seed)
    path = os.path.join(folder, "model.safetensors")
    tensors = load_file(path)
    for name in list(tensors):
        t = tensors[name].float()
        if name.endswith((".mix.v", ".mix.o", ".mlp.down")):
            t = t * 4.0
        elif name.endswith((".mlp.gate", ".mlp.up", ".mix.g")):
            t = t * 8.0
        elif name == "loop.step":
            t = t * 3.0
        else:
            continue
        tensors[name] = t.to(torch.bfloat16)
    for name in drop or []:
        del tensors[name]
    for name, shape in (add or {}).items():
        tensors[name] = torch.ones(shape, dtype=torch.bfloat16)
    save_file(tensors, path, metadata={"format": "pt"})
    return folder
