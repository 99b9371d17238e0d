"""Small Nutatar configurations for the tests and their model folders."""

from __future__ import annotations

import os

import torch


def attention(heads, kv_heads, dim, scale=None, window=None, rot=None, mlp=None, vdim=None):
    m = {"heads": heads, "dim": dim}
    for key, v in (("kv_heads", kv_heads), ("vdim", vdim), ("scale", scale)):
        if v is not None:
            m[key] = v
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def gla(heads, dim, vdim, tau, mlp=None):
    m = {"heads": heads, "dim": dim}
    for key, v in (("vdim", vdim), ("tau", tau)):
        if v is not None:
            m[key] = v
    return {"type": "gla", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale=None, base=10000.0, scaling=None, kv_from=None, mlp=None):
    """``scaling``: (factor, original, fast, slow)."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "rot": {"dims": rot_dim, "base": base}}
    if scale is not None:
        m["scale"] = scale
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, limit=None, shared=None):
    """``groups``: (count, keep); ``shared``: (ff, limit)."""
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups is not None:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if limit is not None:
        m["expert"]["limit"] = limit
    if shared is not None:
        m["shared"] = {"ff": shared[0]}
        if shared[1] is not None:
            m["shared"]["limit"] = shared[1]
    return m


RAMP = (4.0, 64, 8.0, 1.0)
# Sizes without a tensor-core variant; a cache read across layers of other kinds, and by two of them; a
# layer without a feed-forward; groups; a shared expert of another width and limit.
CASE_A = {
    "architecture": "Nutatar", "vocab": 211, "width": 96, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0},
    "layers": [latent(4, 12, 6, 20, 28, 24, 0.3, 5000.0, RAMP, mlp=dense(176)),
               attention(6, 3, 20, 0.25, 21, (8, 10000.0), moe(24, 6, 2, (3, 2), 0.9, (40, 1.3))),
               latent(2, 16, 6, 7, 36, 24, 0.25, 5000.0, RAMP, kv_from=0, mlp=None),
               gla(3, 12, 20, 4.0, dense(100)),
               latent(5, 8, 6, 24, 20, 24, 0.35, 5000.0, RAMP, kv_from=0, mlp=moe(20, 5, 3, None, 2.0, (20, 0.5)))]}
# What may be left out is left out; sizes that are 1, equal, or no multiple of 8.
CASE_B = {
    "architecture": "Nutatar", "vocab": 133, "width": 100, "norm": {"eps": 1e-6},
    "layers": [gla(1, 5, None, None, moe(30, 4, 4)),
               attention(3, 1, 10, None, 7, None, dense(52)),
               attention(2, None, 14, 0.4, None, (14, 500.0), moe(17, 3, 1, (3, 1), 0.7)),
               gla(2, 9, 6, 30.0, None),
               latent(1, 10, 4, 6, 12, 16, None, 100.0, mlp=dense(36)),
               attention(4, 4, 6, 0.3, 1, (2, 100.0), moe(12, 6, 2, (2, 2), None, (25, None)))]}
# Sizes the tensor-core kernels take; a shared expert that runs as further columns of the experts' products
# with a limit of its own.
CASE_C = {
    "architecture": "Nutatar", "vocab": 301, "width": 128, "norm": {"eps": 2e-6}, "embedding": {"scale": 2.5},
    "layers": [attention(8, 2, 32, 0.2, 50, (16, 10000.0), moe(32, 8, 3, (4, 2), 1.0, (64, 0.6))),
               gla(4, 32, 48, 16.0, dense(192)),
               latent(8, 16, 16, 32, 48, 32, 0.25, 10000.0, (2.0, 32, 4.0, 1.0), mlp=dense(64)),
               latent(4, 32, 16, 16, 64, 32, 0.2, 10000.0, (2.0, 32, 4.0, 1.0), kv_from=2,
                      mlp=moe(64, 6, 2, (2, 1), 1.5, (64, 1.5))),
               attention(4, 4, 64, 0.15, 33, (64, 2000.0), dense(96))]}
# Larger heads and states; two caches of latents with readers of both; many experts in many groups.
CASE_D = {
    "architecture": "Nutatar", "vocab": 280, "width": 192, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
    "layers": [latent(16, 32, 32, 48, 96, 64, 0.14, 100000.0, (8.0, 256, 16.0, 2.0), mlp=moe(16, 20, 4, (5, 2), 0.9, (48, 0.9))),
               latent(4, 64, 16, 64, 40, 32, 0.12, 1000.0, None, mlp=None),
               latent(8, 16, 32, 32, 64, 64, 0.2, 100000.0, (8.0, 256, 16.0, 2.0), kv_from=0, mlp=dense(256)),
               gla(2, 64, 128, 8.0, moe(64, 4, 2)),
               attention(8, 1, 128, 0.08, 128, (32, 50000.0), dense(320)),
               latent(2, 32, 16, 96, 56, 32, 0.2, 1000.0, None, kv_from=1, mlp=dense(100))]}
CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C, "D": CASE_D}
PAGE_SIZES = {"A": 4, "B": 8, "C": 16, "D": 16}


def random_case(seed: int) -> dict:
    """A configuration drawn at random from sizes a small model might have."""
    import random
    rng = random.Random(seed)
    width = rng.choice([128, 192, 224, 256, 352])
    layers, owners = [], []

    def mlp():
        r = rng.random()
        if r < 0.1:
            return None
        if r < 0.5:
            return dense(rng.choice([96, 128, 200, 320]))
        count = rng.choice([1, 2, 3, 4])
        per = rng.randint(2, 5)
        keep = rng.randint(1, count)
        ff = rng.choice([24, 32, 48, 64])
        return moe(ff, count * per, rng.randint(1, keep * per), (count, keep) if count > 1 or rng.random() < 0.5 else None,
                   rng.choice([None, 0.5, 1.0, 2.0]),
                   rng.choice([None, (ff, 1.0), (2 * ff, 0.7), (ff + 8, None), (80, 2.0)]))

    for i in range(rng.randint(3, 6)):
        kind = rng.choice(["attention", "gla", "latent", "latent"])
        if kind == "attention":
            kv = rng.choice([1, 2, 3, 4])
            dim = rng.choice([16, 24, 32, 48, 64, 80, 128])
            rd = rng.choice([0, dim // 4 * 2, dim])
            layers.append(attention(kv * rng.choice([1, 2, 3, 4]), kv, dim, rng.choice([dim ** -0.5, 0.1, 0.2]),
                                    rng.choice([None, 16, 23, 32, 64, 100]),
                                    (rd, rng.choice([100.0, 10000.0, 250000.0])) if rd else None, mlp()))
        elif kind == "gla":
            layers.append(gla(rng.choice([1, 2, 4, 5]), rng.choice([16, 24, 32, 48, 64]), rng.choice([16, 20, 32, 64, 96]),
                              rng.choice([1.0, 4.0, 16.0]), mlp()))
        else:
            heads, dim, vdim = rng.choice([1, 2, 4, 8, 12]), rng.choice([16, 24, 32, 64]), rng.choice([16, 24, 32, 48])
            q_rank, scale = rng.choice([24, 40, 64, 72]), rng.choice([0.1, 0.2, 0.3])
            if owners and rng.random() < 0.6:
                at = rng.choice(owners)
                m = layers[at]["mixer"]
                layers.append(latent(heads, dim, m["rot_dim"], vdim, q_rank, m["kv_rank"], scale, kv_from=at, mlp=mlp()))
                layers[-1]["mixer"]["rot"] = m["rot"]
            else:
                owners.append(i)
                layers.append(latent(heads, dim, rng.choice([8, 16, 32]), vdim, q_rank, rng.choice([16, 32, 40, 64, 96]), scale,
                                     rng.choice([100.0, 10000.0, 500000.0]),
                                     rng.choice([None, (4.0, 64, 8.0, 1.0), (2.0, 512, 32.0, 1.0), (1.0, 128, 4.0, 2.0)]),
                                     mlp=mlp()))
    return {"architecture": "Nutatar", "vocab": rng.choice([150, 211, 300]), "width": width,
            "norm": {"eps": rng.choice([1e-5, 1e-6])}, "embedding": {"scale": rng.choice([1.0, 4.0, 12.0])}, "layers": layers}


CODE = 12  # columns of the stream that hold a token's routing code in a steady model


def margin(z: torch.Tensor, top: int, count: int, keep: int) -> float:
    """How far a token's choice of experts is from another one, in router logits."""
    import plain_nutatar as pn
    E = len(z)
    per = E // count
    best = torch.stack([z[g * per: (g + 1) * per].max() for g in range(count)])
    order = torch.sort(best, descending=True).values
    gap = float(order[keep - 1] - order[keep]) if keep < count else float("inf")
    chosen = {e for e, _ in pn.route(z, top, count, keep)}
    groups = set(torch.argsort(best, descending=True)[:keep].tolist())
    rest = [float(z[e]) for e in range(E) if e // per in groups and e not in chosen]
    if rest:
        gap = min(gap, min(float(z[e]) for e in chosen) - max(rest))
    return gap


def steady_routing(tensors, config: dict, seed: int) -> None:
    """Routers that read a code of the token which no layer writes over, with choices far from one another:
    bfloat16 rounding elsewhere in the model then cannot flip an expert.  The stream's first CODE columns keep
    what the embedding put there (the norms on the sub-layers' results are zero in them)."""
    g = torch.Generator().manual_seed(seed + 5)
    vocab, scale = config["vocab"], (config.get("embedding") or {}).get("scale", 1.0)
    routers = []
    for i, layer in enumerate(config["layers"]):
        for n in ("norm1", "norm2"):
            if f"l{i}.{n}" in tensors:
                tensors[f"l{i}.{n}"][:CODE] = 0.0
        f = layer.get("mlp")
        if f and f["kind"] == "moe":
            r = f["router"]
            w = torch.randn(r["experts"], CODE, generator=g) * 0.5
            full = tensors[f"l{i}.mlp.router"].float() * 0.02
            full[:, :CODE] = w.bfloat16().float()
            tensors[f"l{i}.mlp.router"] = full.to(torch.bfloat16)
            gr = r.get("groups") or {"count": 1, "keep": 1}
            routers.append((full[:, :CODE].double(), r["top"], gr["count"], gr.get("keep", gr["count"])))
    embed = tensors["embed"].float()
    for t in range(vocab):
        best, at = -1.0, None
        for _ in range(60):
            code = (torch.randint(-8, 9, (CODE,), generator=g).float() / 4.0 / scale).bfloat16()
            m = min([margin(w @ (code.double() * scale), top, c, k) for w, top, c, k in routers] or [9.0])
            if m > best:
                best, at = m, code
            if best > 0.3:
                break
        embed[t, :CODE] = at.float()
    tensors["embed"] = embed.to(torch.bfloat16)


def make_folder(folder: str, config: dict, seed: int, sharpen: float = 0.0, steady: bool = False, drop=None,
                add=None) -> str:
    """A random model through the package's writer, reshaped so that faults show: a stream of size one,
    projections that keep it, gates and ups that reach their limits, decays that differ.  ``sharpen``
    multiplies the attention mixers' ``scale`` so that the softmax is peaked and one wrong key shows in the
    logits.  ``steady``: routing far from close calls.  ``drop`` / ``add``: tensors taken out of the file, or
    put in (name -> shape)."""
    import json

    from infernum_b200.weights.random_init import write_random_model
    from safetensors.torch import load_file, save_file

    if sharpen:
        config = json.loads(json.dumps(config))
        for layer in config["layers"]:
            m = layer["mixer"]
            if layer["type"] != "gla":
                m["scale"] = (m["scale"] if m.get("scale") is not None else
                              (m["dim"] + m.get("rot_dim", 0)) ** -0.5) * sharpen
    write_random_model(folder, config, seed)
    path = os.path.join(folder, "model.safetensors")
    tensors = load_file(path)
    for name in list(tensors):
        t = tensors[name].float()
        if name == "embed":
            t = t * (50.0 / (config.get("embedding") or {}).get("scale", 1.0))
        elif t.dim() == 2 and name != "head":
            gain = 2.0 if name.endswith((".gate", ".up", ".a2", ".mix.g", ".router")) else 1.0
            t = t / t.std().clamp(min=1e-6) * gain * t.shape[1] ** -0.5
        else:
            continue
        tensors[name] = t.to(torch.bfloat16)
    if steady:
        steady_routing(tensors, config, seed)
    for name in drop or []:
        del tensors[name]
    for name, shape in (add or {}).items():
        tensors[name] = torch.ones(shape, dtype=torch.bfloat16)
    save_file(tensors, path, metadata={"format": "pt"})
    return folder
