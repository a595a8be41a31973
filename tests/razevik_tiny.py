"""Small Razevik configurations for the tests - they differ from one another in every size and option - and weights of the
tests' own making: large enough that every mechanism moves the logits (router outputs that spread, corrections that make
choice scores negative and reorder them, gates well away from one half, token rows as large as the stream)."""
from __future__ import annotations

import json
import math
import os
import random
from typing import Dict, List

import torch


def _lat(heads, dim, vdim, q_rank, kv_rank, scale, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def _layer(mix, mlp):
    return dict(mix, mlp=mlp)


def _cfg(vocab, width, positions, eps, mult, side, layers, cap=None):
    out = {"architecture": "Razevik", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
           "residual_mult": mult, "token_side": {"dim": side}, "layers": layers}
    if cap is not None:
        out["logit_softcap"] = cap
    return out


# A: two latents, each read by later layers of other head counts and sizes (one of them not the next layer), a shared expert
#    larger and one smaller than the experts, groups and no groups, a layer without feed-forward
TINY_A = _cfg(211, 64, 320, 1e-5, 0.45, 12, [
    _layer(_lat(4, 16, 24, 24, 40, 0.3), _dense(72)),
    _layer(_lat(6, 8, 12, 20, 40, 0.4, kv_from=0), _moe(24, 12, 3, (4, 2), shared=40)),
    _layer(_lat(2, 8, 8, 16, 24, 0.5), None),
    _layer(_lat(3, 24, 16, 32, 40, 0.25, kv_from=0), _moe(16, 4, 1, shared=8)),
    _layer(_lat(4, 8, 8, 12, 24, 0.4, kv_from=2), _dense(40))], cap=9.0)
# B: nothing is a multiple of 8 (the aligned products and the tensor-core attention must find their plain forms by
#    themselves), one head, groups of one expert each, every expert chosen, no shared expert, no soft cap, a factor of one
TINY_B = _cfg(97, 52, 200, 1e-6, 1.0, 5, [
    _layer(_lat(3, 10, 7, 11, 13, 0.35), _moe(10, 6, 6, (3, 3))),
    _layer(_lat(1, 6, 9, 5, 13, 0.5, kv_from=0), _moe(9, 5, 2, (5, 4), shared=7)),
    _layer(_lat(5, 3, 5, 7, 9, 0.6), _dense(18))])
# C: sizes the tensor-core kernels take (multiples of 8), sixteen heads on one latent, many experts in many groups, a factor
#    above one
TINY_C = _cfg(130, 96, 300, 1e-6, 1.3, 16, [
    _layer(_lat(16, 16, 8, 32, 48, 0.25), _moe(32, 24, 4, (8, 3), shared=24)),
    _layer(_lat(8, 8, 32, 40, 48, 0.35, kv_from=0), _dense(64)),
    _layer(_lat(2, 32, 16, 24, 64, 0.2), _moe(16, 8, 2, (2, 1), shared=16)),
    _layer(_lat(4, 16, 16, 48, 64, 0.25, kv_from=2), None)], cap=25.0)
# D: what a small real model looks like (width 256, heads of 128, pages of 64): in bfloat16 the products and the attention
#    run on the tensor cores, and longer portions rebuild keys and values per head (not in TINY: its tests name it)
TINY_D = _cfg(500, 256, 700, 1e-5, 0.8, 32, [
    _layer(_lat(4, 128, 128, 192, 192, 0.11), _dense(512)),
    _layer(_lat(2, 128, 128, 64, 192, 0.1, kv_from=0), _moe(64, 16, 4, (4, 2), shared=128)),
    _layer(_lat(3, 128, 128, 128, 64, 0.12), _moe(64, 8, 2, (4, 3), shared=64))], cap=20.0)
TINY = {"A": (TINY_A, 51, 8), "B": (TINY_B, 52, 4), "C": (TINY_C, 53, 16)}      # config, weight seed, page size


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """float32 tensors for every name the model declares, drawn by the tensor's role (read off its name)."""
    from reinfer_b200.config.razevik import RazevikConfig
    from reinfer_b200.models.razevik import build_spec
    from reinfer_b200.parts.model import expected_params
    expected = expected_params(build_spec(RazevikConfig.from_dict(cfg)))
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, ps in expected.items():
        shape = tuple(ps.shape)
        n = lambda std=1.0, mean=0.0: torch.randn(shape, generator=g) * std + mean
        last = name.split(".")[-1]
        if name == "embed":
            t = n(0.8)
        elif name == "pos":
            t = n(0.4)
        elif name == "side.embed":
            t = n(1.5)
        elif "norm" in last:
            t = n(0.15, 1.0)
        elif last == "correction":
            t = n(0.4, -1.0)                # most choice scores are then negative
        elif last in ("router", "sg", "g"):
            t = n(2.0 / math.sqrt(shape[1]))
        else:
            t = n(1.4 / math.sqrt(shape[-1]))
        out[name] = t.float()
    return out


def make_model_dir(path: str, which: str, store_dtype=torch.float32, cfg=None, seed=None, edit=None) -> str:
    from reinfer_b200.weights.safetensors_io import write_safetensors
    base, s, _ = TINY[which] if which in TINY else (cfg, seed, None)
    cfg = cfg or base
    seed = s if seed is None else seed
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    w = make_weights(cfg, seed)
    if edit is not None:
        w = edit(w)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: v.to(store_dtype) for k, v in w.items()})
    return path


def sequences(which: str, lengths=None, seed=7) -> Dict[str, List[int]]:
    cfg = TINY[which][0]
    rnd = random.Random(seed)
    lengths = lengths or {"A": [5, 17, 33, 70, 40, 26, 51], "B": [1, 9, 24, 50, 90, 37, 64, 12], "C": [3, 44, 21, 60, 30]}[which]
    return {f"r{i}": [rnd.randrange(cfg["vocab"]) for _ in range(n)] for i, n in enumerate(lengths)}


def random_config(seed: int) -> dict:
    """A configuration drawn from a seed: two to six layers, each with a latent of its own or any earlier layer's, head counts
    and sizes (also ones the tensor-core kernels pad or refuse), dense feed-forwards, mixtures with and without groups and
    shared experts, or none."""
    rnd = random.Random(seed)
    width = rnd.choice([48, 64, 128, 192])
    layers, owners = [], {}
    for i in range(rnd.randint(2, 6)):
        dim = rnd.choice([8, 12, 16, 32, 64, 128])
        src = rnd.choice(list(owners)) if owners and rnd.random() < 0.5 else None
        rank = owners[src] if src is not None else rnd.choice([16, 20, 24, 56, 64, 96, 136])
        if src is None:
            owners[i] = rank
        mix = _lat(rnd.choice([1, 2, 3, 4, 6, 16]), dim, rnd.choice([8, 16, 20, 48, 128, dim]), rnd.choice([12, 32, 96]), rank,
                   rnd.choice([dim ** -0.5, 0.15]), kv_from=src)
        r = rnd.random()
        if r < 0.15:
            mlp = None
        elif r < 0.4:
            mlp = _dense(rnd.choice([40, 64, 96]))
        else:
            count, size = rnd.choice([1, 2, 4, 5]), rnd.choice([1, 2, 3, 4])
            keep = rnd.randint(1, count)
            mlp = _moe(rnd.choice([8, 24, 32]), count * size, rnd.randint(1, min(keep * size, 4)),
                       (count, keep) if rnd.random() < 0.8 or keep < count else None, rnd.choice([None, 8, 20, 48]))
        layers.append(_layer(mix, mlp))
    return _cfg(rnd.choice([97, 300, 500]), width, 256, rnd.choice([1e-5, 1e-6]), rnd.choice([0.3, 0.9, 1.0, 1.5]), rnd.choice([3, 8, 20, 64]),
                layers, cap=rnd.choice([None, 6.0, 30.0]))
