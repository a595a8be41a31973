"""Small Kibatar configurations for the tests - they differ from one another in every size and option - and weights of the
tests' own making: large enough that every mechanism moves the logits (router outputs that spread, corrections that reorder
the choice, gates and ups beyond their limits, decays from nearly none to nearly all, mixes on both sides of 0 and 1, sinks as
large as the scores)."""
from __future__ import annotations

import json
import math
import os
import random
from typing import Dict, List

import torch


def _lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=10000.0, scaling=None, dims=None):
    rot = {"base": base, "dims": rot_dim if dims is None else dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
                                                  "kv_rank": kv_rank, "scale": scale, "rot": rot}}


def _wkv(heads, dim, decay_rank):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "decay_rank": decay_rank}}


def _moe(ff, limit, experts, top, scale, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def _layer(mix, mlp):
    return dict(mix, mlp=mlp)


def _cfg(vocab, width, eps, emb_scale, bigram, logit_scale, loop, layers):
    out = {"architecture": "Kibatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": emb_scale},
           "logit_scale": logit_scale, "layers": layers}
    if bigram is not None:
        out["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# A: a loop in the middle that starts with attention, a shared expert larger and one smaller than the experts, limits that
#    differ, no frequency scaling beside scaling, value heads of another size, a layer without feed-forward
TINY_A = _cfg(211, 64, 1e-5, 0.7, (83, 7, 5), 0.6, (1, 3, 2), [
    _layer(_wkv(3, 16, 6), _moe(24, 1.2, 6, 2, 1.7, (40, 0.8))),
    _layer(_lat(4, 16, 8, 24, 24, 40, 0.3), _moe(16, 0.9, 5, 1, 2.2, (8, 2.1))),
    _layer(_wkv(2, 24, 5), None),
    _layer(_lat(2, 8, 12, 8, 16, 24, 0.4, base=500.0, scaling=(3.0, 64, 8.0, 1.0)), _moe(20, 1.5, 4, 3, 0.9))])
# B: nothing is a multiple of 8 (the aligned products and the tensor-core attention must find their plain forms by
#    themselves), one head, the loop from the first layer to the last, every expert chosen, factors of one, a part of the rotated
#    part rotated
TINY_B = _cfg(97, 52, 1e-6, 1.0, (31, 2, 3), 1.0, (0, 3, 2), [
    _layer(_lat(1, 10, 6, 7, 11, 13, 0.35, base=200.0, scaling=(2.0, 40, 4.0, 2.0)), _moe(9, 1.1, 3, 3, 1.0, (7, 1.1))),
    _layer(_wkv(1, 13, 3), _moe(10, 0.7, 5, 2, 1.3)),
    _layer(_lat(3, 6, 10, 9, 5, 9, 0.5, dims=6), _moe(11, 1.9, 7, 1, 1.9, (5, 0.6)))])
# C: sizes the tensor-core kernels take, sixteen heads on one latent, a loop of one layer run often, no pair rows' buckets to
#    spare, two recurrent layers in a row
TINY_C = _cfg(130, 128, 1e-6, 1.4, (17, 1, 1), 0.3, (2, 3, 4), [
    _layer(_lat(16, 16, 16, 8, 32, 48, 0.2, base=10000.0, scaling=(8.0, 128, 16.0, 1.0)), _moe(32, 1.4, 12, 4, 2.0, (24, 1.0))),
    _layer(_wkv(4, 32, 16), _moe(16, 1.0, 8, 2, 1.1, (16, 1.6))),
    _layer(_wkv(2, 64, 8), _moe(16, 0.8, 8, 3, 1.5, (16, 0.8))),
    _layer(_lat(4, 32, 32, 32, 48, 64, 0.15), _moe(24, 1.3, 9, 2, 1.2, (32, 1.3)))])
# D: what a small real model looks like (width 256, heads of 64 with a rotated part of 32, pages of 64): in bfloat16 products and
#    attention run on the tensor cores, decode steps take the products' cluster forms (not in TINY: its tests name it)
TINY_D = _cfg(500, 256, 1e-5, 1.0, (251, 11, 3), 0.8, (1, 3, 2), [
    _layer(_lat(4, 64, 32, 64, 96, 128, 0.1, base=50000.0, scaling=(4.0, 256, 32.0, 1.0)), _moe(64, 1.5, 16, 4, 1.8, (128, 1.2))),
    _layer(_wkv(4, 64, 32), _moe(64, 1.5, 16, 4, 1.8, (128, 1.2))),
    _layer(_lat(8, 32, 32, 48, 64, 224, 0.12), _moe(64, 1.0, 8, 2, 1.4, (64, 1.0))),
    _layer(_wkv(2, 128, 16), _moe(96, 1.1, 8, 4, 1.6))])
TINY = {"A": (TINY_A, 61, 8), "B": (TINY_B, 62, 4), "C": (TINY_C, 63, 16)}      # config, weight seed, page size


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """float32 tensors for every name the model declares, drawn by the tensor's role (read off its name)."""
    from reinfer_b200.config.kibatar import KibatarConfig
    from reinfer_b200.models.kibatar import build_spec
    from reinfer_b200.parts.model import expected_params
    expected = expected_params(build_spec(KibatarConfig.from_dict(cfg)))
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, ps in expected.items():
        shape = tuple(ps.shape)
        n = lambda std=1.0, mean=0.0: torch.randn(shape, generator=g) * std + mean
        last, parts = name.split(".")[-1], name.split(".")
        if name in ("embed", "bigram"):
            t = n(0.8)
        elif last.startswith("ls"):
            t = n(0.3, 0.8)
        elif "norm" in last:
            t = n(0.15, 1.0)
        elif "mu" in parts:
            t = n(0.5, 0.5)
        elif last == "w0":
            t = n(1.5, -2.0)                # decays from e^-e to nearly one
        elif last == "u":
            t = n(0.7)
        elif last == "sink":
            t = n(1.0, 1.0)
        elif last == "correction":
            t = n(0.15)
        elif last in ("router", "sg", "g"):
            t = n(1.5 / math.sqrt(shape[1]))
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
    w = make_weights(cfg, seed)
    if edit is not None:
        w = edit(w)
    stored = json.loads(json.dumps(cfg))
    for l in stored["layers"]:
        l["mixer"].pop("decay_rank", None)          # the rank is read off the tensor
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(stored, f)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: v.to(store_dtype) for k, v in w.items()})
    return path


def sequences(which: str, lengths=None, seed=7) -> Dict[str, List[int]]:
    cfg = TINY[which][0]
    rnd = random.Random(seed)
    lengths = lengths or {"A": [5, 17, 33, 70, 40, 26, 51], "B": [1, 9, 24, 50, 90, 37, 64, 12], "C": [3, 44, 21, 60, 30]}[which]
    return {f"r{i}": [rnd.randrange(cfg["vocab"]) for _ in range(n)] for i, n in enumerate(lengths)}


def random_config(seed: int) -> dict:
    """A configuration drawn from a seed: two to five layers of either type, head counts and sizes (also ones the tensor-core
    kernels pad or refuse), mixtures with and without a shared expert, or none, loops anywhere."""
    rnd = random.Random(seed)
    layers = []
    for i in range(rnd.randint(2, 5)):
        if rnd.random() < 0.5:
            mix = _wkv(rnd.choice([1, 2, 3, 4]), rnd.choice([8, 12, 16, 32, 64]), rnd.choice([3, 8, 16, 20]))
        else:
            dim, rot = rnd.choice([8, 12, 16, 32, 64]), rnd.choice([4, 8, 16, 24, 32])
            scaling = rnd.choice([None, (rnd.choice([2.0, 4.0, 16.0]), rnd.choice([32, 128, 2048]), rnd.choice([32.0, 6.0]), rnd.choice([1.0, 2.0]))])
            mix = _lat(rnd.choice([1, 2, 3, 4, 6, 16]), dim, rot, rnd.choice([8, 16, 20, 48, dim]), rnd.choice([12, 32, 96]),
                       rnd.choice([16, 20, 24, 56, 64, 96, 136]), rnd.choice([(dim + rot) ** -0.5, 0.15]),
                       base=rnd.choice([300.0, 10000.0, 1e6]), scaling=scaling)
        experts = rnd.choice([2, 3, 4, 8, 12])
        mlp = None if rnd.random() < 0.15 else _moe(rnd.choice([8, 10, 24, 32]), rnd.choice([0.7, 1.3, 4.0]), experts, rnd.randint(1, min(experts, 4)),
                                                    rnd.choice([1.0, 1.6, 2.5]), rnd.choice([None, (8, 0.9), (20, 1.3), (48, 3.0)]))
        layers.append(_layer(mix, mlp))
    loop = None
    if rnd.random() < 0.8:
        a = rnd.randrange(len(layers))
        loop = (a, rnd.randint(a + 1, len(layers)), rnd.choice([1, 2, 3]))
    return _cfg(rnd.choice([97, 300, 500]), rnd.choice([48, 64, 100, 128, 192]), rnd.choice([1e-5, 1e-6]), rnd.choice([0.5, 1.0, 3.0]),
                rnd.choice([None, (7, 3, 2), (251, 1000003, 7919), (64, 0, 1), (97, 2654435761, 40503)]), rnd.choice([0.4, 1.0, 1.5]), loop, layers)
