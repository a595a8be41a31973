"""A plain, slow statement of the Razevik forward pass: one whole sequence at a time, no cache, no batch, one
function per mechanism, torch on the CPU only (float64 unless told otherwise).  It shares no code with
`reinfer_b200`; the tests compare the engine with it.

Notation.  x is the residual stream [T, width]; `lin(x, W) = x W^T` with W stored [out, in];
rms(v) = v / sqrt(mean(v^2) + eps); m is `residual_mult`.  One layer:

    x <- x + m (mixer(rms(x) * w1) + ff(rms(x) * w2))           (ff may be missing)
    x <- x + m rms(P (gelu_tanh(G x) * e_i[token])) * w3        the token's own row for this layer

with x = embed[token] + pos[position] before the first layer and cap * tanh(lin(rms(x) * w, head) / cap) behind the
last.  The mixer is latent attention without positions whose heads' outputs take one gate each; a layer may use
the latent of an earlier layer.  Feed-forwards: dense with squared relu, or a mixture of gelu experts taken from
the first-ranked groups, with a shared expert beside them.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import numpy as np
import torch


# ---------------------------------------------------------------- file reading
def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        raw = f.read()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    data = raw[8 + n:]
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        b, en = e["data_offsets"]
        if e["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(data[b:en], dtype="<f4").copy()).double()
        elif e["dtype"] == "BF16":
            u = np.frombuffer(data[b:en], dtype="<u2").astype(np.uint32) << 16
            t = torch.from_numpy(u.view(np.float32).copy()).double()
        else:
            raise ValueError(f"{name}: dtype {e['dtype']}")
        out[name] = t.reshape(e["shape"])
    return out


def read_model(model_dir: str):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


# ---------------------------------------------------------------- small pieces
def lin(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return x @ w.t()


def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) ** 2


# ---------------------------------------------------------------- attention
def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, d], k [T, d], v [T, dv] of one head: position i sees every j <= i."""
    T = q.shape[0]
    s = (q @ k.t()) * scale
    i = torch.arange(T)
    s = s.masked_fill(i[None, :] > i[:, None], float("-inf"))
    return torch.softmax(s, dim=-1) @ v


def latent_of(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    return rms(lin(h, w[p + "dkv"]), eps) * w[p + "dkv.norm"]


def latent_attention(h: torch.Tensor, c: torch.Tensor, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """c: the latent rows [T, kv_rank] the layer works with (its own or an earlier layer's)."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    cq = rms(lin(h, w[p + "dq"]), eps) * w[p + "dq.norm"]
    q = lin(cq, w[p + "uq"]).view(T, H, d)
    k = lin(c, w[p + "uk"]).view(T, H, d)
    v = lin(c, w[p + "uv"]).view(T, H, dv)
    gate = torch.sigmoid(lin(h, w[p + "g"]))                            # [T, H]: one number per token and head
    heads = [softmax_attention(q[:, hd], k[:, hd], v[:, hd], m["scale"]) * gate[:, hd:hd + 1] for hd in range(H)]
    return lin(torch.cat(heads, dim=-1), w[p + "o"])


# ---------------------------------------------------------------- feed-forwards
def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(relu_squared(lin(h, w[p + "up"])), w[p + "down"])


def route(z: torch.Tensor, correction: torch.Tensor, top: int, groups: Optional[dict]):
    """One token's router outputs z [E] -> (chosen experts, their weights)."""
    E = z.shape[0]
    s = torch.sigmoid(z)
    choice = (s + correction).tolist()
    allowed = set(range(E))
    if groups is not None:
        size = E // groups["count"]
        score = [sum(sorted(choice[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(groups["count"])]
        best = sorted(range(groups["count"]), key=lambda g: -score[g])[:groups["keep"]]
        allowed = {e for g in best for e in range(g * size, (g + 1) * size)}
    chosen = sorted(allowed, key=lambda e: -choice[e])[:top]
    wt = s[chosen]
    return chosen, wt / (wt.sum() + 1e-20)


def expert(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(gelu_erf(lin(h, w[p + "up"])), w[p + "down"])


def shared_expert(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return torch.sigmoid(lin(h, w[p + "sg"])) * expert(h, w, p)


def expert_mixture(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    z = lin(h, w[p + "router"])
    out = shared_expert(h, w, p + "shared.") if mlp.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, wt = route(z[t], w[p + "correction"], r["top"], r.get("groups"))
        for e, a in zip(chosen, wt):
            out[t] = out[t] + a * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


def feed_forward(h, w, p, mlp):
    return dense_ff(h, w, p) if mlp["kind"] == "dense" else expert_mixture(h, w, p, mlp)


# ---------------------------------------------------------------- the token's own row of a layer
def token_side(x: torch.Tensor, rows: torch.Tensor, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    """rows [T, dim]: the tokens' rows for this layer."""
    y = lin(gelu_tanh(lin(x, w[p + "gate"])) * rows, w[p + "proj"])
    return rms(y, eps) * w[p + "norm"]


# ---------------------------------------------------------------- the model
def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, dtype=torch.float64, trace: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence.  `trace`, if a list, gets the stream after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    ids = torch.as_tensor(tokens, dtype=torch.long)
    T = ids.shape[0]
    eps, m, dim = cfg["norm"]["eps"], cfg["residual_mult"], cfg["token_side"]["dim"]
    x = w["embed"][ids] + w["pos"][:T]
    latents: Dict[int, torch.Tensor] = {}
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h1 = rms(x, eps) * w[p + "norm1"]
        src = L["mixer"].get("kv_from")
        latents[i] = latent_of(h1, w, p + "mix.", eps) if src is None else latents[src]
        y = latent_attention(h1, latents[i], w, p + "mix.", L["mixer"], eps)
        if L.get("mlp") is not None:
            y = y + feed_forward(rms(x, eps) * w[p + "norm2"], w, p + "mlp.", L["mlp"])
        x = x + m * y
        x = x + m * token_side(x, w["side.embed"][ids][:, i * dim:(i + 1) * dim], w, p + "side.", eps)
        if trace is not None:
            trace.append(x.clone())
    z = lin(rms(x, eps) * w["final.norm"], w["head"])
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z
