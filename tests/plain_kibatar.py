"""A plain, slow statement of the Kibatar forward pass: one whole sequence at a time, no cache, no batch,
one function per mechanism, torch on the CPU only (float64 unless told otherwise).  It shares no code with
`reinfer_b200`; the tests compare the engine with it.

Notation.  x is the residual stream [T, width]; `lin(x, W) = x W^T` with W stored [out, in];
rms(v) = v / sqrt(mean(v^2) + eps).  A layer is a sandwich with a vector of scales behind each output norm:

    x += ls1 * rms(mixer(rms(x) w1)) w1b;      x += ls2 * rms(ff(rms(x) w2)) w2b        (ff may be missing)

Embedding: x0 = scale * embed[token] + bigram[row], the row picked by the token and the one before it.
Layers `loop.start .. loop.stop - 1` run `loop.times` times in a row with the same weights (each pass is
a layer of its own as far as memories go), and every pass begins with x <- W_in [x; x0].

* `wkv`               a matrix memory per head with a decay per key channel, read before it is written, the
                      present token entering with a bonus of its own; inputs mixed with the token before
* `latent_attention`  keys and values rebuilt per head from one normalised latent per token plus one rotated
                      key part shared by the heads; a sink in the softmax; an elementwise output gate

Feed-forward: experts with clamped gates, weighted by their softmax scores, and one shared expert.
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
    out = {}
    for name, e in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        lo, hi = e["data_offsets"]
        buf = raw[8 + n + lo:8 + n + hi]
        if e["dtype"] == "BF16":
            a = (np.frombuffer(buf, dtype="<u2").astype(np.uint32) << 16).view(np.float32)
        else:
            a = np.frombuffer(buf, dtype={"F32": "<f4", "I32": "<i4"}[e["dtype"]])
        t = torch.from_numpy(a.copy()).reshape(e["shape"])
        out[name] = t.double() if t.is_floating_point() else t.long()
    return out


def read_model(model_dir: str):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


# ---------------------------------------------------------------- small pieces
ROUND = None        # a function on tensors: what every product (but the router's) reads and puts out goes through it first


def lin(x: torch.Tensor, w: torch.Tensor, exact: bool = False) -> torch.Tensor:
    if ROUND is None or exact:
        return x @ w.t()
    return ROUND(ROUND(x) @ w.t())


def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(dim=-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------- embedding
def bigram_row(prev: Optional[int], token: int, mul_prev: int, mul_cur: int, buckets: int) -> int:
    return buckets if prev is None else (prev * mul_prev + token * mul_cur) % buckets


def embed(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    b = cfg["embedding"].get("bigram")
    if b:
        rows = [bigram_row(tokens[i - 1] if i else None, t, b["mul_prev"], b["mul_cur"], b["buckets"]) for i, t in enumerate(tokens)]
        x = x + w["bigram"][torch.tensor(rows)]
    return x


# ---------------------------------------------------------------- rotation
def stretched_frequencies(dims: int, base: float, scaling: Optional[dict]):
    """([f_i], factor on cosine and sine), f_i = base^(-2i/dims); with `scaling` the slow ones are divided by the factor, by a ramp
    over the pairs' indices between those that turn `fast` and `slow` times within `original` positions."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0

    def index(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index(scaling["fast"])), 0)
    hi = min(math.ceil(index(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * r + fi * (1.0 - r))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_half_split(x: torch.Tensor, positions: torch.Tensor, freqs: List[float], mag: float) -> torch.Tensor:
    """x [T, ..., d]: dimension i of the first 2 n turns together with dimension i + n, n = len(freqs)."""
    n = len(freqs)
    ang = positions.to(x.dtype)[:, None] * torch.tensor(freqs, dtype=x.dtype)[None, :]
    while ang.dim() < x.dim():
        ang = ang.unsqueeze(1)
    c, s = torch.cos(ang) * mag, torch.sin(ang) * mag
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


# ---------------------------------------------------------------- mixers
def softmax_with_sink(scores: torch.Tensor, sink: float) -> torch.Tensor:
    """scores [T, T] (masked with -inf): exp(s) / (sum exp(s) + exp(sink))."""
    m = torch.clamp(scores.max(dim=-1, keepdim=True).values, min=sink)
    e = torch.exp(scores - m)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(torch.as_tensor(sink, dtype=scores.dtype) - m))


def latent_attention(h: torch.Tensor, m: dict, eps: float, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    T = h.shape[0]
    H, dn, dr, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    freqs, mag = stretched_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    pos = torch.arange(T)
    q = lin(rms(lin(h, w[p + "dq"]), eps) * w[p + "dq.norm"], w[p + "uq"]).view(T, H, dn + dr)
    down = lin(h, w[p + "dkv"])
    c = rms(down[:, :rank], eps) * w[p + "dkv.norm"]
    kr = rotate_half_split(down[:, rank:], pos, freqs, mag)
    qr = rotate_half_split(q[..., dn:], pos, freqs, mag)
    k, v = lin(c, w[p + "uk"]).view(T, H, dn), lin(c, w[p + "uv"]).view(T, H, dv)
    unseen = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    heads = []
    for i in range(H):
        s = (q[:, i, :dn] @ k[:, i].t() + qr[:, i] @ kr.t()) * m["scale"]
        heads.append(softmax_with_sink(s.masked_fill(unseen, -math.inf), float(w[p + "sink"][i])) @ v[:, i])
    return lin(torch.cat(heads, dim=-1) * torch.sigmoid(lin(h, w[p + "g"])), w[p + "o"])


def wkv_scan(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, u: torch.Tensor) -> torch.Tensor:
    """All [T, H, d] (u [H, d]): o_t = (S + diag(u) k v^T)^T r, then S <- diag(decay) S + k v^T, from S = 0."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=r.dtype)
    out = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(((S + u[:, :, None] * kv) * r[t][:, :, None]).sum(dim=1))
        S = decay[t][:, :, None] * S + kv
    return torch.stack(out)


def wkv(h: torch.Tensor, m: dict, eps: float, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    T, H, d = h.shape[0], m["heads"], m["dim"]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])

    def mixed(s):
        return h + (before - h) * w[p + "mu." + s]

    r, k, v = (lin(mixed(s), w[p + s]).view(T, H, d) for s in ("r", "k", "v"))
    gate = silu(lin(mixed("g"), w[p + "g"]))
    decay = torch.exp(-torch.exp(lin(torch.tanh(lin(mixed("w"), w[p + "w1"])), w[p + "w2"]) + w[p + "w0"])).view(T, H, d)
    o = rms(wkv_scan(r, k, v, decay, w[p + "u"].view(H, d)), eps).reshape(T, H * d)
    return lin(o * w[p + "norm"] * gate, w[p + "o"])


MIXERS = {"latent_attention": latent_attention, "wkv": wkv}


# ---------------------------------------------------------------- feed-forward
def clamped_expert(h: torch.Tensor, limit: float, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    g = torch.clamp(lin(h, w[p + "gate"]), max=limit)
    u = torch.clamp(lin(h, w[p + "up"]), min=-limit, max=limit)
    return lin(g * torch.sigmoid(1.702 * g) * (u + 1.0), w[p + "down"])


def route(h: torch.Tensor, r: dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    """Weights [T, experts], zero where an expert was not chosen."""
    s = torch.softmax(lin(h, w[p + "router"], exact=True), dim=-1)
    chosen = torch.topk(s + w[p + "correction"], r["top"], dim=-1).indices
    return torch.zeros_like(s).scatter(1, chosen, torch.gather(s, 1, chosen)) * r["scale"]


def mixture(h: torch.Tensor, mlp: dict, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    g = route(h, mlp["router"], w, p)
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        y = y + g[:, e:e + 1] * clamped_expert(h, mlp["expert"]["limit"], w, f"{p}e{e}.")
    if mlp.get("shared"):
        y = y + torch.sigmoid(lin(h, w[p + "shared.sg"])) * clamped_expert(h, mlp["shared"]["limit"], w, p + "shared.")
    return y


# ---------------------------------------------------------------- the whole
def layer(x: torch.Tensor, l: dict, eps: float, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    y = MIXERS[l["type"]](rms(x, eps) * w[p + "norm1"], l["mixer"], eps, w, p + "mix.")
    x = x + rms(y, eps) * w[p + "norm1b"] * w[p + "ls1"]
    if l.get("mlp") is not None:
        y = mixture(rms(x, eps) * w[p + "norm2"], l["mlp"], w, p + "mlp.")
        x = x + rms(y, eps) * w[p + "norm2b"] * w[p + "ls2"]
    return x


def run_order(cfg: dict):
    """(layer, whether a pass of the loop begins with it) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64, trace: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab]; `trace` gets the stream after every layer run."""
    w = {k: t.to(dtype) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x0 = x = embed(cfg, w, tokens)
    for i, begins in run_order(cfg):
        if begins:
            x = lin(torch.cat([x, x0], dim=-1), w["loop.in"])
        x = layer(x, cfg["layers"][i], eps, w, f"l{i}.")
        if trace is not None:
            trace.append(x.clone())
    return lin(rms(x, eps) * w["final.norm"], w["head"]) * cfg["logit_scale"]


def rounded_forward(cfg: dict, w: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    """The same with every product's input and output rounded to bfloat16: how far the logits move by rounding alone."""
    global ROUND
    ROUND = lambda t: t.to(torch.bfloat16).to(t.dtype)
    try:
        return forward(cfg, w, tokens)
    finally:
        ROUND = None


def greedy(cfg: dict, w: Dict[str, torch.Tensor], prompt: List[int], n: int) -> List[int]:
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
