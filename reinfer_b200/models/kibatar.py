"""Kibatar as a ModelSpec.  The embedding adds a row for the pair of neighbouring tokens; layers are sandwiches (block
`sandwich`): an RMS norm before every sublayer and a second one on what the sublayer puts out (`rms_out`, which carries the
layer's scale per channel).  Per layer one of two mixers - `latent_attention` (half-split rotation with stretched slow
frequencies, a sink, an elementwise gate) or `wkv` (token shift, a matrix state read before it is written) - and a mixture of
clamped gated experts taken by softmax scores with a shared expert, or no feed-forward.  A stretch of layers may run several
times with the same weights; before every pass a block `stream_map` joins stream and embedding (`stream_recall`), and every run
has a cache of its own (the run order repeats the layers' indices).  An output matrix of its own; the scale on the logits is
folded into the last norm's weight.  Layer i's tensors start with `l<i>.`.
"""
from __future__ import annotations

from ..config.kibatar import KibatarConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec


def _mixer(cfg: KibatarConfig, kind: str, m, prefix: str) -> PartSpec:
    if kind == "wkv":
        return PartSpec("wkv", {"hidden": cfg.width, "heads": m["heads"], "dim": m["dim"], "decay_rank": m["decay_rank"],
                                "eps": cfg.norm_eps}, prefix)
    rot = m["rot"]
    return PartSpec("latent_attention", {"hidden": cfg.width, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"],
                                         "vdim": m["vdim"], "q_rank": m["q_rank"], "kv_rank": m["kv_rank"], "scale": m["scale"],
                                         "eps": cfg.norm_eps, "gate": True, "sink": True,
                                         "position": {"kind": "rope_pairs", "dims": rot["dims"], "base": rot["base"],
                                                      "scaling": rot["scaling"], "pairing": "half"}}, prefix)


def _ffn(cfg: KibatarConfig, mlp, prefix: str) -> PartSpec:
    shared = None
    if mlp["shared"] is not None:
        shared = {"inner": mlp["shared"]["ff"], "limit": mlp["shared"]["limit"], "gate_name": "shared.sg",
                  "names": ("shared.gate", "shared.up", "shared.down")}
    r = mlp["router"]
    return PartSpec("expert_mixture", {"hidden": cfg.width, "experts": r["experts"], "top": r["top"], "weight_scale": r["scale"],
                                       "inner": mlp["expert"]["ff"], "limit": mlp["expert"]["limit"], "gated": True,
                                       "expert_names": ("e{}.gate", "e{}.up", "e{}.down"), "activation": "clamp_swish",
                                       "route": "scores", "shared": shared}, prefix)


def build_spec(cfg: KibatarConfig) -> ModelSpec:
    h, n = cfg.width, len(cfg.layers)

    def norm(name: str, gain: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"width": h, "eps": cfg.norm_eps, "weight_name": "", "gain": gain}, name)

    def out_norm(prefix: str, name: str, scale: str) -> PartSpec:
        return PartSpec("rms_out", {"width": h, "eps": cfg.norm_eps, "weight_name": name, "scale_name": scale}, prefix)

    layers, ignorable = [], []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        roles = dict(mixer_norm=norm(p + "norm1"), mixer=_mixer(cfg, l.type, l.mixer, p + "mix."), mixer_out_norm=out_norm(p, "norm1b", "ls1"))
        if l.mlp is not None:
            roles.update(ffn_norm=norm(p + "norm2"), ffn=_ffn(cfg, l.mlp, p + "mlp."), ffn_out_norm=out_norm(p, "norm2b", "ls2"))
        else:
            ignorable += [p + "norm2", p + "norm2b", p + "ls2"]         # tensors nobody reads
        layers.append(LayerSpec(f"l{i}", block="sandwich", **roles))
    order = tuple(range(n))
    if cfg.loop is not None:
        a, b, times = cfg.loop
        layers.append(LayerSpec("loop", block="stream_map", map_ffn=PartSpec("stream_recall", {"hidden": h, "weight_name": ""}, "loop.in")))
        order = tuple(range(a)) + ((n,) + tuple(range(a, b))) * times + tuple(range(b, n))
    pairs = None
    if cfg.bigram is not None:
        pairs = {"buckets": cfg.bigram[0], "mul_prev": cfg.bigram[1], "mul_cur": cfg.bigram[2], "table_name": "bigram"}
    return ModelSpec(
        hidden_size=h, vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", {"vocab": cfg.vocab, "hidden": h, "table_name": "embed", "scale": cfg.embedding_scale,
                                         "pairs": pairs, "keep_output": cfg.loop is not None}, ""),
        layers=tuple(layers),
        final_norm=norm("final.norm", gain=cfg.logit_scale),
        lm_head=PartSpec("linear", {"vocab": cfg.vocab, "hidden": h, "weight_name": ""}, "head"),
        order=order, ignorable_tensors=tuple(ignorable))


def register() -> None:
    register_architecture("Kibatar", KibatarConfig, build_spec, aliases=("kibatar",))
