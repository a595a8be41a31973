"""Razevik as a ModelSpec.  Token table plus a table of learned position vectors; layers of block `parallel_norms`: mixer and
feed-forward read an RMS norm each of the same stream and are added at once, then the token's own row for this layer
comes in (`token_side`) through an output norm (`rms_out`).  The mixer is `latent_attention` without a rotated part, with
one gate per head and optionally the latent of an earlier layer; feed-forwards are dense with squared relu
(`activated_ffn`), mixtures of gelu experts taken by sigmoid scores from the first-ranked groups, with a shared expert, or
none.  The residual multiplier is a factor on the activations behind which the last products stand.  An output matrix
of its own, logits with a soft cap.  Layer i's tensors start with `l<i>.`.
"""
from __future__ import annotations

from ..config.razevik import RazevikConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec


def _mixer(cfg: RazevikConfig, m, prefix: str) -> PartSpec:
    return PartSpec("latent_attention", {"hidden": cfg.width, "heads": m["heads"], "dim": m["dim"], "rot_dim": 0, "vdim": m["vdim"],
                                         "q_rank": m["q_rank"], "kv_rank": m["kv_rank"], "scale": m["scale"], "eps": cfg.norm_eps,
                                         "gate": "heads", "own_kv": m["kv_from"] is None, "out_scale": cfg.residual_mult}, prefix)


def _ffn(cfg: RazevikConfig, mlp, prefix: str) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("activated_ffn", {"hidden": cfg.width, "intermediate": mlp["ff"], "activation": "relu2",
                                          "names": ("up", "down"), "out_scale": cfg.residual_mult}, prefix)
    shared = None
    if mlp["shared"] is not None:
        shared = {"inner": mlp["shared"], "names": ("shared.up", "shared.down"), "gate_name": "shared.sg"}
    return PartSpec("expert_mixture", {"hidden": cfg.width, "experts": mlp["experts"], "top": mlp["top"], "inner": mlp["ff"],
                                       "activation": "gelu", "route": "group_sigmoid", "groups": mlp["groups"], "shared": shared,
                                       "out_scale": cfg.residual_mult}, prefix)


def build_spec(cfg: RazevikConfig) -> ModelSpec:
    h, n = cfg.width, len(cfg.layers)

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"width": h, "eps": cfg.norm_eps, "weight_name": ""}, name)

    layers, ignorable = [], []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        roles = dict(mixer_norm=norm(p + "norm1"), mixer=_mixer(cfg, l.mixer, p + "mix."))
        if l.mlp is not None:
            roles.update(ffn_norm=norm(p + "norm2"), ffn=_ffn(cfg, l.mlp, p + "mlp."))
        else:
            ignorable.append(p + "norm2")                      # a norm nobody reads
        if cfg.side_dim is not None:
            roles.update(side_ffn=PartSpec("token_side", {"hidden": h, "dim": cfg.side_dim, "vocab": cfg.vocab, "index": i, "count": n,
                                                          "table_name": "side.embed", "names": (p + "side.gate", p + "side.proj")}, ""),
                         side_norm=PartSpec("rms_out", {"width": h, "eps": cfg.norm_eps, "mult": cfg.residual_mult,
                                                        "weight_name": ""}, p + "side.norm"))
        src = l.mixer["kv_from"]
        layers.append(LayerSpec(f"l{i}", block="parallel_norms", cache_from=None if src is None else f"l{src}", **roles))
    return ModelSpec(
        hidden_size=h, vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", {"vocab": cfg.vocab, "hidden": h, "positions": cfg.max_positions, "table_name": "embed",
                                         "positions_name": "pos"}, ""),
        layers=tuple(layers),
        final_norm=norm("final.norm"),
        lm_head=PartSpec("linear", {"vocab": cfg.vocab, "hidden": h, "weight_name": "", "softcap": cfg.logit_softcap or 0.0}, "head"),
        ignorable_tensors=tuple(ignorable))


def register() -> None:
    register_architecture("Razevik", RazevikConfig, build_spec, aliases=("razevik",))
