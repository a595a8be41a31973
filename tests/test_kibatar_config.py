"""Kibatar on the host: the configuration's parsing and its errors, the model description's tensor names, run order and cache
needs, the plain implementation's small pieces, and that the tests' weights let a fault show."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import kibatar_tiny as kt
import plain_kibatar as plain
from reinfer_b200.config.errors import InvalidValue, MissingKey
from reinfer_b200.config.kibatar import KibatarConfig
from reinfer_b200.config.registry import load_config, resolve_architecture
from reinfer_b200.models.kibatar import build_spec
from reinfer_b200.parts.model import Model, expected_params


@pytest.mark.parametrize("cfg", [kt.TINY_A, kt.TINY_B, kt.TINY_C, kt.TINY_D] + [kt.random_config(s) for s in range(8)])
def test_round_trip_and_registry(cfg):
    arch = resolve_architecture(cfg)
    assert arch.name == "Kibatar" and arch.config_cls is KibatarConfig
    c = KibatarConfig.from_dict(cfg)
    assert KibatarConfig.from_dict(c.to_dict()) == c
    assert c.vocab_size == cfg["vocab"] and c.hidden_size == cfg["width"]
    assert set(kt.make_weights(cfg, 0)) == set(expected_params(build_spec(c)))


def test_the_decays_rank_is_read_off_its_tensor(tmp_path):
    d = kt.make_model_dir(str(tmp_path / "m"), "A")
    _, c = load_config(d)
    assert c == KibatarConfig.from_dict(kt.TINY_A) and c.layers[0].mixer["decay_rank"] == 6 and c.layers[2].mixer["decay_rank"] == 5
    bare = copy.deepcopy(kt.TINY_A)
    bare["layers"][0]["mixer"].pop("decay_rank")
    with pytest.raises(MissingKey):
        KibatarConfig.from_dict(bare)


@pytest.mark.parametrize("edit,error", [
    (lambda d: d.pop("vocab"), MissingKey),
    (lambda d: d.pop("logit_scale"), MissingKey),
    (lambda d: d["embedding"].pop("scale"), MissingKey),
    (lambda d: d["embedding"]["bigram"].pop("buckets"), MissingKey),
    (lambda d: d["embedding"]["bigram"].__setitem__("mul_cur", -1), InvalidValue),
    (lambda d: d["norm"].pop("eps"), MissingKey),
    (lambda d: d["loop"].__setitem__("stop", 5), InvalidValue),
    (lambda d: d["loop"].__setitem__("start", 3), InvalidValue),
    (lambda d: d["loop"].__setitem__("times", 0), InvalidValue),
    (lambda d: d["layers"][0].__setitem__("type", "attention"), InvalidValue),
    (lambda d: d["layers"][1]["mixer"].pop("scale"), MissingKey),
    (lambda d: d["layers"][1]["mixer"].pop("rot"), MissingKey),
    (lambda d: d["layers"][1]["mixer"]["rot"].__setitem__("dims", 10), InvalidValue),
    (lambda d: d["layers"][3]["mixer"]["rot"]["scaling"].pop("fast"), MissingKey),
    (lambda d: d["layers"][3]["mixer"]["rot"]["scaling"].__setitem__("factor", 0), InvalidValue),
    (lambda d: d["layers"][0]["mixer"].__setitem__("heads", 0), InvalidValue),
    (lambda d: d["layers"][0]["mlp"]["router"].__setitem__("top", 7), InvalidValue),
    (lambda d: d["layers"][0]["mlp"]["router"].pop("scale"), MissingKey),
    (lambda d: d["layers"][0]["mlp"]["expert"].__setitem__("limit", 0.0), InvalidValue),
    (lambda d: d["layers"][0]["mlp"]["shared"].pop("limit"), MissingKey),
    (lambda d: d["layers"][0]["mlp"].__setitem__("kind", "dense"), InvalidValue),
])
def test_errors_say_what_is_wrong(edit, error):
    d = copy.deepcopy(kt.TINY_A)
    edit(d)
    with pytest.raises(error):
        KibatarConfig.from_dict(d)


def test_tensor_names_and_shapes():
    spec = build_spec(KibatarConfig.from_dict(kt.TINY_A))
    ps = {n: tuple(p.shape) for n, p in expected_params(spec).items()}
    assert ps["embed"] == (211, 64) and ps["bigram"] == (84, 64) and ps["loop.in"] == (64, 128) and ps["head"] == (211, 64) and ps["final.norm"] == (64,)
    assert all(ps["l0.mix." + s] == (48, 64) for s in "rkvg") and all(ps["l0.mix.mu." + s] == (64,) for s in "rkvgw")
    assert ps["l0.mix.w1"] == (6, 64) and ps["l0.mix.w2"] == (48, 6) and ps["l0.mix.w0"] == (48,) and ps["l0.mix.u"] == (3, 16)
    assert ps["l0.mix.norm"] == (48,) and ps["l0.mix.o"] == (64, 48)
    assert ps["l1.mix.dq"] == (24, 64) and ps["l1.mix.uq"] == (4 * 24, 24) and ps["l1.mix.dkv"] == (48, 64) and ps["l1.mix.uk"] == (64, 40)
    assert ps["l1.mix.uv"] == (96, 40) and ps["l1.mix.sink"] == (4,) and ps["l1.mix.g"] == (96, 64) and ps["l1.mix.o"] == (64, 96)
    assert ps["l0.mlp.e5.gate"] == (24, 64) and ps["l0.mlp.e5.down"] == (64, 24) and ps["l0.mlp.router"] == (6, 64) and ps["l0.mlp.correction"] == (6,)
    assert ps["l0.mlp.shared.gate"] == (40, 64) and ps["l0.mlp.shared.sg"] == (1, 64)
    assert all(ps["l0." + n] == (64,) for n in ("norm1", "norm1b", "norm2", "norm2b", "ls1", "ls2"))
    assert not any(n.startswith("l2.mlp") or n in ("l2.norm2", "l2.norm2b", "l2.ls2") for n in ps)
    assert {"l2.norm2", "l2.norm2b", "l2.ls2"} <= set(spec.ignorable_tensors)
    assert not any(".shared." in n for n in ps if n.startswith("l3."))
    bare = {k: v for k, v in kt.TINY_A.items() if k != "loop"}
    bare["embedding"] = {"scale": 2.0}
    ps = expected_params(build_spec(KibatarConfig.from_dict(bare)))
    assert "bigram" not in ps and "loop.in" not in ps


def test_run_order_and_what_is_kept():
    m = Model(build_spec(KibatarConfig.from_dict(kt.TINY_A)))
    assert [k for _, k in m.run] == ["l0", "loop", "l1", "l2", "loop#1", "l1#1", "l2#1", "l3"]
    paged, states = m.cache_layout()
    assert {k: (v.kv_heads, v.head_dim, v.value_dim, v.window) for k, v in paged.items()} == \
        {"l1": (1, 48, 0, None), "l1#1": (1, 48, 0, None), "l3": (1, 36, 0, None)}
    assert set(states) == {"embedding", "l0", "l2", "l2#1"}
    assert states["embedding"].shape == (1,) and states["embedding"].dtype == "int32"
    assert states["l2"]["S"].shape == (2, 24, 24) and states["l2"]["S"].dtype == "float32" and states["l2"]["last"].shape == (64,)
    assert ("embedding", None, False) in m.cache_bindings()


# ---------------------------------------------------------------- the plain implementation's pieces
def test_plain_bigram_rows():
    assert plain.bigram_row(None, 5, 7, 3, 10) == 10 and plain.bigram_row(0, 5, 7, 3, 10) == 5 and plain.bigram_row(4, 5, 7, 3, 10) == 3
    cfg = {"embedding": {"scale": 2.0, "bigram": {"buckets": 3, "mul_prev": 1, "mul_cur": 2}}}
    w = {"embed": torch.eye(3), "bigram": torch.arange(4.0)[:, None].expand(4, 3) * 10}
    x = plain.embed(cfg, w, [1, 2, 0])
    assert x.tolist() == [[30.0, 32.0, 30.0], [20.0, 20.0, 22.0], [22.0, 20.0, 20.0]]        # rows 3, (1 + 4) % 3, (2 + 0) % 3


def test_plain_rotation_keeps_lengths_and_pairs_halves():
    x = torch.randn(5, 2, 10, dtype=torch.float64)
    f, mag = plain.stretched_frequencies(8, 100.0, None)
    assert mag == 1.0 and len(f) == 4
    y = plain.rotate_half_split(x, torch.arange(5), f, 1.0)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 8:], x[..., 8:])
    for i in range(4):
        assert torch.allclose(y[..., i] ** 2 + y[..., i + 4] ** 2, x[..., i] ** 2 + x[..., i + 4] ** 2)
    f2, mag2 = plain.stretched_frequencies(8, 100.0, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
    assert abs(mag2 - (0.1 * math.log(4.0) + 1.0)) < 1e-12 and f2[0] == f[0] and abs(f2[3] - f[3] / 4.0) < 1e-12


def test_plain_wkv_by_hand():
    """One head of size one: o_t = r_t (S + u k_t v_t), S <- w S + k v."""
    one = lambda *v: torch.tensor(v, dtype=torch.float64).view(-1, 1, 1)
    o = plain.wkv_scan(one(1, 2, 3), one(1, 1, 2), one(5, 7, 1), one(0.5, 0.25, 0.1), torch.tensor([[10.0]], dtype=torch.float64))
    assert o.flatten().tolist() == [50.0, 2 * (5 + 70), 3 * (0.25 * 5 + 7 + 20)]


def test_plain_sink_and_expert():
    s = torch.tensor([[0.0, -math.inf], [1.0, 2.0]], dtype=torch.float64)
    p = plain.softmax_with_sink(s, 0.5)
    assert torch.allclose(p[0], torch.tensor([1.0 / (1.0 + math.exp(0.5)), 0.0], dtype=torch.float64))
    assert abs(p[1].sum().item() - (math.e + math.e ** 2) / (math.e + math.e ** 2 + math.exp(0.5))) < 1e-12
    w = {"gate": torch.tensor([[1.0]]), "up": torch.tensor([[-1.0]]), "down": torch.tensor([[1.0]])}
    y = plain.clamped_expert(torch.tensor([[5.0], [-5.0], [0.5]]), 2.0, w, "")
    want = [2 / (1 + math.exp(-3.404)) * -1.0, -5 / (1 + math.exp(8.51)) * 3.0, 0.5 / (1 + math.exp(-0.851)) * 0.5]
    assert torch.allclose(y.flatten(), torch.tensor(want), atol=1e-6)


def test_plain_route():
    w = {"router": torch.eye(4, dtype=torch.float64), "correction": torch.tensor([0.0, 0.0, 1.0, 0.0], dtype=torch.float64)}
    z = torch.tensor([[2.0, 1.0, -3.0, 0.0]], dtype=torch.float64)
    g = plain.route(z, {"top": 2, "scale": 3.0}, w, "")
    s = torch.softmax(z, -1)
    assert torch.allclose(g, torch.tensor([[3 * s[0, 0], 0.0, 3 * s[0, 2], 0.0]], dtype=torch.float64))


# ---------------------------------------------------------------- faults planted in the plain implementation
def _attention_fault(**change):
    right = plain.latent_attention

    def wrong(h, m, eps, w, p):
        if change.get("no_sink"):
            w = {**w, p + "sink": torch.full_like(w[p + "sink"], -1e4)}
        if change.get("no_gate"):
            w = {**w, p + "g": torch.zeros_like(w[p + "g"])}
        return right(h, m, eps, w, p)
    return wrong


def _wkv_fault(**change):
    right = plain.wkv

    def wrong(h, m, eps, w, p):
        if change.get("no_shift"):
            w = {**w, **{p + "mu." + s: torch.zeros_like(w[p + "mu." + s]) for s in "rkvgw"}}
        if change.get("no_bonus"):
            w = {**w, p + "u": torch.zeros_like(w[p + "u"])}
        if change.get("no_decay"):
            w = {**w, p + "w0": torch.full_like(w[p + "w0"], -50.0)}
        return right(h, m, eps, w, p)
    return wrong


def _mixture_fault(edit):
    right = plain.mixture
    return lambda h, mlp, w, p: right(h, edit(copy.deepcopy(mlp)), w, p)


def _layer_fault(drop):
    right = plain.layer
    return lambda x, l, eps, w, p: right(x, l, eps, {k: (torch.ones_like(t) if k.endswith(drop) else t) for k, t in w.items()}, p)


FAULTS = {
    "previous_token_forgotten": ("bigram_row", lambda prev, tok, mp, mc, b: b if prev is None else tok * mc % b),
    "first_token_as_any": ("bigram_row", lambda prev, tok, mp, mc, b: ((prev or 0) * mp + tok * mc) % b),
    "no_sink": ("MIXERS", {"latent_attention": _attention_fault(no_sink=True), "wkv": plain.wkv}),
    "no_output_gate": ("MIXERS", {"latent_attention": _attention_fault(no_gate=True), "wkv": plain.wkv}),
    "no_rotation": ("rotate_half_split", lambda x, pos, f, mag: x),
    "no_stretching": ("stretched_frequencies", lambda dims, base, sc: ([base ** (-2.0 * i / dims) for i in range(dims // 2)], 1.0)),
    "no_token_shift": ("MIXERS", {"latent_attention": plain.latent_attention, "wkv": _wkv_fault(no_shift=True)}),
    "no_bonus": ("MIXERS", {"latent_attention": plain.latent_attention, "wkv": _wkv_fault(no_bonus=True)}),
    "no_decay": ("MIXERS", {"latent_attention": plain.latent_attention, "wkv": _wkv_fault(no_decay=True)}),
    "no_limits": ("mixture", _mixture_fault(lambda m: {**m, "expert": {**m["expert"], "limit": 1e9}})),
    "one_limit_for_all": ("mixture", _mixture_fault(lambda m: {**m, "shared": m.get("shared") and {**m["shared"], "limit": m["expert"]["limit"]}})),
    "no_shared_expert": ("mixture", _mixture_fault(lambda m: {**m, "shared": None})),
    "no_weight_scale": ("mixture", _mixture_fault(lambda m: {**m, "router": {**m["router"], "scale": 1.0}})),
    "no_correction": ("layer", lambda x, l, eps, w, p, right=plain.layer: right(x, l, eps, {k: t * 0 if k.endswith("correction") else t for k, t in w.items()}, p)),
    "no_layer_scale": ("layer", _layer_fault(("ls1", "ls2"))),
    "no_map_before_a_pass": ("run_order", lambda cfg, right=plain.run_order: [(i, False) for i, _ in right(cfg)]),
    "map_once_only": ("run_order", lambda cfg, right=plain.run_order: [(i, b and not any(x for _, x in right(cfg)[:n])) for n, (i, b) in enumerate(right(cfg))]),
}


@pytest.mark.parametrize("fault", list(FAULTS))
def test_a_fault_shows_with_these_weights(fault, monkeypatch):
    """A mistake in one mechanism, made in the plain implementation, moves the logits far beyond the engine tests'
    tolerances."""
    cfg = kt.TINY_A
    w = {k: v.double() for k, v in kt.make_weights(cfg, kt.TINY["A"][1]).items()}
    toks = kt.sequences("A")["r2"]
    right = plain.forward(cfg, w, toks)
    name, wrong = FAULTS[fault]
    monkeypatch.setattr(plain, name, wrong)
    err = (plain.forward(cfg, w, toks) - right).abs().amax(dim=1) / right.abs().amax(dim=1)
    assert err.max().item() > 2e-2 and (err > 1e-3).double().mean().item() > 0.3, (err.max().item(), err.median().item())


def test_random_configurations_cover_the_options():
    seen = set()
    for s in range(40):
        c = kt.random_config(s)
        seen |= {"loop" if "loop" in c else "straight", "pairs" if "bigram" in c["embedding"] else "single"}
        for l in c["layers"]:
            seen.add(l["type"])
            if l["type"] == "latent_attention":
                seen.add("stretched" if "scaling" in l["mixer"]["rot"] else "as it is")
            m = l["mlp"]
            seen.add("none" if m is None else "shared" if "shared" in m else "alone")
    assert seen == {"loop", "straight", "pairs", "single", "wkv", "latent_attention", "stretched", "as it is", "none", "shared", "alone"}
