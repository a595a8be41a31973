"""Razevik on the host: the configuration's parsing and its errors, the model description's tensor names and cache needs, the
plain implementation's small pieces, and that the tests' weights let a fault show."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_razevik as plain
import razevik_tiny as rt
from reinfer_b200.config.errors import InvalidValue, MissingKey
from reinfer_b200.config.razevik import RazevikConfig
from reinfer_b200.config.registry import resolve_architecture
from reinfer_b200.models.razevik import build_spec
from reinfer_b200.parts.model import Model, expected_params


@pytest.mark.parametrize("cfg", [rt.TINY_A, rt.TINY_B, rt.TINY_C, rt.TINY_D] + [rt.random_config(s) for s in range(8)])
def test_round_trip_and_registry(cfg):
    arch = resolve_architecture(cfg)
    assert arch.name == "Razevik" and arch.config_cls is RazevikConfig
    c = RazevikConfig.from_dict(cfg)
    assert RazevikConfig.from_dict(c.to_dict()) == c
    assert c.vocab_size == cfg["vocab"] and c.hidden_size == cfg["width"]
    assert set(rt.make_weights(cfg, 0)) == set(expected_params(build_spec(c)))


@pytest.mark.parametrize("edit,error", [
    (lambda d: d.pop("vocab"), MissingKey),
    (lambda d: d.pop("residual_mult"), MissingKey),
    (lambda d: d.pop("max_positions"), MissingKey),
    (lambda d: d["norm"].pop("eps"), MissingKey),
    (lambda d: d.__setitem__("logit_softcap", 0), InvalidValue),
    (lambda d: d["token_side"].__setitem__("dim", 0), InvalidValue),
    (lambda d: d["layers"][0].__setitem__("type", "attention"), InvalidValue),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), MissingKey),
    (lambda d: d["layers"][0]["mixer"].__setitem__("kv_from", 0), InvalidValue),            # itself
    (lambda d: d["layers"][1]["mixer"].__setitem__("kv_from", 3), InvalidValue),            # a later layer
    (lambda d: d["layers"][4]["mixer"].__setitem__("kv_from", 1), InvalidValue),            # a layer without a latent of its own
    (lambda d: d["layers"][4]["mixer"].__setitem__("kv_from", 0), InvalidValue),            # another kv_rank
    (lambda d: d["layers"][1]["mlp"]["router"].__setitem__("top", 7), InvalidValue),        # of 2 groups of 3
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].__setitem__("count", 5), InvalidValue),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].__setitem__("keep", 5), InvalidValue),
    (lambda d: d["layers"][3]["mlp"]["router"].__setitem__("top", 5), InvalidValue),
    (lambda d: d["layers"][1]["mlp"].__setitem__("kind", "sparse"), InvalidValue),
    (lambda d: d["layers"][1]["mlp"]["shared"].pop("ff"), MissingKey),
    (lambda d: d["layers"][1]["mlp"].pop("expert"), MissingKey),
])
def test_errors_say_what_is_wrong(edit, error):
    d = copy.deepcopy(rt.TINY_A)
    edit(d)
    with pytest.raises(error):
        RazevikConfig.from_dict(d)


def test_tensor_names_and_shapes():
    ps = {n: tuple(p.shape) for n, p in expected_params(build_spec(RazevikConfig.from_dict(rt.TINY_A))).items()}
    assert ps["embed"] == (211, 64) and ps["pos"] == (320, 64) and ps["head"] == (211, 64) and ps["final.norm"] == (64,)
    assert ps["side.embed"] == (211, 5 * 12) and ps["l3.side.gate"] == (12, 64) and ps["l3.side.proj"] == (64, 12) and ps["l3.side.norm"] == (64,)
    assert ps["l0.mix.dq"] == (24, 64) and ps["l0.mix.dq.norm"] == (24,) and ps["l0.mix.uq"] == (4 * 16, 24)
    assert ps["l0.mix.dkv"] == (40, 64) and ps["l0.mix.dkv.norm"] == (40,) and ps["l0.mix.g"] == (4, 64) and ps["l0.mix.o"] == (64, 4 * 24)
    assert "l1.mix.dkv" not in ps and "l1.mix.dkv.norm" not in ps and ps["l1.mix.uk"] == (6 * 8, 40) and ps["l1.mix.uv"] == (6 * 12, 40)
    assert ps["l0.mlp.up"] == (72, 64) and ps["l0.mlp.down"] == (64, 72)
    assert ps["l1.mlp.router"] == (12, 64) and ps["l1.mlp.correction"] == (12,) and ps["l1.mlp.e11.up"] == (24, 64)
    assert ps["l1.mlp.shared.up"] == (40, 64) and ps["l1.mlp.shared.down"] == (64, 40) and ps["l1.mlp.shared.sg"] == (1, 64)
    assert ps["l0.norm1"] == ps["l0.norm2"] == (64,) and "l2.norm2" not in ps and not any(n.startswith("l2.mlp") for n in ps)
    assert "l2.norm2" in build_spec(RazevikConfig.from_dict(rt.TINY_A)).ignorable_tensors
    ps = expected_params(build_spec(RazevikConfig.from_dict(rt.TINY_B)))
    assert not any(".shared." in n for n in ps if n.startswith("l0."))


def test_who_caches_and_who_reads():
    m = Model(build_spec(RazevikConfig.from_dict(rt.TINY_A)))
    paged, states = m.cache_layout()
    assert set(paged) == {"l0", "l2"} and not states
    assert (paged["l0"].kv_heads, paged["l0"].head_dim, paged["l0"].value_dim) == (1, 40, 0) and paged["l2"].head_dim == 24
    assert m.cache_bindings() == [("l0", "l0", True), ("l1", "l0", False), ("l2", "l2", True), ("l3", "l0", False), ("l4", "l2", False)]


def test_plain_route():
    z = torch.tensor([2.0, -1.0, 0.5, 0.0, -3.0, 1.0], dtype=torch.float64)
    none = torch.zeros(6, dtype=torch.float64)
    chosen, wt = plain.route(z, none, 2, None)
    assert chosen == [0, 5] and abs(wt.sum().item() - 1.0) < 1e-12
    s = torch.sigmoid(z)
    assert torch.allclose(wt, s[[0, 5]] / s[[0, 5]].sum())
    # three groups of two, one kept: the pair with the largest sum, although the best single expert sits elsewhere
    chosen, _ = plain.route(torch.tensor([3.0, -9.0, 1.0, 1.2, -1.0, 0.0], dtype=torch.float64), none, 2, {"count": 3, "keep": 1})
    assert sorted(chosen) == [2, 3]
    # scores made negative by the correction: an expert of a dropped group is never taken for its "zero"
    corr = torch.tensor([-5.0, -5.0, -9.0, -9.0, -9.5, -9.5], dtype=torch.float64)
    chosen, wt = plain.route(z, corr, 2, {"count": 3, "keep": 1})
    assert sorted(chosen) == [0, 1] and (wt > 0).all()


def test_plain_activations():
    z = torch.linspace(-4, 4, 41, dtype=torch.float64)
    assert torch.allclose(plain.gelu_erf(z), torch.nn.functional.gelu(z))
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert plain.relu_squared(torch.tensor([-2.0, 3.0])).tolist() == [0.0, 9.0]
    assert torch.allclose(plain.gelu_erf(torch.tensor(0.7, dtype=torch.float64)), torch.tensor(0.7 * 0.5 * (1 + math.erf(0.7 / math.sqrt(2))), dtype=torch.float64))


FAULTS = {
    "group_scores_by_their_best": ("route", lambda z, c, top, g: _route_variant(z, c, top, g, best_one=True)),
    "dropped_experts_count_as_zero": ("route", lambda z, c, top, g: _route_variant(z, c, top, g, dropped=0.0)),
    "weights_with_the_correction": ("route", lambda z, c, top, g: _route_variant(z, c, top, g, corrected=True)),
    "no_weights_normalised": ("route", lambda z, c, top, g: _route_variant(z, c, top, g, normalise=False)),
    "the_other_gelu": ("gelu_erf", plain.relu_squared),
    "no_shared_gate": ("shared_expert", lambda h, w, p: plain.expert(h, w, p)),
    "no_latent_norm": ("latent_of", lambda h, w, p, eps: plain.lin(h, w[p + "dkv"])),
    "first_key_lost": ("softmax_attention", lambda q, k, v, scale: _lossy_attention(q, k, v, scale)),
    "no_side_norm": ("token_side", lambda x, rows, w, p, eps: plain.lin(plain.gelu_tanh(plain.lin(x, w[p + "gate"])) * rows, w[p + "proj"])),
}


def _route_variant(z, corr, top, groups, best_one=False, dropped=float("-inf"), corrected=False, normalise=True):
    E = z.shape[0]
    s = torch.sigmoid(z)
    choice = (s + corr).tolist()
    if groups is not None:
        size = E // groups["count"]
        score = [sum(sorted(choice[g * size:(g + 1) * size], reverse=True)[:1 if best_one else 2]) for g in range(groups["count"])]
        best = sorted(range(groups["count"]), key=lambda g: -score[g])[:groups["keep"]]
        choice = [c if e // size in best else dropped for e, c in enumerate(choice)]
    chosen = sorted(range(E), key=lambda e: -choice[e])[:top]
    wt = (s + corr if corrected else s)[chosen]
    return chosen, wt / (wt.sum() + 1e-20) if normalise else wt


def _lossy_attention(q, k, v, scale):
    T = q.shape[0]
    s = (q @ k.t()) * scale
    i = torch.arange(T)
    s = s.masked_fill((i[None, :] > i[:, None]) | ((i[None, :] == 0) & (i[:, None] > 0)), float("-inf"))
    return torch.softmax(s, dim=-1) @ v


@pytest.mark.parametrize("fault", list(FAULTS))
def test_a_fault_shows_with_these_weights(fault, monkeypatch):
    """A mistake in one mechanism, made in the plain implementation, moves the logits far beyond the engine tests'
    tolerances."""
    cfg = rt.TINY_A
    w = {k: v.double() for k, v in rt.make_weights(cfg, rt.TINY["A"][1]).items()}
    toks = rt.sequences("A")["r2"]
    right = plain.forward(cfg, w, toks)
    name, wrong = FAULTS[fault]
    monkeypatch.setattr(plain, name, wrong)
    err = (plain.forward(cfg, w, toks) - right).abs().amax(dim=1) / right.abs().amax(dim=1)
    assert err.max().item() > 2e-2 and (err > 1e-3).double().mean().item() > 0.3, (err.max().item(), err.median().item())


def test_random_configurations_cover_the_options():
    seen = set()
    for s in range(40):
        for l in rt.random_config(s)["layers"]:
            seen.add("from" if "kv_from" in l["mixer"] else "own")
            m = l["mlp"]
            seen.add("none" if m is None else m["kind"])
            if m and m["kind"] == "moe":
                seen.add("groups" if "groups" in m["router"] else "free")
                seen.add("shared" if "shared" in m else "alone")
    assert {"from", "own", "none", "dense", "moe", "groups", "free", "shared", "alone"} <= seen
