"""Tuganex without a GPU: the configuration, the model's weight slots against the tests' own list of tensor names, which
layer writes and which reads a cache layer, and the plain statement against itself."""
import copy

import numpy as np
import pytest

import plain_tuganex as P
import tuganex_util as U


def _config(cfg):
    from kestrel_llm_b200.config import resolve_architecture
    arch = resolve_architecture("Tuganex")
    return arch, arch.config_class.from_dict(cfg)


@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_configuration_round_trip_and_weight_slots(name):
    import torch
    cfg, seed = U.CONFIGS[name]
    arch, c = _config(cfg)
    assert arch.config_class.from_dict(c.to_json_dict()) == c
    model = arch.build(c, torch.bfloat16, "meta")
    slots = {s.name: tuple(s.dest.shape) for s in model.weight_slots()}
    assert slots == {n: a.shape for n, a in U.tensors_of(cfg, seed).items()}
    assert set(model.optional_tensors) == {f"l{i}.norm2" for i, L in enumerate(cfg["layers"]) if L["mlp"] is None}
    # a layer on another's keys uses that layer's cache and does not write it; all others have a memory of their own
    for i, (call, L) in enumerate(zip(model.order, cfg["layers"])):
        j = L["mixer"].get("kv_from")
        assert call.block == i and call.writes_cache == (j is None)
        assert call.cache == model.order[i if j is None else j].cache
    assert len(model.cache_specs()) == sum(L["mixer"].get("kv_from") is None for L in cfg["layers"])
    assert model.graph_safe


def test_absent_keys_mean_none():
    cfg = copy.deepcopy(U.T1)
    for key in ("groups", "identity"):
        del cfg["layers"][0]["mlp"]["router"][key]
    del cfg["layers"][0]["mlp"]["shared"]
    del cfg["layers"][1]["mixer"]["rot"]
    _, c = _config(cfg)
    f = c.layers[0].mlp
    assert (f.identity, f.groups, f.keep, f.shared_ff) == (0, 1, 1, 0) and c.layers[1].mixer.rot is None


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "window"), (("layers", 0, "mixer", "kv_heads"), 4), (("layers", 2, "mixer", "kv_from"), 1),
    (("layers", 2, "mixer", "kv_from"), 3), (("layers", 2, "mixer", "dim"), 32), (("layers", 1, "mixer", "decay"), [0.5]),
    (("layers", 1, "mixer", "decay"), [0.5, 0.5, 1.5]), (("layers", 0, "mixer", "rot"), {"dims": 15, "base": 10.0}),
    (("layers", 0, "mixer", "rot"), {"dims": 26, "base": 10.0}), (("layers", 0, "mlp", "router", "identity"), 2),
    (("layers", 0, "mlp", "router", "groups"), {"count": 3, "keep": 4}), (("layers", 0, "mlp", "kind"), "sparse"), (("norm",), {"eps": 0})])
def test_configuration_refuses(path, value):
    from kestrel_llm_b200.config.model_config import ConfigError
    cfg = copy.deepcopy(U.T1)
    at = cfg
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        _config(cfg)


@pytest.mark.parametrize("name", list(U.CONFIGS))
def test_plain_statement_is_causal(name):
    cfg, seed = U.CONFIGS[name]
    W = U.bf16_round(U.tensors_of(cfg, seed))
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], size=40).tolist()
    whole = P.forward(toks, W, cfg)
    assert np.abs(whole[:23] - P.forward(toks[:23], W, cfg)).max() < 1e-9


def test_plain_retention_is_its_sum_over_keys():
    """The recurrence unrolled: o_t = sum over j <= t of decay^(t - j) (q_t . k_j) v_j."""
    rng = np.random.default_rng(1)
    T, H, d, dv = 30, 2, 5, 3
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((T, H, d)), rng.standard_normal((T, H, dv))
    decay = np.array([0.8, 1.0])
    t = np.arange(T)
    far = t[:, None] - t[None, :]
    for h in range(H):
        m = np.where(far >= 0, decay[h] ** np.maximum(far, 0), 0.0)
        want = (q[:, h] @ k[:, h].T * m) @ v[:, h]
        assert np.abs(P.retention_scan(q, k, v, decay)[:, h] - want).max() < 1e-12


def test_plain_xielu_meets_at_zero_and_differs_on_its_sides():
    z = np.array([-1e-9, 0.0, 1e-9])
    assert np.abs(P.xielu(z, 0.3, -0.2) - 0.5 * z).max() < 1e-15
    assert np.isclose(P.xielu(np.array([2.0]), 0.3, -0.2)[0], np.log1p(np.exp(0.3)) * 4 + 1)
    assert np.isclose(P.xielu(np.array([-2.0]), 0.3, -0.2)[0], (0.5 + np.log1p(np.exp(-0.2))) * (np.exp(-2) + 1) - 1)


def test_plain_router_closes_groups_and_weighs_without_the_correction():
    rng = np.random.default_rng(2)
    h = rng.standard_normal((50, 12))
    W = {"router": rng.standard_normal((8, 12)), "correction": np.array([0, 0, -5, -5, -2, -2, -9, -9.0])}
    ids, ws = P.route(h, W, "", {"experts": 6, "identity": 2, "top": 3, "groups": {"count": 4, "keep": 2}})
    assert set(np.unique(ids)) == {0, 1, 4, 5}           # the groups of outputs 0, 1 and 4, 5: negative choice scores, still the best left
    s = P.softmax_rows(h @ W["router"].T)
    assert np.allclose(ws, np.take_along_axis(s, ids, axis=1)) and ws.sum(axis=1).max() < 1
