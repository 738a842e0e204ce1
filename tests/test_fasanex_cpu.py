"""Fasanex without a GPU: its configuration class, the registry, the weight slots against the tensors a checkpoint holds and what the layers
ask of the cache, norm weights stored around zero, the frequencies, and the plain implementation against itself."""
import json
import math
import os

import numpy as np
import pytest

import fasanex_util as T
import plain_fasanex as P


def test_config_round_trip_and_registry(tmp_path):
    from kestrel_llm_b200.config import ConfigError, FasanexConfig, load_config
    for name, (raw, _) in T.CONFIGS.items():
        d = tmp_path / name
        os.makedirs(d)
        with open(d / "config.json", "w") as f:
            json.dump(raw, f)
        cfg = load_config(str(d))
        assert isinstance(cfg, FasanexConfig) and cfg.num_hidden_layers == len(raw["layers"])
        assert FasanexConfig.from_dict(cfg.to_json_dict()) == cfg
    c = FasanexConfig.from_dict(T.F1)
    m = c.layers[0].mixer
    assert (m.left.heads, m.left.kv_heads, m.left.dim, m.left.conv, m.left.window, m.left.softcap, m.left.rot.dims) == (6, 2, 24, 3, 21, 8.0, 16)
    assert (m.left.rot.scaling.factor, m.left.rot.scaling.original, m.left.rot.scaling.fast, m.left.rot.scaling.slow) == (4.0, 64.0, 8.0, 0.5)
    assert (m.right.heads, m.right.dim, m.right.decay_rank, m.left_scale, m.right_scale) == (2, 24, 9, 0.7, 1.2)
    assert c.embedding_scale == 3.5 and c.layers[1].mlp is None and c.layers[2].mlp.limit == 1.5
    c2 = FasanexConfig.from_dict(T.F2)
    left = c2.layers[1].mixer.left
    assert c2.embedding_scale == 1.0 and left.rot is None and left.window == 0 and left.softcap == 0.0
    for breaker in (lambda r: r["layers"][0]["mixer"]["left"].update(kv_heads=4),         # 6 heads on 4 kv heads
                    lambda r: r["layers"][0]["mixer"].pop("right"),
                    lambda r: r["layers"][0]["mixer"].pop("left_scale"),
                    lambda r: r["layers"][0]["mixer"]["left"].update(vdim=32),             # the values are the keys
                    lambda r: r["layers"][0]["mixer"]["left"].update(softcap=-1.0),
                    lambda r: r["layers"][0]["mixer"]["left"].update(mask={}),
                    lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=26),      # more than the head
                    lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=7),
                    lambda r: r["layers"][1]["mixer"].update(groups=4),                    # 6 heads in 4 groups
                    lambda r: r["layers"][1]["mixer"].update(norm_groups=5),
                    lambda r: r["layers"][2]["mixer"].update(kv_heads=3),
                    lambda r: r["layers"][2]["mlp"].update(limit=0),
                    lambda r: r["layers"][2]["mlp"].update(kind="moe"),
                    lambda r: r["layers"][0].update(type="mamba"),
                    lambda r: r.pop("norm")):
        bad = json.loads(json.dumps(T.F1))
        breaker(bad)
        with pytest.raises(ConfigError):
            FasanexConfig.from_dict(bad)


def test_the_rank_of_the_decay_comes_from_the_checkpoint():
    from kestrel_llm_b200.config import ConfigError, FasanexConfig
    raw = json.loads(json.dumps(T.F1))
    for L in raw["layers"]:
        if "right" in L["mixer"]:
            L["mixer"]["right"].pop("decay_rank")
    c = FasanexConfig.from_dict(raw)
    assert c.layers[0].mixer.right.decay_rank == 0
    shapes = {n: a.shape for n, a in T.tensors_of(T.F1, 1).items()}
    assert c.with_tensor_shapes(shapes) == FasanexConfig.from_dict(T.F1)
    with pytest.raises(ConfigError):
        c.with_tensor_shapes({})


def test_weight_slots_and_cache_layers():
    import torch
    from kestrel_llm_b200.config import FasanexConfig, resolve_architecture
    from kestrel_llm_b200.parts import CombinedSpec, FixedStateSpec, PagedKVSpec
    for name, (raw, seed) in T.CONFIGS.items():
        W = T.tensors_of(raw, seed)
        model = resolve_architecture("Fasanex").build(FasanexConfig.from_dict(raw), torch.bfloat16, "meta")
        slots = {s.name: s for s in model.weight_slots()}
        assert {n: tuple(s.dest.shape) for n, s in slots.items()} == {n: a.shape for n, a in W.items()}
        assert all((s.add == 1.0) == (n.split(".")[-1].startswith("norm") and ".mix." not in n or n == "final.norm") for n, s in slots.items())
        assert model.graph_safe and model.step_program(None) is None      # decode steps are captured; other steps walk the parts
        assert [(c.block, c.cache) for c in model.order] == [(i, i) for i in range(len(raw["layers"]))]
        for a, b in zip(model.blocks, model.blocks[1:]):
            assert a.following is b.norm1
        for L, block, spec in zip(raw["layers"], model.blocks, model.cache_specs()):
            m = L["mixer"]
            if L["type"] == "parallel":
                a, b = m["left"], m["right"]
                assert isinstance(spec, CombinedSpec)
                assert spec.paged == PagedKVSpec(a["kv_heads"], a["dim"], (a.get("mask") or {}).get("size", 0), 0, a["dim"])
                tail = (a["conv"] - 1) * (a["heads"] + a["kv_heads"]) * a["dim"]
                off, size = block.mixer.right.state_off, spec.state.shape[0]
                assert off % 4 == 0 and off >= tail and size % 4 == 0
                assert size >= off + b["heads"] * b["dim"] ** 2 + raw["width"] and block.mixer.left.state_off == 0
            else:
                assert isinstance(spec, FixedStateSpec) and spec.shape[0] % 4 == 0
                kept = m["heads"] * m["vdim"] * (m["state"] if L["type"] == "mamba2" else m["dim"])
                channels = m["heads"] * m["vdim"] + (2 * m["groups"] * m["state"] if L["type"] == "mamba2" else 2 * m["kv_heads"] * m["dim"])
                assert 0 <= spec.shape[0] - kept - (m["conv"] - 1) * channels < 8


def test_norm_weights_and_filters_as_a_checkpoint_stores_them(tmp_path):
    """What the loader puts in place: 1 + w for the norms of the width, filters laid out by tap."""
    import torch
    from kestrel_llm_b200.weights import load_model
    d = T.write_model(T.F1, T.tensors_of(T.F1, 3), tmp_path)
    model = load_model(d["float32"], "float32", "cpu")
    _, W = P.read_model(d["float32"])
    assert np.allclose(model.blocks[0].norm1.weight.numpy(), 1.0 + W["l0.norm1"], atol=1e-6)
    assert np.allclose(model.final_norm.weight.numpy(), 1.0 + W["final.norm"], atol=1e-6)
    assert np.array_equal(model.blocks[1].mixer.conv_w.numpy(), W["l1.mix.conv"].T.astype(np.float32))
    assert np.array_equal(model.blocks[1].mixer.norm_w.numpy(), W["l1.mix.norm"].astype(np.float32))
    out = model.blocks[0].mixer.out.weight
    assert np.array_equal(out.numpy(), np.concatenate([W["l0.mix.left.o"], W["l0.mix.right.o"]], axis=1).astype(np.float32))
    assert isinstance(out, torch.Tensor)


def test_frequencies_of_a_ramp():
    """The engine's frequencies against the plain ones: below, on and above the ramp; the factor on cosines and sines."""
    import torch
    from kestrel_llm_b200.config import FasanexConfig, resolve_architecture
    for name in ("F1", "F3"):
        raw = T.CONFIGS[name][0]
        model = resolve_architecture("Fasanex").build(FasanexConfig.from_dict(raw), torch.float32, "cpu")
        for L, block in zip(raw["layers"], model.blocks):
            if L["type"] != "parallel":
                continue
            freq, mag = P.rotary_frequencies(L["mixer"]["left"]["rot"])
            rot = block.mixer.left.rotation
            assert rot.dim == L["mixer"]["left"]["rot"]["dims"] and rot.pairing == "half" and abs(rot.scale - mag) < 1e-12
            assert np.array_equal(rot.inv_freq.numpy(), freq.astype(np.float32))
    plain = np.array([100.0 ** (-2.0 * i / 16) for i in range(8)])
    freq, mag = P.rotary_frequencies(T.F1["layers"][0]["mixer"]["left"]["rot"])
    assert freq[0] == plain[0] and abs(freq[-1] - plain[-1] / 4.0) < 1e-15 and abs(mag - (0.1 * math.log(4.0) + 1.0)) < 1e-15
    assert any(p / 4.0 < f < p for f, p in zip(freq, plain))


def test_the_plain_implementation_against_itself():
    """Prefixes of a sequence give the first rows; the window's edge; the recurrences in closed form."""
    cfg, seed = T.CONFIGS["F1"]
    W = {n: a.astype(np.float64) for n, a in T.tensors_of(cfg, seed).items()}
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], size=40).tolist()
    whole = P.forward(cfg, W, toks)
    assert np.allclose(P.forward(cfg, W, toks[:23]), whole[:23], atol=1e-10)
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((30, 2, 8)), rng.standard_normal((30, 1, 8)), rng.standard_normal((30, 1, 8))
    a = P.window_attention(q, k, v, 0.5, 3.0, 7)
    k2, v2 = k.copy(), v.copy()
    k2[:13], v2[:13] = 9.0, 9.0
    b = P.window_attention(q, k2, v2, 0.5, 3.0, 7)
    assert np.allclose(a[19:], b[19:]) and not np.allclose(a[18], b[18])          # token 19 sees 13 .. 19, token 18 sees 12
    # a state space without decay, with equal steps, is a causal sum
    x, B, C = rng.standard_normal((12, 1, 3)), rng.standard_normal((12, 1, 4)), rng.standard_normal((12, 1, 4))
    y = P.state_space(x, B, C, np.full((12, 1), 0.5), np.array([-80.0]), np.array([2.0]))
    want = np.stack([sum(0.5 * (C[t, 0] @ B[j, 0]) * x[j, 0] for j in range(t + 1)) + 2.0 * x[t, 0] for t in range(12)])
    assert np.allclose(y[:, 0], want)
    # time mixing: the read-out sees the old state and the bonus, not the new write
    r, kk, vv = (rng.standard_normal((6, 1, 5)) for _ in range(3))
    w, u = np.full((6, 1, 5), 0.5), rng.standard_normal((1, 5))
    o = P.bonus_recurrence(r, kk, vv, w, u)
    t = 4
    want = sum((r[t, 0] * 0.5 ** (t - 1 - j)) @ kk[j, 0] * vv[j, 0] for j in range(t)) + (r[t, 0] * u[0]) @ kk[t, 0] * vv[t, 0]
    assert np.allclose(o[t, 0], want)
    # the delta rule with full writes recalls what was last stored along a unit key
    key = P.unit_vectors(rng.standard_normal((1, 1, 6)))
    k6, v6 = np.repeat(key, 3, axis=0), rng.standard_normal((3, 1, 4))
    o = P.delta_rule(k6, k6, v6, np.ones((3, 1)), np.ones((3, 1)))
    assert np.allclose(o[2], v6[2], atol=1e-4)
