"""The Tuganex decoder in the engine against its plain statement (`plain_tuganex`): every mechanism alone, then whole
models under every way of cutting and batching the work, then generation through the scheduler (GPU)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import plain_tuganex as P
import replay_util as R
import tuganex_util as U

pytestmark = pytest.mark.gpu

DTYPES = ("float32", "bfloat16")
PART_TOL = {"float32": 3e-5, "bfloat16": 4e-2}      # of the largest entry of the plain result
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def udirs(tmp_path_factory):
    return {name: U.write_model(cfg, U.tensors_of(cfg, seed), tmp_path_factory.mktemp("tuganex_" + name)) for name, (cfg, seed) in U.CONFIGS.items()}


def _close(got, want, dtype, what, scale=None, tol=None):
    scale = float(np.abs(want).max()) if scale is None else scale
    assert np.isfinite(got).all(), f"{what}: not finite"
    err = float(np.abs(got - want).max()) / scale
    allowed = PART_TOL[dtype] if tol is None else tol
    assert err <= allowed, f"{what}: error {err:.3e} of the largest entry, allowed {allowed:.1e}"
    return err


def _torch_dtype(dtype):
    import torch
    return {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]


def _exact(h):
    """Rows that both number formats hold exactly, so that the parts' inputs are the same."""
    import torch
    return torch.from_numpy(np.asarray(h, dtype=np.float32)).to(torch.bfloat16).to(torch.float64).numpy()


def _model_of(layers, width, dtype, eps=1e-6, seed=0, vocab=11):
    from kestrel_llm_b200.config import resolve_architecture
    cfg = {"architecture": "Tuganex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}
    W = U.tensors_of(cfg, seed)
    arch = resolve_architecture("Tuganex")
    return arch.build(arch.config_class.from_dict(cfg), _torch_dtype(dtype), "cuda:0"), W, cfg


def _plain_mixer(layer, h, W, eps=1e-6, p="l0.mix."):
    m = layer["mixer"]
    if layer["type"] == "retention":
        return P.mix_retention(h, W, p, m, eps)
    return P.mix_attention(h, W, p, m, eps, P.keys_values(h, W, p, m, eps))


def _mixer_case(layer, dtype, page, n_tokens, cuts, seed=0, width=48, prepare=None, eps=1e-6):
    """One mixer alone; ``cuts`` are the portion sizes the tokens arrive in.  ``prepare(W, h)`` may shape weights and inputs
    and return other inputs whose plain result is handed back as well.  Returns (engine, plain, plain of the other inputs
    or the harness)."""
    rng = np.random.default_rng(seed)
    model, W, _ = _model_of([U.layer(layer, None)], width, dtype, eps=eps, seed=seed)
    mixer = model.blocks[0].mixer
    h = _exact(rng.standard_normal((n_tokens, width)))
    other = None
    if prepare is not None:
        other = prepare(W, h)
        h = _exact(h)
    assert U.load_part(mixer, W) == {k for k in W if k.startswith("l0.mix.")}
    Wr = U.bf16_round(W)
    want = _plain_mixer(layer, h, Wr, eps)
    hs = U.PartHarness(mixer, dtype, max_tokens=((n_tokens + 63) // 64) * 64 + 64, page_size=page)
    got, at = [], 0
    for n in cuts:
        got.append(hs.step([(7, h[at:at + n])])[0])
        at += n
    assert at == n_tokens
    if other is not None:
        return np.concatenate(got), want, _plain_mixer(layer, _exact(other), Wr, eps)
    return np.concatenate(got), want, hs


# one entry per mechanism and shape of sizes
MIXERS = [
    ("attention 6/2 x 24/40, 16 of 24 turned", U.attn(6, 2, 24, 40, 0.21, 0.3, (16, 100.0))),
    ("attention 3/3 x 16/16, no rotation", U.attn(3, 3, 16, 16, 0.3, 0.8)),
    ("attention 5/1 x 10/14 (no multiples of 8)", U.attn(5, 1, 10, 14, 0.4, 0.2, (6, 20.0))),
    ("attention 4/2 x 64/128", U.attn(4, 2, 64, 128, 0.125, 0.35, (64, 10000.0))),
    ("attention 2/1 x 128/64", U.attn(2, 1, 128, 64, 0.1, 0.6, (32, 10000.0))),
    ("attention 6/2 x 32/64, all turned", U.attn(6, 2, 32, 64, 0.19, 0.45, (32, 10000.0))),
    ("attention 8/1 x 8/24", U.attn(8, 1, 8, 24, 0.5, 0.1, (8, 10.0))),
    ("attention 2/1 x 144/32 (maps beyond the tensor-core kernels' sizes)", U.attn(2, 1, 144, 32, 0.08, 0.5, (144, 1000.0))),
    ("retention 3 x 40/24, 16 of 40 turned", U.retention(3, 40, 24, (0.75, 0.99, 1.0), (16, 50.0))),
    ("retention 2 x 14/10 (no multiples of 8), no rotation", U.retention(2, 14, 10, (0.0, 0.97))),
    ("retention 2 x 128/128", U.retention(2, 128, 128, (0.984375, 0.998), (128, 10000.0))),
    ("retention 4 x 32/72", U.retention(4, 32, 72, (0.875, 0.96875, 0.9921875, 0.998046875), (32, 500.0))),
    ("retention 1 x 200/16", U.retention(1, 200, 16, (0.95,), (64, 500.0))),
    ("retention 2 x 64/256", U.retention(2, 64, 256, (0.95, 0.999), (64, 500.0))),
]


# ---- each mechanism alone --------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("label,layer", MIXERS, ids=[m[0] for m in MIXERS])
def test_mixer_alone_whole_and_cut(dtype, label, layer):
    n = 90
    whole, want, _ = _mixer_case(layer, dtype, 16, n, [n], seed=len(label))
    _close(whole, want, dtype, f"{label}, whole")
    cut, want, _ = _mixer_case(layer, dtype, 8, n, [33, 2, 17, 2, 7, 8, 9, 6] + [1] * 6, seed=len(label))
    _close(cut, want, dtype, f"{label}, portions and single tokens")
    single, want, _ = _mixer_case(layer, dtype, 16, 21, [1] * 21, seed=len(label))
    _close(single, want, dtype, f"{label}, token by token from the first")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[700], [1, 299, 400], [64, 65, 63, 508], [520, 2, 178], [900, 400]])
@pytest.mark.parametrize("which", [3, 10, 11, 8])
def test_mixers_in_long_portions(which, dtype, cuts):
    """Portions long enough for the kernels of many tokens: the tcgen05 attention (also over key ranges in slices) and the
    recurrence in chunks, whose first chunk starts from the state an earlier portion left and whose last is cut short."""
    label, layer = MIXERS[which]
    got, want, _ = _mixer_case(layer, dtype, 16, sum(cuts), cuts, seed=which)
    _close(got, want, dtype, f"{label}, portions {cuts}", tol=1e-4 if dtype == "float32" else None)


def _spike(layer, map_, i, j):
    """Weights and inputs so that token i asks for token j above all others (beside itself) in one map.  Keys are made from the
    first half of a token's input and values from the second, that map's queries by the keys' own weights, and token i gets
    the first half of token j's input - so its q_i . k_j is a squared length while the two tokens' values differ.  The
    recurrence does not forget: token j's input is made large.  Returns inputs in which another token stands in j's place."""
    m = layer["mixer"]

    def prepare(W, h):
        p, half = "l0.mix.", h.shape[1] // 2
        if layer["type"] == "retention":
            other = h.copy()
            h[j] *= 6.0
            return other
        H, G, d = m["heads"], m["kv_heads"], m["dim"]
        W[p + "k"][:, half:] = 0.0
        W[p + "v"][:, :half] = 0.0
        for n in range(H):
            at = (n * 2 + map_) * d
            g = (n // (H // G) * 2 + map_) * d
            W[p + "q"][at:at + d] = W[p + "k"][g:g + d]
        W[p + "q.norm"][:] = W[p + "k.norm"]
        for name, x in (("lq1", 0.6), ("lk1", 1.0), ("lq2", 0.0), ("lk2", 1.0)):
            W[p + name][:] = x / np.sqrt(d)          # lambda = exp(0.6) - 1 + diff: both maps weigh
        h[i, :half] = h[j, :half]
        other = h.copy()
        other[j] = np.random.default_rng(5).standard_normal(h.shape[1])
        return other
    return prepare


SPIKES = {"first map": (U.attn(4, 2, 24, 40, 0.5, 0.4), 0), "second map": (U.attn(4, 2, 24, 40, 0.5, 0.4), 1),
          "second map of 64": (U.attn(4, 2, 64, 128, 0.25, 0.4), 1), "first map of 64": (U.attn(4, 2, 64, 128, 0.25, 0.4), 0),
          "retention": (U.retention(2, 32, 24, (1.0, 1.0), (4, 1e6)), 0), "retention of 128": (U.retention(2, 128, 128, (1.0, 0.9998), (4, 1e6)), 0)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("where", ["far", "page_end", "page_start", "first_token", "previous_token"])
@pytest.mark.parametrize("kind", list(SPIKES))
def test_mixer_reads_what_lies_far_back(kind, dtype, decode, where):
    """One token stands out and one later token asks for it: hundreds of tokens back, on either side of a page border, at
    the request's first position, and right before.  The plain result with an ordinary token in its place differs widely:
    the engine must match the true one, in a prompt's portions and decoded token by token."""
    page, n, i = 16, 300, 297
    j = {"far": 3, "page_end": 255, "page_start": 256, "first_token": 0, "previous_token": i - 1}[where]
    layer, map_ = SPIKES[kind]
    cuts = [290] + [1] * 10 if decode else [140, 160]
    got, want, other = _mixer_case(layer, dtype, page, n, cuts, prepare=_spike(layer, map_, i, j), width=160)
    scale, told = float(np.abs(want).max()), float(np.abs(want[i] - other[i]).max())
    assert told > 0.1 * np.abs(want[i]).max(), f"{kind}, {where}: the case does not tell whether token {j} was read"
    err = float(np.abs(got - want).max()) / scale
    assert np.isfinite(got).all() and err <= {"float32": 1e-4, "bfloat16": 4e-2}[dtype], f"{kind}, {where}: error {err:.3e}"
    assert np.abs(got[i] - want[i]).max() < 0.2 * told


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [U.attn(2, 1, 16, 24, 0.3, 0.2), U.attn(2, 1, 64, 128, 0.12, 0.9)], ids=["16/24", "64/128"])
def test_the_second_map_is_subtracted_with_the_layers_own_weight(dtype, layer):
    """lambda from its four vectors: with other vectors, or another `diff`, the plain result is another; the engine follows."""
    results = []
    for lq1, lq2 in ((0.0, 0.0), (1.2, 0.0), (0.0, 1.2)):
        def prepare(W, h):
            d = W["l0.mix.lq1"].shape[0]
            for n, x in (("lq1", lq1), ("lk1", 1.0), ("lq2", lq2), ("lk2", 1.0)):
                W["l0.mix." + n][:] = x / np.sqrt(d)
            return h.copy()
        got, want, _ = _mixer_case(layer, dtype, 16, 150, [130] + [1] * 20, prepare=prepare)
        _close(got, want, dtype, f"lambda from {lq1}, {lq2}")
        results.append(want)
    for a in range(3):
        for b in range(a):
            assert np.abs(results[a] - results[b]).max() > 0.05 * np.abs(results[a]).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("src,reader", [(U.attn(6, 2, 24, 40, 0.21, 0.3, (16, 100.0)), U.attn(4, 2, 24, 40, 0.35, 0.55, (16, 100.0), kv_from=0)),
                                        (U.attn(4, 2, 64, 128, 0.125, 0.35, (64, 1e4)), U.attn(2, 2, 64, 128, 0.2, 0.7, (64, 1e4), kv_from=0)),
                                        (U.attn(5, 1, 10, 14, 0.4, 0.2, (6, 20.0)), U.attn(2, 1, 10, 14, 0.6, 0.45, (6, 20.0), kv_from=0))])
def test_a_layer_on_anothers_keys(dtype, src, reader):
    """The reader has queries, lambda, scale and head count of its own; its keys and values are the pages an earlier layer of
    the same step wrote - from another input than its own."""
    model, W, _ = _model_of([U.layer(src, None), U.layer(reader, None)], 48, dtype, seed=4)
    a, b = model.blocks[0].mixer, model.blocks[1].mixer
    U.load_part(a, W)
    U.load_part(b, W)
    Wr = U.bf16_round(W)
    rng = np.random.default_rng(4)
    ha, hb = (_exact(rng.standard_normal((90, 48))) for _ in range(2))
    kv = P.keys_values(ha, Wr, "l0.mix.", src["mixer"], 1e-6)
    want = P.mix_attention(hb, Wr, "l1.mix.", reader["mixer"], 1e-6, kv)
    hs = U.PartHarness(a, dtype, max_tokens=128, page_size=16)
    got, at = [], 0
    for n in [50, 2, 30] + [1] * 8:
        hs.step([(7, ha[at:at + n])], commit=False)
        got.append(hs.step([(7, hb[at:at + n])], writable=False, mixer=b)[0])
        hs.commit()
        at += n
    _close(np.concatenate(got), want, dtype, "reader")


@pytest.mark.parametrize("dtype", DTYPES)
def test_positions_turn_queries_and_keys_far_out(dtype):
    """Rotation alone tells the tokens apart: all keys of a layer are one vector before they are turned, hundreds of positions
    with fast and slow pairs; and a recurrence whose q and k are one vector each."""
    for layer in (U.attn(2, 1, 16, 24, 0.9, 0.3, (16, 300.0)), U.retention(2, 16, 24, (1.0, 0.99), (12, 300.0))):
        def prepare(W, h):
            h[:, 0] = 1.0
            W["l0.mix.q"][:, 1:] = 0.0
            W["l0.mix.k"][:, 1:] = 0.0
            return h.copy()
        got, want, _ = _mixer_case(layer, dtype, 16, 500, [333, 147] + [1] * 20, prepare=prepare)
        _close(got, want, dtype, layer["type"], tol={"float32": 2e-4, "bfloat16": 4e-2}[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
def test_retention_in_chunks_of_unequal_requests(dtype):
    """Three requests in one step, 400, 129 and 2 tokens: the grid is sized by the longest, the others' chunks end early."""
    for layer in (MIXERS[8][1], MIXERS[10][1]):
        rng = np.random.default_rng(3)
        model, W, _ = _model_of([U.layer(layer, None)], 48, dtype, seed=3)
        mixer = model.blocks[0].mixer
        U.load_part(mixer, W)
        Wr = U.bf16_round(W)
        hs_ = [_exact(rng.standard_normal((n, 48))) for n in (430, 140, 5)]
        want = [P.mix_retention(h, Wr, "l0.mix.", layer["mixer"], 1e-6) for h in hs_]
        hs = U.PartHarness(mixer, dtype, max_tokens=640, page_size=16, slots=3)
        o1 = hs.step([(1, hs_[0][:400]), (2, hs_[1][:129]), (3, hs_[2][:2])])
        o2 = hs.step([(3, hs_[2][2:5]), (1, hs_[0][400:430]), (2, hs_[1][129:140])])
        for r, (a, b) in enumerate(((o1[0], o2[1]), (o1[1], o2[2]), (o1[2], o2[0]))):
            _close(np.concatenate([a, b]), want[r], dtype, f"request {r}", tol=1e-4 if dtype == "float32" else None)


@pytest.mark.parametrize("which", [8, 10, 11, 12, 13])
def test_retention_forms_against_each_other(which):
    """One kernel for few tokens, chunks, and the sequential scan: the same portions through each form that takes them."""
    from kestrel_llm_b200.parts import RetentionMixer
    label, layer = MIXERS[which]
    for dtype, cuts in (("bfloat16", [100, 1, 2, 200, 64, 4, 129]), ("float32", [3, 1, 2, 4, 30, 1, 1])):
        both, want, _ = _mixer_case(layer, dtype, 16, sum(cuts), cuts, seed=which)
        RetentionMixer.chunked = RetentionMixer.one_kernel = False
        try:
            scan, _, _ = _mixer_case(layer, dtype, 16, sum(cuts), cuts, seed=which)
        finally:
            RetentionMixer.chunked = RetentionMixer.one_kernel = True
        scale = float(np.abs(want).max())
        _close(both, scan, dtype, f"{label}, forms", scale=scale, tol={"float32": 1e-5, "bfloat16": 2e-2}[dtype])


@pytest.mark.parametrize("cuts", [[130, 1, 1, 70], [33, 20, 500, 2, 90]])
@pytest.mark.parametrize("which", [0, 3, 4, 5])
def test_attention_kernels_against_their_plain_twin(which, cuts):
    """bfloat16: the tcgen05 kernel, the mma.sync kernel's two tilings and its shares of the keys against the plain kernel."""
    from kestrel_llm_b200.csrc import ops
    from kestrel_llm_b200.parts import DifferentialAttention
    label, layer = MIXERS[which]
    runs = {}
    for name, plain, tc, splits in (("default", False, True, True), ("mma", False, False, True), ("one share", False, False, False), ("plain", True, True, True)):
        DifferentialAttention.force_plain, DifferentialAttention.tcgen05, DifferentialAttention.decode = plain, tc, tc
        ops.attention_window_set_splits(splits)
        try:
            runs[name], want, _ = _mixer_case(layer, "bfloat16", 16, sum(cuts), cuts, seed=which)
        finally:
            DifferentialAttention.force_plain, DifferentialAttention.tcgen05, DifferentialAttention.decode = False, True, True
            ops.attention_window_set_splits(True)
    for name in ("default", "mma", "one share"):
        _close(runs[name], runs["plain"], "bfloat16", f"{label}, {name}", scale=float(np.abs(want).max()), tol=2e-2)


def _ffn_case(mlp, dtype, n, seed=0, width=48, prepare=None, h_scale=1.0):
    import torch
    model, W, _ = _model_of([U.layer(U.retention(1, 8, 8, (0.5,)), mlp)], width, dtype, seed=seed)
    ffn = model.blocks[0].ffn
    if prepare is not None:
        prepare(W)
    assert U.load_part(ffn, W) == {k for k in W if k.startswith("l0.mlp.")}
    Wr = U.bf16_round(W)
    h = _exact(np.random.default_rng(seed).standard_normal((n, width)) * h_scale)
    x = torch.from_numpy(h.astype(np.float32)).to("cuda:0").to(_torch_dtype(dtype))
    got = ffn.forward(x, None).reduce(torch.float32).cpu().numpy().astype(np.float64)
    return got, h, Wr


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 9, 300, 700])
@pytest.mark.parametrize("width,ff", [(48, 96), (70, 30), (128, 512)])
def test_dense_feed_forward_alone(dtype, n, width, ff):
    """Both signs of the activation, small and large arguments, biases on both products; few tokens (slices) and many (the
    activation in the product's epilogue)."""
    for p, q in ((0.4, -0.9), (-3.0, 4.0)):
        def prepare(W):
            W["l0.mlp.act"][:] = (p, q)
        got, h, Wr = _ffn_case(U.dense(ff), dtype, n, seed=n, width=width, prepare=prepare, h_scale=1.5)
        want = P.ff_dense(h, Wr, "l0.mlp.")
        _close(got, want, dtype, f"dense {width} x {ff}, {n} tokens")


MOES = [("9 experts and 3 identity in 3 groups, 2 kept, 3 chosen, shared", U.moe(9, 3, 3, 40, 3, 2, 56)),
        ("10 and 2 in 4 groups, 3 kept, 4 chosen", U.moe(10, 2, 4, 24, 4, 3, 0)),
        ("6 groups of one, 3 kept, 2 chosen", U.moe(6, 0, 2, 22, 6, 3, 18)),
        ("more identity than experts, one group", U.moe(2, 4, 2, 12, 1, 1, 0)),
        ("16 in 4 groups, all kept, 1 chosen", U.moe(16, 0, 1, 48, 4, 4, 32)),
        ("one group of 40 and 8, 8 chosen", U.moe(40, 8, 8, 16, 1, 1, 24)),
        ("all outputs of one expert and one identity", U.moe(1, 1, 2, 8, 1, 1, 8))]


@pytest.mark.parametrize("n", [1, 5, 700])
@pytest.mark.parametrize("label,mlp", MOES, ids=[m[0] for m in MOES])
def test_routed_experts_alone(label, mlp, n):
    """float32, so that the engine's router and the plain one make the same calls."""
    got, h, Wr = _ffn_case(mlp, "float32", n, seed=len(label))
    _close(got, P.ff_moe(h, Wr, "l0.mlp.", mlp), "float32", label)


@pytest.mark.parametrize("n", [9, 1500])
def test_routed_experts_in_bfloat16_where_no_call_is_close(n):
    """bfloat16 on the tensor cores (few pairs: mma.sync; many: tcgen05).  Corrections far apart decide the groups and the
    outputs whatever the rounding; the scores still weigh.  One of the chosen is an identity expert."""
    mlp = U.moe(9, 3, 3, 40, 3, 2, 56)

    def prepare(W):
        W["l0.mlp.correction"][:] = np.array([5, 1, 3, 0, 2, 9, 4, 8, 6, 7, 11, 10], dtype=np.float32) * 3.0
    got, h, Wr = _ffn_case(mlp, "bfloat16", n, prepare=prepare)
    ids, _ = P.route(h, Wr, "l0.mlp.", mlp["router"])
    assert set(np.unique(ids)) == {5, 10, 11}
    _close(got, P.ff_moe(h, Wr, "l0.mlp.", mlp), "bfloat16", "experts in bfloat16")
    mlp = U.moe(10, 2, 3, 40, 3, 2, 0)
    got, h, Wr = _ffn_case(mlp, "bfloat16", n, prepare=prepare)
    _close(got, P.ff_moe(h, Wr, "l0.mlp.", mlp), "bfloat16", "experts and one identity in bfloat16")


def test_correction_chooses_but_does_not_weigh():
    """Negative choice scores: closed outputs are never chosen although the open ones' scores lie below zero (closing counts
    as minus infinity, not as zero); a group's score is its largest choice score, not the sum of two."""
    mlp = U.moe(6, 2, 2, 24, 4, 1, 0)

    def prepare(W):
        W["l0.mlp.correction"][:] = np.array([-6, -30, -9, -9.5, -8, -8.2, -20, -40], dtype=np.float32)
    got, h, Wr = _ffn_case(mlp, "float32", 64, prepare=prepare)
    ids, ws = P.route(h, Wr, "l0.mlp.", mlp["router"])
    assert set(np.unique(ids)) == {0, 1} and (ws.sum(-1) < 1).all()
    _close(got, P.ff_moe(h, Wr, "l0.mlp.", mlp), "float32", "negative choice scores")


@pytest.mark.parametrize("chosen", ["identity", "experts"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_identity_experts_alone_and_none_of_them(dtype, chosen):
    """Every token takes identity experts only (no expert has a row), or experts only."""
    mlp = U.moe(4, 2, 2, 16, 1, 1, 8)

    def prepare(W):
        W["l0.mlp.correction"][:] = np.array([0, 0, 5, 6, 0, 0] if chosen == "experts" else [0, 0, 0, 0, 5, 6], dtype=np.float32)
    for n in (1, 40, 800):
        got, h, Wr = _ffn_case(mlp, dtype, n, prepare=prepare)
        _close(got, P.ff_moe(h, Wr, "l0.mlp.", mlp), dtype, chosen)


@pytest.mark.parametrize("dtype", DTYPES)
def test_block_norms_each_sublayers_result(dtype):
    """Layers as the model runs them: the sublayers read the stream itself, their results are normed and added; a layer
    without feed-forward in the middle hands the stream's copy on."""
    import torch
    from kestrel_llm_b200.cache import CacheManager
    from kestrel_llm_b200.csrc import ops
    from kestrel_llm_b200.engine import Entry
    from kestrel_llm_b200.engine.batch import StepBatch
    layers = [U.layer(U.retention(2, 16, 24, (0.5, 0.9), (8, 100.0)), U.dense(40)), U.layer(U.attn(2, 1, 16, 8, 0.3, 0.3), None),
              U.layer(U.retention(1, 8, 8, (0.7,)), U.moe(6, 2, 2, 16, 4, 2, 24))]
    model, W, cfg = _model_of(layers, 48, dtype, vocab=37)
    for s in model.weight_slots():
        with torch.no_grad():
            s.dest.copy_(torch.from_numpy(W[s.name]).to(torch.bfloat16).to(s.dest.dtype))
    Wr = U.bf16_round(W)
    toks = np.random.default_rng(2).integers(0, 37, size=40).tolist()
    want = []
    P.forward(toks, Wr, cfg, want)
    cache = CacheManager(model.cache_specs(), model.dtype, "cuda:0", 16, 8, 2, 1 << 12)
    cache.admit(0)
    cache.reserve(0, len(toks))
    cache.clear_admitted()
    batch = StepBatch([Entry(0, toks, [])], cache, "cuda:0")
    x, pending = model.forward_embed(batch)
    assert np.abs(x.cpu().numpy() - Wr["embed"][toks]).max() == 0
    for i in range(3):
        x, pending = model.forward_calls(x, pending, batch, cache, i, i + 1)
        assert isinstance(pending, ops.StreamCopy) and torch.equal(pending.data, x.to(model.dtype))
        if dtype == "float32" or i < 2:         # bfloat16 may route a token otherwise than the plain statement
            _close(x.cpu().numpy(), want[i], dtype, f"stream after layer {i}")


# ---- requests beside each other, memory used again --------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", [0, 2, 3, 4, 5, 8, 9, 10, 13])
def test_requests_beside_each_other_and_memory_used_again(dtype, which):
    """Three requests of unequal length in one step, portions beside single tokens, against each alone; then two are given
    back and a new request runs on their pages and slot."""
    label, layer = MIXERS[which]
    rng = np.random.default_rng(which)
    model, W, _ = _model_of([U.layer(layer, None)], 48, dtype, seed=which)
    mixer = model.blocks[0].mixer
    U.load_part(mixer, W)
    Wr = U.bf16_round(W)
    ha, hb, hc, hd = (_exact(rng.standard_normal((n, 48))) for n in (170, 33, 5, 64))
    wa, wb, wc, wd = (_plain_mixer(layer, h, Wr) for h in (ha, hb, hc, hd))
    hs = U.PartHarness(mixer, dtype, max_tokens=256, page_size=8, slots=3)
    o1 = hs.step([(1, ha[:140]), (2, hb[:2]), (3, hc[:1])])
    o2 = hs.step([(2, hb[2:30]), (1, ha[140:141]), (3, hc[1:5])])
    o3 = hs.step([(1, ha[141:170]), (2, hb[30:33])])
    _close(np.concatenate([o1[0], o2[1], o3[0]]), wa, dtype, f"{label}, request a beside others")
    _close(np.concatenate([o1[1], o2[0], o3[1]]), wb, dtype, f"{label}, request b beside others")
    _close(np.concatenate([o1[2], o2[2]]), wc, dtype, f"{label}, request c beside others")
    hs.cache.release(2)
    hs.cache.release(3)
    _close(np.concatenate([hs.step([(4, hd[:50])])[0]] + [hs.step([(4, hd[t:t + 1])])[0] for t in range(50, 64)]), wd, dtype,
           f"{label}, a new request on pages and a slot that were given back")


# ---- whole models ----------------------------------------------------------------------------------

LENGTHS = {"T1": (1, 2, 37, 70, 129, 64), "T2": (3, 50, 97, 130, 17), "T3": (2, 150, 33), "T4": (1, 2, 45, 140, 64)}
LENGTHS_MIXED = {"T1": (5, 33, 70, 129, 47, 90, 16, 65, 31), "T2": (3, 50, 97, 130, 64, 81, 17, 49), "T4": (7, 120, 33, 260, 64, 81, 2, 49)}


def _run(udirs, name, dtype, family, lengths=None, page_size=16, batch_max=4, graphs=False, **kw):
    reqs = U.requests(name, lengths or LENGTHS[name], seed=11 + len(name))
    steps, max_tokens = family(reqs, **kw)
    engine = R.make_engine(udirs[name][dtype], dtype, max_tokens, page_size=page_size, batch_max=batch_max, graphs=graphs)
    got = R.run_trace(engine, steps)
    assert engine.cache.live_requests() == 0
    engine.cache.check()
    U.compare_with_plain(udirs[name]["float32"], reqs, got, dtype, f"{name}/{dtype}/{family.__name__}")
    return got


def test_residual_stream_after_every_layer(udirs):
    """float32: the stream after each layer against the plain implementation's, so that a fault names its place."""
    from kestrel_llm_b200.engine import Entry
    from kestrel_llm_b200.engine.batch import StepBatch
    for name in U.CONFIGS:
        toks = U.requests(name, (75,), seed=4)["r0"]
        cfg, W = U._model(udirs[name]["float32"])
        want = []
        P.forward(toks, W, cfg, want)
        engine = R.make_engine(udirs[name]["float32"], "float32", 128)
        engine.cache.admit(0)
        engine.cache.reserve(0, len(toks))
        engine.cache.clear_admitted()
        batch = StepBatch([Entry(0, toks, [])], engine.cache, "cuda:0")
        model = engine.model
        assert len(model.order) == len(want)
        x, pending = model.forward_embed(batch)
        for i in range(len(model.order)):
            x, pending = model.forward_calls(x, pending, batch, engine.cache, i, i + 1)
            err = np.abs(x.cpu().numpy() - want[i]).max() / np.abs(want[i]).max()
            assert err < 2e-5, f"{name}: layer {i}: error {err:.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["T1", "T2", "T3", "T4"])
@pytest.mark.parametrize("family", [R.trace_whole, R.trace_tail_decode, R.trace_portions])
def test_model_alone_whole_decoded_and_in_portions(udirs, name, dtype, family):
    _run(udirs, name, dtype, family)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("T1", 16), ("T2", 16), ("T4", 8), ("T4", 64)])
def test_model_mixed_batches_pages_and_slots_used_again(udirs, name, dtype, page):
    """Up to four live requests, portions beside single tokens; eight or nine requests through four slots and a pool that
    holds four of them, so that pages and slots are used again."""
    _run(udirs, name, dtype, R.trace_mixed, lengths=LENGTHS_MIXED[name], page_size=page, live_max=4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_with_tensor_core_sizes_mixed_batches(udirs, dtype):
    _run(udirs, "T3", dtype, R.trace_mixed, lengths=(150, 33, 129, 90, 300), live_max=4, sizes=(70, 2, 140, 3, 66, 2, 210, 5))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["T1", "T4"])
def test_long_decoding_through_captured_steps(udirs, name, dtype):
    """Five prompt tokens, then 215 tokens one by one through captured decode steps, through pages that fill one by one."""
    _run(udirs, name, dtype, R.trace_tail_decode, lengths=(220,), graphs=True, tail=215)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_then_decoding(udirs, dtype):
    """600 tokens: a prompt in three portions, then 40 tokens one by one."""
    _run(udirs, "T4", dtype, R.trace_portions, lengths=(600,), sizes=(250, 200, 110) + (1,) * 40)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(udirs, dtype):
    """`LLM.generate`: six requests through three slots, prompts in portions of at most 24 tokens."""
    from kestrel_llm_b200 import LLM, SamplingParams
    name = "T4"
    prompts = list(U.requests(name, (1, 40, 70, 9, 33, 55), seed=4).values())
    llm = LLM(udirs[name][dtype], dtype=dtype, page_size=16, batch_max=3, max_tokens=512, prefill_batch=24, max_step_tokens=64)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True))
    cfg, W = U._model(udirs[name]["float32"])
    for prompt, o in zip(prompts, outs):
        toks = list(prompt)
        assert len(o.token_ids) == 8
        for got in o.token_ids:
            logits = P.forward(toks, W, cfg)[-1]
            want = int(np.argmax(logits))
            if got != want:          # a tie within rounding is not a fault; anything else is
                gap = float(logits[want] - logits[got])
                assert gap <= (2e-5 if dtype == "float32" else 4e-2) * float(np.abs(logits).max()), f"{dtype}: token {got} instead of {want}"
            toks.append(got)


# ---- the programs a user runs ------------------------------------------------------------------------

@pytest.mark.parametrize("dtype,graphs", [("float32", 1), ("bfloat16", 1), ("bfloat16", 0)])
def test_trace_replay_program(udirs, dtype, graphs, tmp_path):
    """bin/trace_run in a process of its own on a mixed trace: four slots for seven requests, decode steps replayed from
    captured graphs (the default) and launched kernel by kernel."""
    name = "T2" if dtype == "float32" else "T4"
    reqs = U.requests(name, (5, 33, 70, 47, 90, 16, 65), seed=21)
    steps, max_tokens = R.trace_mixed(reqs, live_max=4, seed=5)
    lines = "".join(json.dumps(dict(step=i, **s)) + "\n" for i, s in enumerate(steps))
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", udirs[name][dtype], "--dtype", dtype, "--out", str(out),
                        "--max-tokens", str(max_tokens), "--cuda-graphs", str(graphs)], input=lines, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    V = U.CONFIGS[name][0]["vocab"]
    pos = {n: 0 for n in reqs}
    got = {n: {} for n in reqs}
    for i, s in enumerate(steps):
        arr = np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V)
        r = 0
        for e in s["entries"]:
            for w in e["want"]:
                got[e["id"]][pos[e["id"]] + w] = arr[r]
                r += 1
            pos[e["id"]] += len(e["tokens"])
        assert r == arr.shape[0]
    U.compare_with_plain(udirs[name]["float32"], reqs, got, dtype, f"trace_run/{dtype}")


def test_command_line_writes_random_weights_and_generates(tmp_path):
    """bin/kestrel: `--random-weights` writes a Tuganex folder from a config.json with the design's own keys, and the
    streaming harness prints the plain implementation's greedy tokens."""
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(U.T1))
    model_dir = tmp_path / "written"
    prompt = R.random_requests(U.T1["vocab"], (23,), seed=2)["r0"]
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "kestrel"), "--model", str(model_dir), "--config", str(cfg_file),
                        "--random-weights", "5", "--dtype", "float32", "--stream-test", "--stream-n", "8", "--prompt-ids",
                        ",".join(str(t) for t in prompt), "--ignore-eos", "--max-tokens", "256", "--batch-max", "2"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stdout[-2000:] + p.stderr[-2000:]
    line = [l for l in p.stdout.splitlines() if l.startswith("[STREAM] TOKIDS:")]
    assert len(line) == 1
    with open(model_dir / "config.json") as f:
        pcfg = json.load(f)
    W = P.read_checkpoint(str(model_dir / "model.safetensors"))
    assert W["l0.mlp.router"].shape == (12, 80) and W["l0.mlp.shared.sg"].shape == (1, 80) and "l1.norm2" not in W and "l2.mix.k" not in W
    toks, want = list(prompt), []
    for _ in range(8):
        want.append(int(np.argmax(P.forward(toks, W, pcfg)[-1])))
        toks.append(want[-1])
    assert [int(t) for t in line[0].split(":")[1].split()] == want
