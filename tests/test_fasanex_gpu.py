"""The Fasanex decoder in the engine against its plain statement (`plain_fasanex`): every mechanism alone, then whole models under
every way of cutting and batching the work, then generation through the scheduler (GPU)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import fasanex_util as T
import plain_fasanex as P
import replay_util as R

pytestmark = pytest.mark.gpu

DTYPES = ("float32", "bfloat16")
PART_TOL = {"float32": 3e-5, "bfloat16": 4e-2}      # of the largest entry of the plain result
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
SC = (4.0, 64, 8.0, 0.5)                            # a ramp that starts and ends inside the pairs used below


@pytest.fixture(scope="module")
def fdirs(tmp_path_factory):
    return {name: T.write_model(cfg, T.tensors_of(cfg, seed), tmp_path_factory.mktemp("fasanex_" + name)) for name, (cfg, seed) in T.CONFIGS.items()}


def _close(got, want, dtype, what, scale=None, tol=None):
    scale = float(np.abs(want).max()) if scale is None else scale
    assert np.isfinite(got).all(), f"{what}: not finite"
    err = float(np.abs(got - want).max()) / scale
    tol = PART_TOL[dtype] if tol is None else tol
    assert err <= tol, f"{what}: error {err:.3e} of the largest entry, allowed {tol:.1e}"
    return err


def _torch_dtype(dtype):
    import torch
    return {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]


def _exact(h):
    """Rows that both number formats hold, so that the parts' inputs are the same."""
    import torch
    return torch.from_numpy(np.asarray(h, dtype=np.float32)).to(torch.bfloat16).to(torch.float64).numpy()


def _rows(rng, n, width):
    return _exact(rng.standard_normal((n, width)))


class Side:
    """One of two joined mixers with the layer's output product behind it: the other one's columns are zero."""

    def __init__(self, whole, which):
        self.whole, self.which = whole, which

    def cache_spec(self):
        return self.whole.cache_spec()

    def forward(self, x, batch, cache):
        import torch
        w = self.whole
        n = w.left.out_features
        heads = torch.zeros((x.shape[0], w.out.in_features), dtype=w.dtype, device=x.device)
        if self.which == "left":
            w.left.heads_into(x, batch, cache, heads[:, :n], w.left_scale)
        else:
            w.right.heads_into(x, batch, cache, heads[:, n:], w.right_scale)
        return w.out.forward(heads)


def _left(H, G, d, conv=3, scale=0.4, cap=6.0, window=21, rotary="all"):
    """A parallel layer whose attention side is what the case is about."""
    return T.parallel(H, G, d, conv, scale, cap, window, T.rot(d, 100.0) if rotary == "all" else rotary, 1, 8, 4)


def _right(H, d, rank):
    return T.parallel(1, 1, 8, 2, 0.3, 0.0, 0, None, H, d, rank)


def _model_of(layers, width, dtype, eps=1e-6, seed=0, vocab=11):
    from kestrel_llm_b200.config import FasanexConfig, resolve_architecture
    cfg = {"architecture": "Fasanex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": [dict(L, mlp=L.get("mlp")) for L in layers]}
    W = T.tensors_of(cfg, seed)
    return resolve_architecture("Fasanex").build(FasanexConfig.from_dict(cfg), _torch_dtype(dtype), "cuda:0"), W, cfg


def _plain_mixer(layer, side, Wr, h, eps):
    m, p = layer["mixer"], "l0.mix."
    if side == "left":
        return m["left_scale"] * P.attention_side(h, Wr, p + "left.", m["left"], eps)
    if side == "right":
        return m["right_scale"] * P.time_mix_side(h, Wr, p + "right.", m["right"], eps)
    return P.MIXERS[layer["type"]](h, Wr, p, m, eps)


def _mixer_case(layer, side, dtype, page, n_tokens, cuts, seed=0, width=48, prepare=None, eps=1e-6):
    """One mixer alone (``side``: "left" / "right" of a parallel mixer, None for the whole); ``cuts`` are the portion sizes the tokens
    arrive in.  ``prepare(W, h)`` may shape weights and inputs and return other inputs, whose plain result is handed back too."""
    rng = np.random.default_rng(seed)
    model, W, _ = _model_of([layer], width, dtype, eps=eps, seed=seed)
    whole = model.blocks[0].mixer
    h = _rows(rng, n_tokens, width)
    other = None
    if prepare is not None:
        other = prepare(W, h)
        h = _exact(h)
    assert T.load_part(whole, W) == {k for k in W if k.startswith("l0.mix.")}
    Wr = T.bf16_round(W)
    want = _plain_mixer(layer, side, Wr, h, eps)
    hs = T.PartHarness(whole if side is None else Side(whole, side), dtype, max_tokens=((n_tokens + 63) // 64) * 64 + 64, page_size=page)
    got, at = [], 0
    for n in cuts:
        got.append(hs.step([(7, h[at:at + n])])[0])
        at += n
    assert at == n_tokens
    return np.concatenate(got), want, None if other is None else _plain_mixer(layer, side, Wr, _exact(other), eps)


# one entry per mechanism and shape of sizes: (label, layer, side)
MIXERS = [
    ("attention 4/2 x 16, part of a head rotated, ramp", _left(4, 2, 16, rotary=T.rot(8, 100.0, SC)), "left"),
    ("attention 3/1 x 40, one tap", _left(3, 1, 40, conv=1, window=7), "left"),
    ("attention 2/2 x 64, no cap", _left(2, 2, 64, conv=4, cap=0.0, rotary=T.rot(32, 1000.0, SC)), "left"),
    ("attention 5/1 x 12 (no multiple of 8), no window", _left(5, 1, 12, conv=9, window=0, rotary=T.rot(6, 50.0, SC)), "left"),
    ("attention 4/2 x 136, no rotation", _left(4, 2, 136, conv=2, scale=0.1, rotary=None), "left"),
    ("time mixing 2 x 24, rank 9", _right(2, 24, 9), "right"),
    ("time mixing 1 x 14, rank 3", _right(1, 14, 3), "right"),
    ("time mixing 2 x 64, rank 16", _right(2, 64, 16), "right"),
    ("time mixing 1 x 136, rank 1", _right(1, 136, 1), "right"),
    ("state space 4 x 16, state 24, 2 groups", T.mamba2(4, 16, 24, 2, 2, 4), None),
    ("state space 6 x 8, state 64, 3 groups, 1 part", T.mamba2(6, 8, 64, 3, 1, 2), None),
    ("state space 3 x 10, state 14, one tap", T.mamba2(3, 10, 14, 1, 3, 1), None),
    ("state space 2 x 128, state 128, 1 group", T.mamba2(2, 128, 128, 1, 2, 4), None),
    ("state space 2 x 72, state 200, 2 groups", T.mamba2(2, 72, 200, 2, 4, 3), None),
    ("delta 4/2 x 16/24", T.delta(4, 2, 16, 24, 3), None),
    ("delta 3/1 x 14/10", T.delta(3, 1, 14, 10, 5), None),
    ("delta 2/2 x 128/64", T.delta(2, 2, 128, 64, 4), None),
    ("delta 2/1 x 72/136, one tap", T.delta(2, 1, 72, 136, 1), None),
    ("delta 4/1 x 64/128", T.delta(4, 1, 64, 128, 4), None),
    ("joined 6/2 x 16 beside 2 x 24", T.parallel(6, 2, 16, 3, 0.3, 9.0, 13, T.rot(8, 100.0, SC), 2, 24, 8), None),
    ("joined 2/2 x 10 beside 3 x 12", T.parallel(2, 2, 10, 2, 0.5, 0.0, 40, T.rot(10, 1000.0), 3, 12, 5, (1.5, -0.4)), None),
    ("attention 4/2 x 64, rotated whole", _left(4, 2, 64, conv=4, window=40), "left"),
    ("attention 2/1 x 128, two taps, no rotation", _left(2, 1, 128, conv=2, rotary=None), "left"),
    ("time mixing 1 x 96, rank 200", _right(1, 96, 200), "right"),
    ("time mixing 2 x 128, rank 32", _right(2, 128, 32), "right"),
    ("time mixing 3 x 40, rank 8", _right(3, 40, 8), "right"),
    ("state space 2 x 136, state 48, 1 part", T.mamba2(2, 136, 48, 2, 1, 4), None),
    ("state space 1 x 300, state 16", T.mamba2(1, 300, 16, 1, 1, 3), None),
    ("delta 1/1 x 200/24", T.delta(1, 1, 200, 24, 2), None),
    ("delta 6/3 x 40/8", T.delta(6, 3, 40, 8, 3), None),
]
IDS = [m[0] for m in MIXERS]


# ---- each mechanism alone --------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("label,layer,side", MIXERS, ids=IDS)
def test_mixer_alone_whole_and_cut(dtype, label, layer, side):
    n = 150
    whole, want, _ = _mixer_case(layer, side, dtype, 16, n, [n], seed=len(label))
    _close(whole, want, dtype, f"{label}, whole")
    cut, want, _ = _mixer_case(layer, side, dtype, 8, n, [33, 2, 17, 2, 67, 8, 9, 6] + [1] * 6, seed=len(label))
    _close(cut, want, dtype, f"{label}, portions and single tokens")
    single, want, _ = _mixer_case(layer, side, dtype, 16, 21, [1] * 21, seed=len(label))
    _close(single, want, dtype, f"{label}, token by token from the first")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", [0, 5, 7, 9, 12, 14, 16, 19])
def test_first_tokens_and_shortest_requests(dtype, which):
    """Requests of one and two tokens; the first positions, where the memory is empty and the filters reach before the start; portions
    that end on and around the eight tokens a scan stages and the sixty-four of a chunk."""
    label, layer, side = MIXERS[which]
    for n, cuts in ((1, [1]), (2, [2]), (2, [1, 1]), (9, [7, 1, 1]), (17, [8, 8, 1]), (40, [3, 2, 30] + [1] * 5), (130, [64, 2, 63, 1]),
                    (200, [129, 64, 5, 2])):
        got, want, _ = _mixer_case(layer, side, dtype, 16, n, cuts, seed=n + which)
        _close(got, want, dtype, f"{label}, {n} tokens as {cuts[:3]}")


def _spike(kind, i, j):
    """Weights and inputs such that what token j wrote decides the output at token i, however far back j lies: the other inputs (returned)
    are the same with token j's value taken away."""
    def prepare(W, h):
        p = "l0.mix."
        h *= 0.05
        h[:, :3] = 0.0
        h[i, 0] = 6.0                          # i asks along channel 0
        h[j, 1] = 6.0                          # j's value stands out along channel 1
        h[j, 2] = 6.0                          # j answers as a key, along channel 2

        def now(name):                         # the filter passes the current token alone
            W[p + name][:] = 0.0
            W[p + name][:, -1] = 1.0
        if kind == "left":
            # a key is its own value: half of a head's dimensions carry the answer (through channel 2), the other half are read
            p += "left."
            now("q.conv")
            now("k.conv")
            d = W[p + "k.norm"].shape[0]
            W[p + "q.norm"][:], W[p + "k.norm"][:] = 1.0, 1.0
            W[p + "q"][:, 0], W[p + "q"][:, 1:3] = 1.0, 0.0
            W[p + "k"][:, :3] = 0.0
            W[p + "k"][:, 2] = 1.0
            W[p + "g"][:] = 0.0
            other = h.copy()
            other[j, 2] = 0.0                  # without it j neither answers nor carries anything
            assert d >= 8
            return other
        if kind == "right":
            p += "right."
            for s in "rkvgw":
                W[p + "mu." + s][:] = 0.0      # no blending with the token before
            W[p + "r"][:, 0] = W[p + "k"][:, 2] = 1.0
            W[p + "v"][:, 1] = 1.0
            W[p + "k"][:, :2] = W[p + "v"][:, [0, 2]] = 0.0
            W[p + "w2"][:] = 0.0
            W[p + "w0"][:] = -12.0             # no decay to speak of
        elif kind == "mamba2":
            now("conv")
            W[p + "conv.b"][:] = 0.0
            inner, heads = W[p + "norm"].shape[0], W[p + "D"].shape[0]
            gn = (W[p + "conv"].shape[0] - inner) // 2
            w = W[p + "in"]
            w[:, :3] = 0.0
            w[inner:2 * inner, 1] = 1.0                           # x
            w[2 * inner:2 * inner + gn, 2] = 1.0                  # B
            w[2 * inner + gn:2 * inner + 2 * gn, 0] = 1.0         # C
            w[2 * inner + 2 * gn:] = 0.0
            W[p + "dt_bias"][:] = 0.5
            W[p + "A_log"][:] = -12.0
            assert heads == W[p + "dt_bias"].shape[0]
        else:
            for s in "qkv":
                now(s + ".conv")
            W[p + "q"][:, 0] = W[p + "k"][:, 2] = 1.0
            W[p + "v"][:, 1] = 1.0
            W[p + "k"][:, :2] = W[p + "v"][:, [0, 2]] = 0.0
            W[p + "q"][:, 1:3] = 0.0
            W[p + "b"][:] = 0.0
            W[p + "b"][:, 2] = 3.0             # j writes; what the others write is small beside it
            h[np.arange(len(h)) != j, 3] = 6.0
            W[p + "b"][:, 3] = -3.0
            W[p + "q"][:, 3] = W[p + "k"][:, 3] = W[p + "v"][:, 3] = 0.0
            W[p + "A_log"][:] = -12.0
        other = h.copy()
        other[j, 1] = 0.0
        return other
    return prepare


SPIKES = {"left": (_left(2, 1, 16, scale=1.0, cap=30.0, window=0, rotary=T.rot(4, 1e6)), "left"), "right": (_right(2, 16, 4), "right"),
          "mamba2": (T.mamba2(4, 16, 24, 2, 2, 4), None), "delta": (T.delta(2, 1, 16, 24, 3), None)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("where", ["far", "page_end", "page_start", "first_token", "previous_token"])
@pytest.mark.parametrize("kind", sorted(SPIKES))
def test_mixer_reads_what_lies_far_back(kind, dtype, decode, where):
    """One token's value stands out and one later token asks for it: hundreds of tokens back, on either side of a page border, at the
    request's first position, and right before.  The plain result without that value differs widely from the true one: the engine must
    match the true one, in a prompt's portions and decoded token by token."""
    page, n, i = 16, 300, 297
    j = {"far": 3, "page_end": 255, "page_start": 256, "first_token": 0, "previous_token": i - 1}[where]
    cuts = [290] + [1] * 10 if decode else [140, 160]
    layer, side = SPIKES[kind]
    got, want, other = _mixer_case(layer, side, dtype, page, n, cuts, prepare=_spike(kind, i, j))
    scale = float(np.abs(want).max())
    assert np.abs(want[i] - other[i]).max() > 0.25 * np.abs(want[i]).max(), f"{kind}, {where}: the case does not tell whether token {j} was read"
    if dtype == "bfloat16" and kind in ("mamba2", "delta"):
        # a token that does not ask reads a state whose one huge entry cancels in its sum: rounding its operands decides what is left
        rows = [t for t in range(n) if t <= j or t == i]
        got, want, i = got[rows], want[rows], rows.index(i)
        other = other[rows]
    _close(got, want, dtype, f"{kind}, {where}", scale=scale, tol={"float32": 3e-4, "bfloat16": 4e-2}[dtype])
    assert np.abs(got[i] - want[i]).max() < 0.1 * np.abs(want[i] - other[i]).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("d", [16, 128])
@pytest.mark.parametrize("window", [16, 21, 64, 100])
def test_window_edges(dtype, decode, d, window):
    """The last key inside the window and the first one outside it, in prompts and in decoding, at heads of both kernels."""
    n, i = 290, 281
    for j, inside in ((i - window + 1, True), (i - window, False)):
        layer = _left(2, 1, d, scale=16.0 / d, cap=30.0, window=window, rotary=T.rot(4, 1e6))
        cuts = [250, 30] + [1] * 10 if decode else [120, 170]
        got, want, other = _mixer_case(layer, "left", dtype, 16, n, cuts, prepare=_spike("left", i, j))
        moved = np.abs(want[i] - other[i]).max() / np.abs(want[i]).max()
        assert (moved > 0.25) == inside and (inside or moved == 0.0)
        _close(got, want, dtype, f"window {window}, key {'inside' if inside else 'outside'}", tol={"float32": 3e-4, "bfloat16": 4e-2}[dtype])
        # the row itself, which is small where the key lies outside
        _close(got[i], want[i], dtype, f"window {window}, the row that asks", tol={"float32": 3e-4, "bfloat16": 5e-2}[dtype])


@pytest.mark.parametrize("captured", [False, True])
@pytest.mark.parametrize("d,G,H", [(128, 2, 4), (64, 1, 4), (128, 1, 16)])
@pytest.mark.parametrize("window,cap", [(0, 5.0), (0, 0.0), (100, 5.0), (700, 8.0), (1500, 0.0), (4000, 6.0)])
def test_single_tokens_on_the_decode_kernel(captured, window, cap, d, G, H):
    """Capped scores over a window, or all keys, on the TMA decode kernel against the mma.sync kernel: requests of very unequal lengths in
    one step, key ranges cut into slices inside a cluster and through scratch, with a recorded step's fixed number of slices."""
    import torch
    from types import SimpleNamespace
    from kestrel_llm_b200.cache import CacheManager
    from kestrel_llm_b200.csrc import ops
    from kestrel_llm_b200.engine.batch import Entry, StepBatch
    from kestrel_llm_b200.parts import PagedKVSpec
    lengths = [1, 63, 64, 65, 700, 1499, 1500, 1501, 2900]
    cache = CacheManager([PagedKVSpec(G, d)], torch.bfloat16, "cuda:0", 16, sum(-(-(n + 1) // 16) for n in lengths) + 4, 12, 1 << 12)
    cache.shuffle_free(3)
    gen = torch.Generator(device="cuda:0").manual_seed(d + window)
    cache.k[0].normal_(0.0, 1.0, generator=gen)
    cache.v[0].normal_(0.0, 1.0, generator=gen)
    entries = []
    for i, n in enumerate(lengths):
        cache.admit(i)
        cache.reserve(i, n)
        cache.commit(i, n)
        cache.reserve(i, 1)
        entries.append(Entry(i, [0], []))
    batch = StepBatch(entries, cache, "cuda:0")
    if captured:
        batch = SimpleNamespace(**{k: getattr(batch, k) for k in ("max_count", "num_seqs", "max_kv_len", "cu_seqlens", "kv_lens", "device_buffer", "layout",
                                                                "positions", "seq_of_token", "num_tokens", "counts")}, captured=True)
    q = torch.empty((len(lengths), H * d), dtype=torch.bfloat16, device="cuda:0").normal_(0.0, 1.0, generator=gen)
    table = StepBatch.block_table(batch, 0) if not captured else StepBatch(entries, cache, "cuda:0").block_table(0)
    out, want = torch.empty_like(q), torch.empty_like(q)
    assert ops.attention_decode_capped(q, cache.k[0], cache.v[0], batch, table, 16, out, H, G, d, window, d ** -0.5, cap)
    ops.raise_on_kernel_error()
    ops.attention_plain_ex(q, cache.k[0], cache.v[0], batch.positions, batch.seq_of_token, table, 16, want, H, G, d, d, window, 0, None, d ** -0.5,
                           ops.ScoreOptions(cap))
    _close(out.float().cpu().numpy(), want.float().cpu().numpy(), "bfloat16", f"window {window}, cap {cap}", tol=1.5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_ramp_and_far_positions(dtype):
    """Positions into the thousands, a rotation over part of the head whose ramp starts and ends inside its pairs; the plain result with
    unstretched frequencies and the one without the magnitude differ widely from the true one."""
    layer = _left(2, 1, 32, scale=0.6, cap=0.0, window=0, rotary=T.rot(24, 200.0, (8.0, 64, 8.0, 1.0)))
    n = 2100
    got, want, _ = _mixer_case(layer, "left", dtype, 32, n, [2048, 40, 2] + [1] * 10, seed=3, width=32)
    tail = slice(2040, n)
    # a float32 angle at position p is off by up to p 2^-24 radians, 1.3e-4 here, and the scores move by as much
    _close(got[tail], want[tail], dtype, "rotation at positions beyond 2,040", scale=float(np.abs(want).max()), tol={"float32": 2e-4, "bfloat16": 4e-2}[dtype])
    _, W, _ = _model_of([layer], 32, "float32", seed=3)
    Wr, h = T.bf16_round(W), _rows(np.random.default_rng(3), n, 32)
    import copy
    plain = copy.deepcopy(layer)
    plain["mixer"]["left"]["rot"] = T.rot(24, 200.0)
    other = _plain_mixer(plain, "left", Wr, h[:400], 1e-6)
    assert np.abs(other[200:] - want[200:400]).max() > 0.1 * np.abs(want).max()


def test_block_norms_around_zero_and_bounded_feed_forward():
    """One layer's block alone, float32: norm, mixer, norm of the result, add; then the same around the feed-forward with both of its
    bounds reached.  Also a block without feed-forward, and what an unbounded feed-forward and plain norm weights would give."""
    import torch
    from kestrel_llm_b200.cache import CacheManager
    from kestrel_llm_b200.engine.batch import Entry, StepBatch
    for layer in (T.layer(T.delta(2, 1, 12, 8, 3), 40, 0.7), T.layer(T.delta(2, 1, 12, 8, 3), None), T.layer(T.mamba2(2, 8, 10, 1, 2, 3), 52, 1.3)):
        model, W, cfg = _model_of([layer], 36, "float32", eps=1e-5, seed=4)
        block = model.blocks[0]
        T.load_part(block, W)
        Wr = T.bf16_round(W)
        x = _rows(np.random.default_rng(1), 23, 36) * 3.0
        want = P.layer_forward(x.copy(), Wr, cfg, 0)
        cache = CacheManager([block.mixer.cache_spec()], torch.float32, "cuda:0", 16, 8, 2, 1 << 12)
        cache.admit(1)
        cache.reserve(1, 23)
        cache.clear_admitted()
        batch = StepBatch([Entry(1, [0] * 23, [])], cache, "cuda:0")
        res, pending = block.forward(torch.from_numpy(x.astype(np.float32)).to("cuda:0"), None, batch, cache.layer(0, True))
        assert pending is None
        _close(res.cpu().numpy().astype(np.float64), want, "float32", f"block, {layer['type']}, mlp {layer['mlp']}")
        if layer["mlp"]:
            loose = json.loads(json.dumps(cfg))
            loose["layers"][0]["mlp"]["limit"] = 50.0
            assert np.abs(P.layer_forward(x.copy(), Wr, loose, 0) - want).max() > 0.05 * np.abs(want).max()


@pytest.mark.parametrize("limit", [0.4, 1.0, 7.0])
@pytest.mark.parametrize("T_,ff,K", [(3, 40, 24), (5, 256, 128), (40, 264, 72), (129, 264, 72), (700, 1024, 256), (2048, 520, 136), (300, 100, 70)])
def test_bounded_activation_in_the_products_epilogue(limit, T_, ff, K):
    """bfloat16: the bounded gated activation as the epilogue of every form of the tcgen05 product, and on slices, against numpy."""
    import torch
    from kestrel_llm_b200.csrc import ops
    rng = np.random.default_rng(T_ + ff)
    x = torch.from_numpy(rng.standard_normal((T_, K)).astype(np.float32)).to(torch.bfloat16)
    w = torch.from_numpy((2.0 * rng.standard_normal((2 * ff, K)) / np.sqrt(K)).astype(np.float32)).to(torch.bfloat16)
    z = x.to(torch.float64).numpy() @ w.to(torch.float64).numpy().T
    g, u = np.minimum(z[:, :ff], limit), np.clip(z[:, ff:], -limit, limit)
    want = g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)
    xd, wd = x.to("cuda:0"), w.to("cuda:0")
    scale = float(np.abs(want).max())
    got = ops.gate_up_swiglu(xd, wd, ff, limit=limit).float().cpu().numpy()
    ops.raise_on_kernel_error()
    _close(got, want, "bfloat16", "fused", scale=scale, tol=1e-2)
    sliced = torch.empty((T_, ff), dtype=torch.bfloat16, device="cuda:0")
    ops.swiglu(ops.Partials(ops.linear(xd, wd)), sliced, limit)
    _close(sliced.float().cpu().numpy(), want, "bfloat16", "on slices", scale=scale, tol=1e-2)


@pytest.mark.parametrize("which", [7, 9, 12, 13, 14, 16, 18, 24, 25, 26, 29])
def test_chunked_and_stepwise_forms_against_the_sequential_scan(which):
    """bfloat16: portions in chunks on the tensor cores and steps of few tokens in one kernel, against the same mixer on the sequential
    float32 scan: they round their operands alike, so they stand closer to each other than to the plain statement; decays from slow to
    so fast that a chunk forgets everything several times over."""
    from kestrel_llm_b200.parts import HeadDeltaMixer, StateSpaceMixer, TimeMixRecurrence
    label, layer, side = MIXERS[which]

    def fast(W, h):
        for name in ("l0.mix.A_log", "l0.mix.right.w0"):
            if name in W:
                W[name][:] = np.linspace(-6.0, 4.0, W[name].size)
        return h.copy()
    n, cuts = 300, [150, 64, 2, 3, 70, 4, 1, 6]
    fused, want, _ = _mixer_case(layer, side, "bfloat16", 16, n, cuts, seed=which, prepare=fast)
    classes = (HeadDeltaMixer, StateSpaceMixer, TimeMixRecurrence)
    for c in classes:
        c.chunked = c.one_kernel = False
    try:
        plain, _, _ = _mixer_case(layer, side, "bfloat16", 16, n, cuts, seed=which, prepare=fast)
    finally:
        for c in classes:
            c.chunked = c.one_kernel = True
    _close(fused, want, "bfloat16", label)
    _close(fused, plain, "bfloat16", f"{label}, against the scan", tol=3e-2)


@pytest.mark.parametrize("T_,K,n,rank", [(5, 128, 256, 64), (40, 72, 128, 8), (100, 256, 384, 384), (300, 136, 256, 40), (1500, 512, 512, 64), (300, 64, 128, 16),
                                         (20, 70, 30, 7)])
def test_products_of_several_inputs_in_one_launch(T_, K, n, rank):
    """Five products over inputs of their own in one launch of the tcgen05 kernel, and a launch a group, against numpy; a last group of
    fewer rows; groups that are no whole number of tiles take the second way by themselves."""
    import torch
    from kestrel_llm_b200.csrc import ops
    rng = np.random.default_rng(T_ + n)
    x = torch.from_numpy(rng.standard_normal((5, T_, K)).astype(np.float32)).to(torch.bfloat16)
    w = torch.from_numpy((rng.standard_normal((4 * n + rank, K)) / np.sqrt(K)).astype(np.float32)).to(torch.bfloat16)
    xs, ws = x.to(torch.float64).numpy(), w.to(torch.float64).numpy()
    want = np.concatenate([xs[g] @ ws[g * n:(g + 1) * n].T for g in range(5)], axis=1)
    xd, wd = x.to("cuda:0"), w.to("cuda:0")
    for on in (True, False):
        ops.linear_groups_fused = on
        try:
            got = ops.linear_groups(xd, wd, n).reduce(torch.float32).cpu().numpy()
        finally:
            ops.linear_groups_fused = True
        ops.raise_on_kernel_error()
        _close(got, want, "bfloat16", f"one launch: {on}", tol=1e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", [0, 7, 9, 12, 14, 18, 19])
def test_requests_beside_each_other_and_memory_used_again(dtype, which):
    """Two requests of unequal portions in one batch against each request alone; a third request then runs on the pages AND the state
    slot the first two gave back: what they left there must not reach it."""
    label, layer, side = MIXERS[which]
    rng = np.random.default_rng(3)
    model, W, _ = _model_of([layer], 48, dtype, seed=2)
    T.load_part(model.blocks[0].mixer, W)
    mixer = model.blocks[0].mixer if side is None else Side(model.blocks[0].mixer, side)
    Wr = T.bf16_round(W)
    ha, hb, hc = _rows(rng, 130, 48), _rows(rng, 107, 48), _rows(rng, 64, 48)
    wa, wb, wc = (_plain_mixer(layer, side, Wr, h, 1e-6) for h in (ha, hb, hc))
    hs = T.PartHarness(mixer, dtype, max_tokens=256, page_size=16, slots=2)
    got_a, got_b, at_a, at_b = [], [], 0, 0
    for ka, kb in [(7, 2), (2, 13), (100, 2), (2, 75), (3, 1), (1, 1), (15, 13)]:
        out = hs.step([(2, ha[at_a:at_a + ka]), (3, hb[at_b:at_b + kb])])
        got_a.append(out[0])
        got_b.append(out[1])
        at_a, at_b = at_a + ka, at_b + kb
    assert (at_a, at_b) == (130, 107)
    _close(np.concatenate(got_a), wa, dtype, f"{label}, request a in portions beside b")
    _close(np.concatenate(got_b), wb, dtype, f"{label}, request b in portions beside a")
    hs.cache.release(2)
    hs.cache.release(3)
    _close(np.concatenate([hs.step([(4, hc[:50])])[0]] + [hs.step([(4, hc[t:t + 1])])[0] for t in range(50, 64)]), wc, dtype,
           f"{label}, a new request on pages and a slot that were given back")


# ---- whole models ----------------------------------------------------------------------------------

LENGTHS = {"F1": (1, 2, 37, 70, 129, 64), "F2": (3, 50, 97, 130, 17), "F3": (2, 210, 33)}
LENGTHS_MIXED = {"F1": (5, 33, 70, 129, 47, 90, 16, 65, 31), "F2": (3, 50, 97, 130, 64, 81, 17, 49)}


def _run(fdirs, name, dtype, family, lengths=None, page_size=16, batch_max=4, graphs=False, **kw):
    reqs = T.requests(name, lengths or LENGTHS[name], seed=11 + len(name))
    steps, max_tokens = family(reqs, **kw)
    engine = R.make_engine(fdirs[name][dtype], dtype, max_tokens, page_size=page_size, batch_max=batch_max, graphs=graphs)
    got = R.run_trace(engine, steps)
    assert engine.cache.live_requests() == 0
    engine.cache.check()
    T.compare_with_plain(fdirs[name]["float32"], reqs, got, dtype, f"{name}/{dtype}/{family.__name__}")
    return got


def test_residual_stream_after_every_layer(fdirs):
    """float32: the stream after each layer against the plain implementation's, so that a fault names its place."""
    import torch
    from kestrel_llm_b200.engine import Entry
    from kestrel_llm_b200.engine.batch import StepBatch
    for name in T.CONFIGS:
        toks = T.requests(name, (75,), seed=4)["r0"]
        pcfg, W = P.read_model(fdirs[name]["float32"])
        want = []
        P.forward(pcfg, W, toks, want)
        engine = R.make_engine(fdirs[name]["float32"], "float32", 128)
        engine.cache.admit(0)
        engine.cache.reserve(0, len(toks))
        engine.cache.clear_admitted()
        batch = StepBatch([Entry(0, toks, [])], engine.cache, "cuda:0")
        model = engine.model
        x, pending = model.forward_embed(batch)
        for i in range(len(model.order)):
            x, pending = model.forward_calls(x, pending, batch, engine.cache, i, i + 1)
            now = x.clone()               # a block hands on at most the normed stream: nothing is left to add
            err = np.abs(now.cpu().numpy() - want[i]).max() / np.abs(want[i]).max()
            assert err < 2e-5, f"{name}: layer {i}: error {err:.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["F1", "F2", "F3"])
@pytest.mark.parametrize("family", [R.trace_whole, R.trace_tail_decode, R.trace_portions])
def test_model_alone_whole_decoded_and_in_portions(fdirs, name, dtype, family):
    _run(fdirs, name, dtype, family)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,page", [("F1", 16), ("F2", 16), ("F1", 8), ("F2", 64)])
def test_model_mixed_batches_pages_and_slots_used_again(fdirs, name, dtype, page):
    """Up to four live requests, portions beside single tokens; more requests than slots and than the pool holds, so that pages and
    slots are used again."""
    _run(fdirs, name, dtype, R.trace_mixed, lengths=LENGTHS_MIXED[name], page_size=page, live_max=4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_model_of_tensor_core_sizes_mixed_batches(fdirs, dtype):
    _run(fdirs, "F3", dtype, R.trace_mixed, lengths=(150, 33, 400, 129, 260, 90, 16), live_max=4, sizes=(70, 2, 140, 3, 66, 2, 210, 5))
    _run(fdirs, "F3", dtype, R.trace_portions, lengths=(300, 131), sizes=(70, 2, 130, 2, 50, 3, 170, 2, 31, 4))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["F1", "F2", "F3"])
def test_long_decoding_through_captured_steps(fdirs, name, dtype):
    """Five prompt tokens, then 215 tokens one by one through captured decode steps."""
    _run(fdirs, name, dtype, R.trace_tail_decode, lengths=(220,), graphs=True, tail=215)


@pytest.mark.parametrize("name", ["F1", "F2"])
def test_cuttings_agree_in_float32(fdirs, name):
    """The float32 logits of a position do not depend on how the work was cut or batched, beyond the order of sums."""
    a = _run(fdirs, name, "float32", R.trace_whole, lengths=LENGTHS_MIXED[name])
    b = _run(fdirs, name, "float32", R.trace_mixed, lengths=LENGTHS_MIXED[name], live_max=4)
    c = _run(fdirs, name, "float32", R.trace_portions, lengths=LENGTHS_MIXED[name])
    scale = max(float(np.abs(a[r][p]).max()) for r in a for p in a[r])
    for r in a:
        for p in a[r]:
            assert max(np.abs(a[r][p] - b[r][p]).max(), np.abs(a[r][p] - c[r][p]).max()) <= 1e-5 * scale, f"{name}: request {r} position {p}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(fdirs, dtype):
    """`LLM.generate`: six requests through three slots, prompts in portions of at most 24 tokens."""
    from kestrel_llm_b200 import LLM, SamplingParams
    name = "F1"
    prompts = list(T.requests(name, (1, 40, 70, 9, 33, 55), seed=4).values())
    llm = LLM(fdirs[name][dtype], dtype=dtype, page_size=16, batch_max=3, max_tokens=512, prefill_batch=24, max_step_tokens=64)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True))
    pcfg, W = P.read_model(fdirs[name]["float32"])
    for prompt, o in zip(prompts, outs):
        toks = list(prompt)
        assert len(o.token_ids) == 8
        for got in o.token_ids:
            logits = P.forward(pcfg, W, toks)[-1]
            want = int(np.argmax(logits))
            if got != want:          # a tie within rounding is not a fault; anything else is
                gap = float(logits[want] - logits[got])
                assert gap <= (2e-5 if dtype == "float32" else 4e-2) * float(np.abs(logits).max()), f"{dtype}: token {got} instead of {want}"
            toks.append(got)


# ---- the programs a user runs ------------------------------------------------------------------------

@pytest.mark.parametrize("dtype,graphs", [("float32", 1), ("bfloat16", 1), ("bfloat16", 0)])
def test_trace_replay_program(fdirs, dtype, graphs, tmp_path):
    """bin/trace_run in a process of its own on a mixed trace: four slots for seven requests, decode steps replayed from captured graphs
    (the default) and launched kernel by kernel."""
    name = "F2"
    reqs = T.requests(name, (5, 33, 70, 47, 90, 16, 65), seed=21)
    steps, max_tokens = R.trace_mixed(reqs, live_max=4, seed=5)
    lines = "".join(json.dumps(dict(step=i, **s)) + "\n" for i, s in enumerate(steps))
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", fdirs[name][dtype], "--dtype", dtype, "--out", str(out),
                        "--max-tokens", str(max_tokens), "--cuda-graphs", str(graphs)], input=lines, capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    V = T.CONFIGS[name][0]["vocab"]
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
    T.compare_with_plain(fdirs[name]["float32"], reqs, got, dtype, f"trace_run/{dtype}")


def test_command_line_writes_random_weights_and_generates(tmp_path):
    """bin/kestrel: `--random-weights` writes a Fasanex folder from a config.json with the design's own keys, and the streaming harness
    prints the plain implementation's greedy tokens."""
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(T.F1))
    model_dir = tmp_path / "written"
    prompt = R.random_requests(T.F1["vocab"], (23,), seed=2)["r0"]
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "kestrel"), "--model", str(model_dir), "--config", str(cfg_file),
                        "--random-weights", "5", "--dtype", "float32", "--stream-test", "--stream-n", "8", "--prompt-ids",
                        ",".join(str(t) for t in prompt), "--ignore-eos", "--max-tokens", "256", "--batch-max", "2"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stdout[-2000:] + p.stderr[-2000:]
    line = [l for l in p.stdout.splitlines() if l.startswith("[STREAM] TOKIDS:")]
    assert len(line) == 1
    pcfg, W = P.read_model(str(model_dir))
    assert "l1.norm2" not in W and "l0.norm2" in W and abs(float(W["l0.norm1"].mean())) < 0.1
    toks, want = list(prompt), []
    for _ in range(8):
        want.append(int(np.argmax(P.forward(pcfg, W, toks)[-1])))
        toks.append(want[-1])
    assert [int(t) for t in line[0].split(":")[1].split()] == want
