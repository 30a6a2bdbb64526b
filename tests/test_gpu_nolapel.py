"""The Nolapel decoder on the GPU against the plain implementation (tests/plain_nolapel.py): every mechanism alone, then
whole models: prompts whole, in portions and token by token, unequal batches, slots and pages used again, keys far away, at
page borders and at the edges of windows, first tokens, long decoding, and greedy generation through the entry point."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import harness as H
import plain_nolapel as P
from harness import MixerRig, max_err as err, random_rows as inputs, whole_portions_and_batches
from nolapel_configs import ALL, att, left, moe, par, random_config, ssm

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": H.TOL_F32, "bfloat16": H.TOL_BF16}


def K():
    from lastengine_b200.ops import kernels
    return kernels


def dev(a, dt=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(DEV, dt)


def host(t):
    return t.double().cpu().numpy()


def batch_of(lens, pos0, slots, tokens=None):
    from lastengine_b200.engine.batch import BatchBuilder
    tokens = tokens or [[0] * n for n in lens]
    return BatchBuilder(torch.device(DEV)).build(slots, tokens, pos0, [], {0: np.zeros((len(slots), 1), dtype=np.int32)})


def att_params(D, m, eps=1e-5):
    return mixer_params(D, m, "attention", eps)


def mixer_params(D, m, kind, eps=1e-5):
    """What the plan gives the mixer of a one-layer model."""
    from lastengine_b200.registry import plan_from_config
    cfg = {"architecture": "Nolapel", "vocab": 8, "width": D, "norm": {"eps": eps},
           "layers": [{"type": kind, "mixer": m, "mlp": None}]}
    return dict(plan_from_config(cfg).layers[0].mixer.params)


def left_params(D, m, eps=1e-5):
    return dict(mixer_params(D, par(m, 1, 8), "parallel", eps)["left"].params)


# ---- pointwise norms, embedding, the stream's product ----------------------------------------------------------
def norm_of(D, seed):
    a, w, b = 0.4 + 0.1 * seed, 1 + 0.3 * inputs(1, D, seed, False)[0], 0.2 * inputs(1, D, seed + 1, False)[0]
    return (a, dev(w), dev(b)), lambda x: P.pointwise_tanh(x, w.astype(np.float32), np.float32(a), b.astype(np.float32))


@pytest.mark.parametrize("M,D", [(1, 40), (7, 42), (5, 64), (3, 1001), (9, 2048), (700, 96), (2, 5000)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16", "added"])
def test_a_pointwise_norm(M, D, dtype):
    (a, w, b), plain = norm_of(D, 2)
    x = dev(inputs(2 * M, D, 3, False, 2.0))
    rows = torch.randperm(2 * M)[:M].to(torch.int32).to(DEV) if dtype != "added" else None
    src = host(x)[rows.cpu().numpy()] if rows is not None else host(x)[:M]
    out = dev(inputs(M, D, 4, False), torch.bfloat16 if dtype == "bfloat16" else torch.float32)
    before = host(out)
    K().pointwise_norm(out, x, a, w, b, rows=rows, add=dtype == "added")
    want = plain(src) + (before if dtype == "added" else 0)
    assert err(host(out), want) < (5e-3 if dtype == "bfloat16" else 1e-6)


@pytest.mark.parametrize("M,D", [(1, 40), (7, 42), (5, 64), (3, 1001), (9, 2048), (300, 96), (1025, 40), (515, 33)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16", None])
@pytest.mark.parametrize("two", [False, True])
def test_a_result_is_normed_added_and_the_stream_normed_again(M, D, dtype, two):
    n1, plain1 = norm_of(D, 2)
    n2, plain2 = norm_of(D, 5)
    x, y, y2 = dev(inputs(M, D, 1, False, 2.0)), dev(inputs(M, D, 2, False)), dev(inputs(M, D, 3, False))
    h = None if dtype is None else torch.zeros(M, D, dtype=DT[dtype], device=DEV)
    y_all = 0.7 * host(y) - 1.5 * host(y2) if two else host(y)
    want = host(x) + plain1(y_all)
    K().pointwise_norm_sum(x, y, n1, h=h, next_norm=n2 if h is not None else None, weighted=(0.7, y2, -1.5) if two else None)
    assert err(host(x), want) < 1e-6
    if h is not None:
        assert err(host(h), plain2(host(x))) < (5e-3 if dtype == "bfloat16" else 1e-6)


@pytest.mark.parametrize("M,D", [(1, 40), (3, 42), (5, 33), (70, 128)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_stream_s_columns_and_its_product_with_the_embedding_output(M, D, dtype):
    bf = dtype == "bfloat16"
    x, x0 = inputs(M, D, 1, False, 2.0), inputs(M, D, 2, False)
    W, s = inputs(D, 2 * D, 3, True, D ** -0.5), inputs(1, D, 4, False)[0]
    pair = torch.zeros(M, 2 * D, dtype=DT[dtype], device=DEV)
    xd, x0d = dev(x), dev(x0)
    K().stream_columns(pair[:, D:], x0d)
    K().stream_columns(pair[:, :D], xd, dev(s), fill=True)
    assert torch.equal(pair[:, D:], x0d.to(DT[dtype])) and torch.equal(pair[:, :D], dev(x).to(DT[dtype]))
    assert err(host(xd), np.broadcast_to(s.astype(np.float32), (M, D))) == 0
    K().linear(xd, pair, dev(W, DT[dtype]), K().ACCUMULATE)
    K().check_device_status()
    assert err(host(xd), np.concatenate([x, x0], 1) @ W.T + s) < (1e-2 if bf else 1e-5)


@pytest.mark.parametrize("D", [40, 42, 1024])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("buckets,mp,mc", [(97, 31, 5), (1, 1, 1), (65521, 2 ** 31, 2 ** 33 + 1), (12, 0, 7)])
def test_token_pairs_over_steps_of_every_kind(D, dtype, buckets, mp, mc):
    """Unequal sequences in steps of many rows, two, one; a padding sequence among them; slots given out in another order.
    Factors beyond 32 bits: the hash is an integer's remainder, not a wrapped one's."""
    V = 50
    table, pairs = inputs(V, D, 1, True), inputs(buckets + 1, D, 2, True)
    seqs = {2: np.random.default_rng(3).integers(0, V, 40).tolist(), 0: [7] * 9, 4: np.random.default_rng(4).integers(0, V, 20).tolist()}
    state = torch.full((5, 1), 777, dtype=torch.int32, device=DEV)
    td, pd = dev(table, DT[dtype]), dev(pairs, DT[dtype])
    at = {s: 0 for s in seqs}
    for cut in ({2: 5, 0: 1, 4: 1}, {2: 1, 0: 1, 4: 1}, {4: 2, 2: 30, 0: 3}, {0: 4, 2: 4}, {4: 16}):
        slots, toks, pos = [], [], []
        for s, n in cut.items():
            slots.append(s), toks.append(seqs[s][at[s]:at[s] + n]), pos.append(at[s])
        slots.append(-1), toks.append([3, 4]), pos.append(0)
        b = batch_of([len(t) for t in toks], pos, slots, toks)
        x = torch.zeros(sum(map(len, toks)), D, device=DEV)
        K().embed_pairs(x, td, pd, b.tokens, state, b, mp, mc)
        r = 0
        for s, t in zip(slots[:-1], toks[:-1]):
            whole = seqs[s][:at[s] + len(t)]
            want = (table[whole] + pairs[P.pair_rows(whole, {"buckets": buckets, "mul_prev": mp, "mul_cur": mc})])[at[s]:]
            assert err(host(x)[r:r + len(t)], want) < 1e-6
            r += len(t)
            at[s] += len(t)
            assert int(state[s, 0]) == t[-1]
    assert int(state[1, 0]) == 777 and int(state[3, 0]) == 777


# ---- attention with convolved keys as values -------------------------------------------------------------------
ATT_CASES = [  # heads, kv heads, dim, taps, scale, window, (coef, every)
    (8, 2, 64, 4, 0.12, 40, (0.4, 16)),         # the tcgen05 prompt kernel, the decode kernel that prepares its rows
    (4, 4, 64, 3, 0.12, 100, None),
    (8, 1, 64, 2, 0.12, 0, (0.2, 10)),
    (6, 2, 128, 4, 0.08, 70, (0.3, 64)),
    (4, 2, 96, 3, 0.1, 33, (0.3, 20)),
    (6, 1, 32, 5, 0.2, 150, (0.5, 7)),
    (12, 3, 48, 3, 0.15, 64, (0.3, 5)),         # stored at 64
    (5, 1, 80, 1, 0.1, 65, (0.3, 33)),          # stored at 96, one tap
    (3, 3, 20, 3, 0.3, 1, (1.0, 2)),            # a window of one position
    (5, 5, 12, 16, 0.3, 21, (0.4, 3)),
    (4, 2, 200, 4, 0.07, 50, (0.3, 16)),        # the general kernel
    (34, 2, 64, 3, 0.12, 50, (0.3, 16)),        # more heads on a key head than the decode kernel takes
    (3, 1, 130, 2, 0.1, 33, None),
]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ATT_CASES)
def test_attention_alone_whole_in_portions_and_batched(case, dtype):
    m = att(*case)
    rig = MixerRig("attention", att_params(48, m), dtype, seed=3)
    whole_portions_and_batches(rig, lambda h: P.biased_attention(h, rig.plain, m, 1e-5), (150, 1, 67), 21,
                               [0, 2, 3, 8, 9, 21], TOL[dtype], dtype == "bfloat16")


LEFT_CASES = [  # heads, kv heads, dim, vdim, scale, rotated, base
    (4, 2, 64, 64, 0.12, 64, 1e4), (8, 1, 64, 64, 0.12, 64, 1e6), (3, 3, 64, 64, 0.12, 20, 500.0), (6, 2, 128, 128, 0.08, 128, 1e6),
    (4, 1, 48, 48, 0.15, 48, 1e5), (4, 2, 64, 32, 0.12, 64, 1e4), (2, 1, 40, 100, 0.15, 24, 2000.0), (5, 5, 12, 20, 0.3, None, 1.0),
    (3, 1, 22, 10, 0.25, 10, 5000.0), (12, 3, 200, 40, 0.07, 100, 1e4), (40, 2, 32, 32, 0.2, 32, 1e4)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", LEFT_CASES)
def test_sink_attention_alone_whole_in_portions_and_batched(case, dtype):
    m = left(*case)
    rig = MixerRig("attention", left_params(48, m), dtype, seed=4)
    whole_portions_and_batches(rig, lambda h: P.sink_attention(h, rig.plain, m), (150, 1, 67), 21,
                               [0, 2, 3, 8, 9, 21], TOL[dtype], dtype == "bfloat16")


def variant(fn, **swap):
    """The plain implementation with some of its functions replaced."""
    saved = {n: getattr(P, n) for n in swap}
    try:
        for n, f in swap.items():
            setattr(P, n, f)
        return fn()
    finally:
        for n, f in saved.items():
            setattr(P, n, f)


def test_every_constant_of_the_attention_shows():
    """Mistakes planted in the plain implementation move the result well beyond the tolerance."""
    m = att(4, 2, 16, 3, 0.4, 30, (0.5, 8))
    rig = MixerRig("attention", att_params(32, m), "float32", seed=4)
    h = inputs(70, 32, 1, False)
    run = lambda mm=m: P.biased_attention(h, rig.plain, mm, 1e-5)  # noqa: E731
    want = run()
    assert err(rig.alone(h), want) < H.TOL_F32
    assert err(variant(run, softmax_with_sink=lambda s, mask, sink, f=P.softmax_with_sink: f(s, mask, None)), want) > 0.02
    assert err(variant(run, slopes=lambda n: 2.0 ** (-8.0 * np.arange(n) / n)), want) > 0.02
    assert err(variant(run, slopes=np.zeros), want) > 0.02
    assert err(variant(run, query_temperature=lambda p, t: 1 + t["coef"] * np.log(np.floor(p / t["every"]) + 1)), want) > 1e-3
    assert err(run(dict(m, q_temp=None)), want) > 0.02
    assert err(run(dict(m, mask={"size": 29})), want) > 1e-3
    # the values are keys before their norm
    normed = lambda q, k, v, *a, f=P.weighted_values: f(q, k, k, *a)  # noqa: E731
    assert err(variant(run, weighted_values=normed), want) > 0.02
    lm = left(4, 2, 16, 16, 0.4, 16, 100.0)
    rig = MixerRig("attention", left_params(32, lm), "float32", seed=4)
    want = P.sink_attention(h, rig.plain, lm)
    assert err(rig.alone(h), want) < H.TOL_F32
    w0 = dict(rig.plain, sink=rig.plain["sink"] * lm["scale"])
    assert err(P.sink_attention(h, w0, lm), want) > 0.02
    assert err(P.sink_attention(h, rig.plain, dict(lm, rot={"dims": 8, "base": 100.0})), want) > 0.02


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [64, 96, 128, 20])
def test_the_sink_takes_its_share_from_the_first_row_on(dim, dtype):
    """Scores far below a sink (a row then gives next to nothing), far above it, and of its size; rows with one key."""
    D, bf = 16, dtype == "bfloat16"
    m = left(2, 1, dim, dim, 1.0, None)

    def edit(t):
        for n in ("q", "k", "v", "o"):
            t[n][:] = 0.0
        t["q"][0, 0] = 1.0
        t["q"][dim + 1, 0] = 1.0
        t["k"][0, 1] = 1.0
        t["k"][1, 2] = 1.0
        t["v"][0, 3] = 1.0
        t["o"][0, 0] = 1.0
        t["o"][1, dim] = 1.0
        t["sink"][:] = [30.0, -1.5]
    rig = MixerRig("attention", left_params(D, m), dtype, seed=2, edit=edit)
    h = np.zeros((40, D))
    h[:, 0], h[:, 3] = 1.0, 1.0
    h[:, 1], h[:, 2] = 2.0, -3.0
    h[20:, 1], h[30:, 2] = 31.0, 6.0
    want = P.sink_attention(h, rig.plain, m)
    assert want[0, 0] < 1e-9 and 0.1 < want[0, 1] < 0.2 and want[20, 0] > 0.7 and want[39, 1] > 0.95
    got, tail = rig.alone(h), token_by_token(rig, h, 25)
    for a in (got, tail):
        assert np.abs(a - want).max() < (6e-3 if bf else 1e-5)
        assert np.all(np.abs(a[:20, 0]) < 1e-6)


def flag_attention(D, m, dtype, seed, max_tokens=2048):
    """An attention whose scores are decided by two input channels: channel 0 of a row drives one number of its queries,
    channel 1 that of its key.  The taps pass the row itself, so the value of a position is its own key."""
    dim = m["dim"]

    def edit(t):
        for n in ("q", "k"):
            t[n][:, :2] = 0.0
            t[f"{n}.conv"][:] = 0.0
            t[f"{n}.conv"][:, -1] = 1.0
            t[f"{n}.norm"][:] = 1.0
        t["q"][dim - 2::dim, 0] = 4.0
        t["k"][dim - 2::dim, 1] = 4.0
    return MixerRig("attention", att_params(D, m), dtype, seed=seed, edit=edit, max_tokens=max_tokens)


def flag_rows(T, D, bf, looking, flagged, seed=5):
    h = inputs(T, D, seed, bf, 0.25)
    h[:, :2] = 0.0
    h[looking, 0] = 32.0
    h[flagged, 1] = 32.0
    return h


def token_by_token(rig, h, first):
    s = rig.cache.alloc_seq()
    out = [rig.step([s], [h[:first]])[0]] if first else []
    out += [rig.step([s], [h[i:i + 1]])[0] for i in range(first, h.shape[0])]
    rig.cache.free_seq(s)
    rig.cache.check()
    return np.concatenate(out)


FLAG_HEADS = {"64": (2, 1, 64), "128": (2, 1, 128), "96": (2, 2, 96), "48": (2, 1, 48), "20": (2, 1, 20)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size,at", [(5, 70), (64, 64), (65, 100), (33, 127), (100, 130), (72, 191), (1, 63), (40, 0)])
@pytest.mark.parametrize("heads", list(FLAG_HEADS))
def test_a_key_just_inside_and_just_outside_the_window(heads, size, at, dtype):
    """A flagged key at position `at` holds most of the weight of every later row whose window keeps it: the row `size - 1`
    positions later still sees it, the next does not.  The same row times 1.5 has the same normed key and another value:
    the rows that see it change, every other row stays the same bit for bit."""
    nh, nkv, dim = FLAG_HEADS[heads]
    D, bf = 24, dtype == "bfloat16"
    m = att(nh, nkv, dim, 2, 40.0 / dim, size)
    rig = flag_attention(D, m, dtype, 11)
    T = at + size + 6
    h = flag_rows(T, D, bf, slice(None), at, seed=6)
    moved = h.copy()
    moved[at] *= 1.5
    want, other = (P.biased_attention(x, rig.plain, m, 1e-5) for x in (h, moved))
    inside = np.arange(T)
    inside = (inside >= at) & (inside < at + size)
    assert np.abs(other[~inside] - want[~inside]).max() < 1e-6 * np.abs(want).max()
    assert np.abs(other[inside] - want[inside]).max(-1).min() > 0.1 * np.abs(want[at:]).max()

    def portions(x):
        s = rig.cache.alloc_seq()
        cuts = sorted({c for c in (0, max(1, at - 1), at + 1, at + size - 1, at + size, at + size + 2, T) if 0 <= c <= T})
        out = [rig.step([s], [x[a:b]])[0] for a, b in zip(cuts[:-1], cuts[1:])]
        rig.cache.free_seq(s)
        return np.concatenate(out)
    for run in (rig.alone, lambda x: token_by_token(rig, x, at + 2), portions):
        a, b = run(h), run(moved)
        assert err(a, want) < TOL[dtype] and err(b, other) < TOL[dtype]
        assert np.array_equal(a[~inside], b[~inside])
        assert np.all(np.abs(a[inside] - b[inside]).max(-1) > 0.05 * np.abs(want[at:]).max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [0, 640])
@pytest.mark.parametrize("heads", ["64", "128", "48", "20"])
def test_a_far_key_among_hundreds_is_found_in_a_prompt_and_while_decoding(heads, size, dtype):
    """Position 2 carries the key that only the last rows look for: a key lost at a page border, or a split of the key range
    merged wrongly, changes their result.  (Of two heads the second loses 2^-8 a position.)"""
    nh, nkv, dim = FLAG_HEADS[heads]
    D, bf = 32, dtype == "bfloat16"
    m = att(nh, nkv, dim, 2, 40.0 / dim, size)
    rig = flag_attention(D, m, dtype, 6, max_tokens=4096)
    h = flag_rows(638, D, bf, slice(600, None), 2)
    want = P.biased_attention(h, rig.plain, m, 1e-5)
    lost = h.copy()
    lost[2, 1] = 0.0
    assert err(P.biased_attention(lost, rig.plain, m, 1e-5)[600:], want[600:]) > 0.1
    assert err(rig.alone(h), want) < TOL[dtype]
    assert err(token_by_token(rig, h, 598), want) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [64, 128, 48])
def test_a_far_key_beside_a_sink_is_found(dim, dtype):
    D, bf = 32, dtype == "bfloat16"
    m = left(2, 1, dim, dim, 30.0 / dim, dim, 1e30)

    def edit(t):
        for n in ("q", "k", "v"):
            t[n][:, :2] = 0.0
        t["q"][dim // 2 - 1::dim, 0] = 0.125
        t["k"][dim // 2 - 1::dim, 1] = 0.125
        t["sink"][:] = [2.0, -1.0]
    rig = MixerRig("attention", left_params(D, m), dtype, seed=8, edit=edit, max_tokens=4096)
    h = inputs(700, D, 5, bf, 0.25)
    h[:, :2] = 0.0
    h[660:, 0] = 64.0
    h[3, 1] = 64.0
    want = P.sink_attention(h, rig.plain, m)
    lost = h.copy()
    lost[3, 1] = 0.0
    assert err(P.sink_attention(lost, rig.plain, m)[660:], want[660:]) > 0.1
    assert err(rig.alone(h), want) < TOL[dtype]
    assert err(token_by_token(rig, h, 655), want) < TOL[dtype]


# ---- time mixing ------------------------------------------------------------------------------------------------------
def tm_rig(D, heads, d, dtype, seed, eps=1e-5, edit=None):
    return MixerRig("time_mixing", dict(hidden_size=D, num_heads=heads, head_dim=d, norm_eps=eps), dtype, seed=seed, std=0.2, edit=edit)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D,heads,d", [(48, 2, 64), (64, 4, 16), (40, 3, 10), (42, 1, 33), (128, 1, 128), (32, 2, 200), (96, 5, 32)])
def test_time_mixing_alone_whole_in_portions_and_batched(D, heads, d, dtype):
    rig = tm_rig(D, heads, d, dtype, 5)
    m = {"heads": heads, "dim": d}
    whole_portions_and_batches(rig, lambda h: P.time_mixing(h, rig.plain, m, 1e-5), (70, 1, 33), 21, [0, 2, 3, 8, 9, 21],
                               TOL[dtype], dtype == "bfloat16")


def test_every_step_of_the_time_mixing_shows():
    D, m = 32, {"heads": 2, "dim": 16}
    rig = tm_rig(D, 2, 16, "float32", 6)
    h = inputs(50, D, 1, False)
    run = lambda w=rig.plain: P.time_mixing(h, w, m, 1e-5)  # noqa: E731
    want = run()
    assert err(rig.alone(h), want) < H.TOL_F32

    def decays_first(r, k, v, w, u):       # the read-out of a state that has already decayed
        S, o = np.zeros((2, 16, 16)), np.zeros(r.shape)
        for t in range(len(r)):
            kv = k[t][:, :, None] * v[t][:, None, :]
            S = w[t][:, :, None] * S
            o[t] = np.einsum("hij,hi->hj", S + u[:, :, None] * kv, r[t])
            S = S + kv
        return o
    assert err(variant(run, bonus_recurrence=decays_first), want) > 0.02
    assert err(variant(run, row_before=lambda x: np.concatenate([x[:1], x[:-1]])), want) > 0.02     # the first row mixed with itself
    assert err(variant(run, row_before=lambda x: x), want) > 0.02
    assert err(run(dict(rig.plain, u=np.ones((2, 16)))), want) > 0.02
    assert err(variant(run, silu=P.sigmoid), want) > 0.02
    for n in "rkvgw":
        assert err(run(dict(rig.plain, **{f"mu.{n}": rig.plain[f"mu.{n}"][::-1]})), want) > 0.005, n


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_state_lasts_over_hundreds_of_rows_and_is_zero_in_a_slot_used_again(dtype):
    """Channels that hardly decay (w0 = -9): the first row's write is most of what row 400 reads.  The same slot then
    serves another sequence, whose first rows must not see it."""
    D, d, bf = 24, 16, dtype == "bfloat16"

    def edit(t):
        t["w0"][:] = -9.0
        t["w2"][:] = 0.0
        t["u"][:] = 0.0
        for n in "rkvgw":
            t["mu." + n][:] = 0.0
        t["k"][:, 1:] = 0.0
    rig = tm_rig(D, 1, d, dtype, 7, edit=edit)
    m = {"heads": 1, "dim": d}
    h = inputs(400, D, 1, bf)
    h[1:, 0] = 0.0
    h[0, 0] = 4.0
    want = P.time_mixing(h, rig.plain, m, 1e-5)
    gone = h.copy()
    gone[0, 0] = 0.0
    assert np.abs(P.time_mixing(gone, rig.plain, m, 1e-5)[300:]).max() < 1e-9 and np.abs(want[399]).max() > 0.05
    assert err(rig.alone(h), want) < TOL[dtype]
    s = rig.cache.alloc_seq()
    rig.step([s], [h[:50]])
    rig.cache.free_seq(s)
    again = token_by_token(rig, gone[:20], 3)
    assert np.abs(again[2:]).max() < 1e-9
    assert err(token_by_token(rig, h[:120], 90), want[:120]) < TOL[dtype]


@pytest.mark.parametrize("M,C,rank", [(1, 40, 8), (5, 130, 16), (16, 64, 3), (17, 200, 65), (300, 128, 64), (40, 1024, 130)])
def test_decay_of_a_low_rank_pair(M, C, rank):
    low, w2, w0 = inputs(M, rank, 1, False), inputs(rank, C, 2, False, 0.3), inputs(1, C, 3, False)[0]
    out = torch.zeros(M, C, device=DEV)
    wide = dev(inputs(M, rank + 3, 4, False))
    wide[:, :rank] = dev(low)
    K().low_rank_decay(out, wide[:, :rank], dev(w2), dev(w0))
    assert np.abs(host(out) - np.exp(-np.exp(np.tanh(low) @ w2 + w0))).max() < 2e-6


# ---- the state-space layer and two mixers side by side ------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", [(6, 16, 24, 3, 2, 3), (4, 24, 16, 1, 4, 4), (5, 6, 10, 5, 3, 2), (3, 40, 200, 1, 1, 1), (8, 20, 32, 4, 1, 6)])
def test_state_space_alone_whole_in_portions_and_batched(case, dtype):
    m = ssm(*case)
    rig = MixerRig("state_space", mixer_params(48, m, "mamba2"), dtype, seed=5, std=0.2)
    whole_portions_and_batches(rig, lambda h: P.mamba2(h, rig.plain, m, 1e-5), (70, 1, 33), 21, [0, 2, 3, 8, 9, 21],
                               TOL[dtype], dtype == "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", [par(left(4, 2, 64, 64, 0.12, 64), 3, 16, 0.7, 1.3), par(left(3, 1, 20, 12, 0.3, 10, 100.0), 1, 24, None, 0.5),
                               par(left(2, 2, 48, 48, 0.2), 2, 32, 1.5)])
def test_two_mixers_side_by_side(m, dtype):
    rig = MixerRig("parallel_mixers", mixer_params(48, m, "parallel"), dtype, seed=6, std=0.2, hidden_size=48)
    whole_portions_and_batches(rig, lambda h: P.side_by_side(h, rig.plain, m, 1e-5), (70, 1, 33), 21, [0, 2, 3, 8, 9, 21],
                               TOL[dtype], dtype == "bfloat16")


# ---- experts ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows", [1, 3, 17, 130, 700])
@pytest.mark.parametrize("D,f", [(64, moe(6, 2, 48, 32)), (42, moe(5, 5, 30)), (48, moe(12, 1, 64, 16)), (96, moe(9, 4, 24, 20))])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts_on_weighted_rows_and_a_shared_one(rows, D, f, dtype):
    from lastengine_b200.engine.workspace import Workspace
    from lastengine_b200.parts.base import BuildEnv
    from lastengine_b200.registry import FEED_FORWARDS, plan_from_config
    cfg = {"architecture": "Nolapel", "vocab": 8, "width": D, "norm": {"eps": 1e-5},
           "layers": [{"type": "mamba2", "mixer": ssm(1, 4, 4, 1, 1, 1), "mlp": f}]}
    spec = plan_from_config(cfg).layers[0].ffn
    part = FEED_FORWARDS.get(spec.kind)(**spec.params)
    env = BuildEnv(device=torch.device(DEV), dtype=DT[dtype], workspace=Workspace(torch.device(DEV)))
    w = {n: inputs(*s.shape, 10 + i, True) * (0.5 if n == "router" else s.shape[1] ** -0.5) for i, (n, s) in enumerate(part.tensors().items())}
    w = {n: H.bf16_round_np(v) for n, v in w.items()}
    part.load({n: dev(v, torch.float32 if n == "router" else DT[dtype]) for n, v in w.items()}, env)
    h = inputs(rows, D, 5, dtype == "bfloat16")
    start = inputs(rows, D, 6, False)
    out = dev(start)
    part.forward(dev(h, DT[dtype]), out, True, None, env)
    K().check_device_status()
    gap = P.route(h, w, f)[2]
    keep = gap > 1e-5
    assert keep.sum() >= 0.9 * rows
    assert err((host(out) - start.astype(np.float32))[keep], P.expert_mixture(h, w, f)[keep]) < TOL[dtype]


# ---- whole models --------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    from lastengine_b200.weights import write_model_dir
    return {n: write_model_dir(cfg, str(tmp_path_factory.mktemp("n" + n)), seed=81 + i, norm_init="random")
            for i, (n, cfg) in enumerate(ALL.items())}


_tensors, _plain = {}, {}


def tensors_of(name, dirs):
    if name not in _tensors:
        _tensors[name] = P.read_safetensors(os.path.join(dirs[name], "model.safetensors"))
    return _tensors[name]


def plain(name, dirs, tokens):
    """(logits, smallest routing gap of any layer run per position)"""
    key = (name, tuple(tokens))
    if key not in _plain:
        gaps = []
        lg = P.forward(ALL[name], tensors_of(name, dirs), tokens, gaps=gaps)
        _plain[key] = lg, (np.stack(gaps).min(0) if gaps else np.full(len(tokens), np.inf))
    return _plain[key]


def close(got, want, dtype) -> bool:
    """`want` = (logits, routing gaps).  32-bit: every position within the tolerance up to the first whose choice of
    experts rounding may turn.  bfloat16: such choices are no rarity over the layer runs of a looped model, and a turned one
    moves its position and, through the mixers, later ones; over the positions the median error stays within the
    tolerance and nine in ten within three times it."""
    lg, gap = want
    got = host(got) if isinstance(got, torch.Tensor) else np.asarray(got)
    e = np.abs(got - lg).max(-1) / np.abs(lg).max()
    if dtype == "float32":
        near = np.nonzero(gap < 1e-5)[0]
        return bool(np.all(e[: near[0] if len(near) else len(e)] < H.TOL_F32))
    if e.size < 8:
        return bool(np.all(e[gap > 2e-2] < 3 * H.TOL_BF16))
    return bool(np.median(e) < H.TOL_BF16 and np.quantile(e, 0.9) < 3 * H.TOL_BF16)


def part_of(want, a, b=None):
    return want[0][a:b], want[1][a:b]


def reqs_for(name, lengths, seed):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, ALL[name]["vocab"], size=n).tolist() for n in lengths]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ALL))
def test_model_whole_tail_portions_and_batches(name, dtype, dirs):
    from lastengine_b200 import Engine
    eng = Engine.from_pretrained(dirs[name], dtype=dtype, max_tokens=1024, max_seqs=6)
    reqs = reqs_for(name, [150, 3, 70, 1], 40)
    want = [plain(name, dirs, r) for r in reqs]
    for r, w in zip(reqs, want):
        assert close(H.run_whole(eng, r), w, dtype), f"whole, {len(r)} tokens"
    assert close(H.run_tail(eng, reqs[0], tail=90), want[0], dtype)          # decoding across page and window borders
    assert close(H.run_tail(eng, reqs[2], tail=69), want[2], dtype)          # from the first token on
    # a prompt in portions of several sizes, down to two tokens and one
    s = eng.new_sequence()
    outs, at = [], 0
    for n in (2, 1, 2, 59, 1, 64, 3, 18):
        outs.append(H.to_host(eng.step([s], [reqs[0][at:at + n]], [list(range(n))], check=True)))
        at += n
    eng.release(s)
    assert at == 150 and close(torch.cat(outs), want[0], dtype)
    # unequal requests in one batch (prompts of different lengths, then token by token, leaving one by one)
    got = H.run_batch(eng, reqs, [100, 1, 64, 1])
    for g, w, r in zip(got, want, reqs):
        assert close(g, w, dtype), f"batched, {len(r)} tokens"
    # the same again in the slots and pages that were just given back, in another order
    got = H.run_batch(eng, reqs[::-1], [1, 7, 2, 149])
    for g, w in zip(got, want[::-1]):
        assert close(g, w, dtype)
    assert eng.cache.slots.n_held == 0
    eng.cache.check()


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_stream_after_every_layer(name, dirs):
    """The stream after the first 1, 2, ... layers, seen through the final norm and the head: models whose later layers
    are cut off (and the loop with them) against the plain implementation."""
    from lastengine_b200 import Engine
    from lastengine_b200.weights.safetensors_io import SafetensorsFile, save_file
    cfg = ALL[name]
    toks = reqs_for(name, [60], 47)[0]
    src = dirs[name]
    sf = SafetensorsFile(os.path.join(src, "model.safetensors"))
    for n_layers in range(1, len(cfg["layers"])):
        cut = dict(cfg, layers=cfg["layers"][:n_layers])
        if cut.get("loop"):
            cut["loop"] = dict(cut["loop"], start=min(cut["loop"]["start"], n_layers), stop=min(cut["loop"]["stop"], n_layers))
        d = os.path.join(src, f"cut{n_layers}")
        os.makedirs(d, exist_ok=True)
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cut, f)
        keep = {n: sf.tensor(n).clone() for n in sf.names() if not (n[0] == "l" and n[1].isdigit()) or int(n.split(".")[0][1:]) < n_layers}
        save_file(keep, os.path.join(d, "model.safetensors"))
        eng = Engine.from_pretrained(d, dtype="float32", max_tokens=256, max_seqs=2)
        w = P.read_safetensors(os.path.join(d, "model.safetensors"))
        want = P.forward(cut, w, toks)
        assert close(H.run_whole(eng, toks), (want, np.full(60, np.inf)), "float32"), f"after {n_layers} layers"


def test_every_pass_enters_through_the_product_and_has_a_memory_of_its_own(dirs):
    """Passes that skip the product, use the stream alone, the wrong row, or share a memory give other numbers."""
    from lastengine_b200 import Engine
    name = "B"
    cfg, w = ALL[name], tensors_of(name, dirs)
    toks = reqs_for(name, [80], 48)[0]
    want = plain(name, dirs, toks)
    run = lambda: P.forward(cfg, w, toks)  # noqa: E731
    D = cfg["width"]
    first_only = lambda x, x0, t, tensors, f=P.enter_pass: f(x, x0, t, tensors) if t == 0 else x  # noqa: E731
    assert err(variant(run, enter_pass=first_only), want[0]) > 0.02
    assert err(variant(run, enter_pass=lambda x, x0, t, tensors, f=P.enter_pass: f(x, np.zeros_like(x0), t, tensors)), want[0]) > 0.02
    assert err(variant(run, enter_pass=lambda x, x0, t, tensors, f=P.enter_pass: f(x0, x, t, tensors)), want[0]) > 0.02
    assert err(variant(run, enter_pass=lambda x, x0, t, tensors, f=P.enter_pass: f(x, x0, 0, tensors)), want[0]) > 0.005
    eng = Engine.from_pretrained(dirs[name], dtype="float32", max_tokens=512, max_seqs=2)
    assert len(eng.model.blocks) == 4 and len(eng.cache._where) == 1 + 6 and eng.model.stream_matrices["loop.in"].shape == (D, 2 * D)
    assert close(H.run_tail(eng, toks, tail=60), want, "float32")


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_logits_do_not_depend_on_the_cut_or_the_batch_beyond_rounding(name, dirs):
    from lastengine_b200 import Engine
    eng = Engine.from_pretrained(dirs[name], dtype="float32", max_tokens=1024, max_seqs=6)
    reqs = reqs_for(name, [140, 9], 41)
    assert plain(name, dirs, reqs[0])[1].min() > 1e-5
    whole = H.run_whole(eng, reqs[0])
    tail = H.run_tail(eng, reqs[0], tail=80)
    batched = H.run_batch(eng, reqs, [61, 4])[0]
    assert H.rel_err(tail, whole) < 1e-5 and H.rel_err(batched, whole) < 1e-5


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("D", "float32"), ("B", "bfloat16"), ("C", "float32"), ("E", "bfloat16")])
def test_long_decoding_from_a_short_prompt(name, dtype, dirs):
    """Several windows pass while decoding; pages behind them are given back on the way."""
    from lastengine_b200 import Engine
    eng = Engine.from_pretrained(dirs[name], dtype=dtype, max_tokens=512, max_seqs=2)
    r = reqs_for(name, [330], 42)[0]
    got = H.run_tail(eng, r, tail=328)
    assert close(got, plain(name, dirs, r), dtype)
    eng.cache.check()


@pytest.mark.parametrize("seed", list(range(401, 415)))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layer order, loops, sizes and windows drawn at random: whole prompts, a tail token by token and an unequal batch in
    32-bit against the plain implementation, every position held; bfloat16 over the positions."""
    from lastengine_b200 import Engine
    from lastengine_b200.weights import write_model_dir
    rng = np.random.default_rng(seed)
    cfg = random_config(rng)
    d = write_model_dir(cfg, str(tmp_path / "m"), seed=seed, norm_init="random")
    w = P.read_safetensors(os.path.join(d, "model.safetensors"))
    reqs = [rng.integers(0, cfg["vocab"], size=n).tolist() for n in (210, 40)]
    want = []
    for r in reqs:
        gaps = []
        lg = P.forward(cfg, w, r, gaps=gaps)
        want.append((lg, np.stack(gaps).min(0) if gaps else np.full(len(r), np.inf)))
    eng = Engine.from_pretrained(d, dtype="float32", max_tokens=1024, max_seqs=4)
    for r, wv in zip(reqs, want):
        assert close(H.run_whole(eng, r), wv, "float32"), cfg
    assert close(H.run_tail(eng, reqs[0], tail=90), want[0], "float32"), cfg
    for g, wv in zip(H.run_batch(eng, reqs, [130, 9]), want):
        assert close(g, wv, "float32"), cfg
    eng.cache.check()
    eng16 = Engine.from_pretrained(d, dtype="bfloat16", max_tokens=1024, max_seqs=4)
    for got in (H.run_whole(eng16, reqs[0]), H.run_tail(eng16, reqs[0], tail=90)):
        e = np.abs(host(got) - want[0][0]).max(-1) / np.abs(want[0][0]).max()
        assert np.median(e) < H.TOL_BF16, cfg


def test_a_step_longer_than_a_pass_runs_in_pieces(dirs):
    """A prompt step of more rows than a pass takes is cut where the pass ends: the last token, the last row, the taps and
    the states go on from piece to piece."""
    from lastengine_b200 import Engine
    reqs = reqs_for("A", [150, 40], 49)
    eng = Engine.from_pretrained(dirs["A"], dtype="float32", max_tokens=512, max_seqs=4, max_batch_tokens=47)
    seqs = [eng.new_sequence() for _ in reqs]
    got = H.to_host(eng.step(seqs, reqs, [list(range(len(r))) for r in reqs]))
    eng.release(seqs)
    assert close(got[:150], plain("A", dirs, reqs[0]), "float32") and close(got[150:], plain("A", dirs, reqs[1]), "float32")
    eng.cache.check()


def plain_greedy(name, dirs, prompt, n):
    """Greedy tokens of the plain implementation, and per token the gap between the two best logits (0 where a choice of
    experts on the way is close)."""
    toks, out, margins = list(prompt), [], []
    for _ in range(n):
        lg, gap = plain(name, dirs, toks)
        top = np.sort(lg[-1])[-2:]
        margins.append((float((top[1] - top[0]) / np.abs(lg[-1]).max()), float(gap.min())))
        out.append(int(np.argmax(lg[-1])))
        toks.append(out[-1])
    return out, margins


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "bfloat16"), ("B", "float32"), ("C", "float32"), ("D", "float32"), ("E", "bfloat16")])
def test_greedy_generation_through_the_entry_point(name, dtype, graphs, dirs):
    from lastengine_b200 import Engine, SamplingParams
    eng = Engine.from_pretrained(dirs[name], dtype=dtype, max_tokens=1024, use_graphs=graphs)
    prompts = reqs_for(name, [5, 1, 38, 66], 43)
    steps = 10
    res = eng.generate(prompts, SamplingParams(temperature=0.0), max_new_tokens=steps, stop_token_ids=[])
    compared = 0
    for p, got in zip(prompts, res.tokens):
        want, margins = plain_greedy(name, dirs, p, steps)
        assert len(got) == steps
        for i in range(steps):
            if margins[i][0] < (2 if dtype == "float32" else 4) * TOL[dtype] or margins[i][1] < (1e-5 if dtype == "float32" else 5e-3):
                break
            assert got[i] == want[i], f"{name} {dtype}: prompt of {len(p)}, token {i}"
            compared += 1
    assert compared >= (steps * len(prompts) // 2 if dtype == "float32" else 2)
    assert eng.cache.slots.n_held == 0
    eng.cache.check()


def test_graphs_and_plain_steps_generate_the_same_over_several_windows(dirs):
    """Replayed steps take their tokens on the device, one step ahead: the pair's previous token and the carried rows are the
    ones a step by step run has."""
    from lastengine_b200 import Engine, SamplingParams
    for name in ("A", "E"):
        out = []
        for graphs in (True, False):
            eng = Engine.from_pretrained(dirs[name], dtype="float32", max_tokens=1024, use_graphs=graphs)
            res = eng.generate(reqs_for(name, [30, 61, 2], 44), SamplingParams(temperature=0.0), max_new_tokens=150, stop_token_ids=[])
            out.append([list(t) for t in res.tokens])
            eng.cache.check()
        assert out[0] == out[1]


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "bfloat16"), ("D", "float32")])
def test_a_sequence_written_out_and_read_back_goes_on_where_it_stood(name, dtype, dirs):
    """The last token, keys, taps and states go out as bytes and come back into another slot and other pages."""
    from lastengine_b200 import Engine
    eng = Engine.from_pretrained(dirs[name], dtype=dtype, max_tokens=768, max_seqs=4)
    r = reqs_for(name, [120], 44)[0]
    s = eng.new_sequence()
    eng.step([s], [r[:100]], None)
    data = eng.export_sequence(s)
    a = H.to_host(eng.step([s], [r[100:]], [list(range(20))]))
    other = eng.new_sequence()
    eng.step([other], [r[:5]], None)
    t = eng.import_sequence(data)
    assert t != s and eng.length(t) == 100
    b = H.to_host(eng.step([t], [r[100:]], [list(range(20))]))
    eng.release([s, other, t])
    assert H.rel_err(b, a) < 1e-6
    eng.cache.check()


def test_replay_program_with_a_cache_sized_to_the_tokens_alone(dirs, tmp_path):
    """bin/trace_run with --max-tokens equal to the tokens the live requests hold: three unequal requests start
    together (the shortest with one token), go on token by token and leave one by one."""
    name = "A"
    reqs = dict(zip("xyz", reqs_for(name, [12, 95, 3], 45)))
    first = {"x": 9, "y": 70, "z": 1}
    steps = [{"step": 0, "entries": [{"id": r, "tokens": reqs[r][:first[r]], "want": list(range(first[r]))} for r in "xyz"],
              "end": []}]
    fed, live, n = dict(first), ["x", "y", "z"], 1
    while live:
        ent = [{"id": r, "tokens": [reqs[r][fed[r]]], "want": [0]} for r in live]
        for r in live:
            fed[r] += 1
        ended = [r for r in live if fed[r] >= len(reqs[r])]
        steps.append({"step": n, "entries": ent, "end": ended})
        live = [r for r in live if r not in ended]
        n += 1
    out = str(tmp_path / "out")
    p = subprocess.run([sys.executable, os.path.join(H.ROOT, "bin", "trace_run"), "--model", dirs[name], "--dtype", "float32",
                        "--out", out, "--max-tokens", str(sum(len(t) for t in reqs.values()))],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(n)]
    V = ALL[name]["vocab"]
    got = {r: [] for r in reqs}
    for st in steps:
        lg = np.fromfile(os.path.join(out, f"{st['step']}.f32"), dtype="<f4").reshape(-1, V)
        at = 0
        for e in st["entries"]:
            got[e["id"]].append(lg[at:at + len(e["want"])])
            at += len(e["want"])
        assert at == lg.shape[0]
    for r, t in reqs.items():
        assert close(np.concatenate(got[r]), plain(name, dirs, t), "float32"), r


def test_command_line_generates_and_inspects(dirs):
    exe = os.path.join(H.ROOT, "bin", "lastengine")
    d = dirs["A"]
    base = [sys.executable, exe, "generate", "--model", d, "--prompt-ids", "1,2,3", "--prompt-ids", "9 8 7 6 5", "--max-new-tokens", "6",
            "--stop-token-id", "199"]
    p = subprocess.run(base + ["--dtype", "float32", "--temperature", "0"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-1500:]
    rows = [json.loads(l) for l in p.stdout.splitlines()]
    assert len(rows) == 2 and all(1 <= len(r["tokens"]) <= 6 for r in rows)
    want, margins = plain_greedy("A", dirs, [1, 2, 3], 1)
    if margins[0][0] > 1e-4 and margins[0][1] > 1e-5:
        assert rows[0]["tokens"][0] == want[0]
    sampled = [subprocess.run(base + ["--temperature", "0.9", "--top-k", "20", "--seed", "5"], capture_output=True, text=True, timeout=600)
               for _ in range(2)]
    assert sampled[0].returncode == 0, sampled[0].stderr[-1500:]
    assert sampled[0].stdout == sampled[1].stdout
    p2 = subprocess.run([sys.executable, exe, "inspect", d], capture_output=True, text=True, timeout=600)
    assert p2.returncode == 0, p2.stderr[-1500:]
    assert "Nolapel" in p2.stdout and "parallel_mixers (attention | time_mixing)" in p2.stdout and "state_space" in p2.stdout
