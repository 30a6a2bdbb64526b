"""The Zafilix decoder on the GPU against the plain implementation (tests/plain_zafilix.py): every mechanism alone, then
whole models: prompts whole, in portions and token by token, unequal batches, slots and pages used again, keys far
away, at page borders and at the edges of chunks and windows, long decoding, and greedy generation through the entry
point."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import harness as H
import plain_zafilix as P
from harness import MixerRig, max_err as err, random_rows as inputs, whole_portions_and_batches
from zafilix_configs import ALL, att, lat, random_config

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": H.TOL_F32, "bfloat16": H.TOL_BF16}
NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "gate": "g", "q_norm": "q.norm", "k_norm": "k.norm"}


def K():
    from lastengine_b200.ops import kernels
    return kernels


def rope(rot, style):
    from lastengine_b200.parts.base import PartSpec
    if not rot or not rot.get("dims"):
        return PartSpec("none")
    return PartSpec("rope", {"rope_dim": rot["dims"], "theta": rot["base"], "style": style,
                             "scaling_factor": (rot.get("scaling") or {}).get("factor", 1.0)})


def att_params(D, m, eps=1e-5, **more):
    return dict(hidden_size=D, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
                norm_eps=eps, qk_norm="row", position=rope(m.get("rot"), "adjacent"), scale=m["scale"],
                chunk=(m.get("mask") or {}).get("size", 0), output_gate="numbers", wide_weights=True, names=NAMES, **more)


def lat_params(D, m, eps=1e-5, **more):
    return dict(hidden_size=D, num_heads=m["heads"], head_dim=m["dim"], rope_dim=m["rot_dim"], v_head_dim=m["vdim"], q_rank=0,
                kv_rank=m["kv_rank"], norm_eps=eps, scale=m["scale"], position=rope(m.get("rot"), "neox"),
                window=(m.get("mask") or {}).get("size", 0), wide_weights=True, **more)


# ---- chunked attention ------------------------------------------------------------------------------------
ATT_CASES = [  # heads, kv heads, dim, vdim, scale, rotated, base, factor, chunk
    (4, 2, 64, 64, 0.12, 64, 10000.0, 3.0, 40),       # the tcgen05 prompt kernel, the decode kernel that prepares its rows
    (8, 1, 64, 64, 0.12, 64, 500.0, 1.0, 100),
    (3, 3, 64, 64, 0.12, 20, 10000.0, 2.0, 64),       # a partial rotation: the rows are prepared by a launch of their own
    (6, 2, 128, 128, 0.08, 128, 1e6, 1.0, 70),
    (4, 4, 96, 96, 0.1, 96, 1e5, 2.0, 33),
    (6, 1, 32, 32, 0.2, 8, 300.0, 4.0, 150),
    (4, 2, 64, 32, 0.12, 64, 10000.0, 1.5, 90),       # cached at the wider of the two
    (2, 1, 48, 128, 0.15, 24, 2000.0, 1.0, 21),
    (5, 5, 12, 20, 0.3, 0, 1.0, 1.0, 1),              # off the 16-byte grid, a chunk of one position
    (3, 1, 22, 10, 0.25, 10, 5000.0, 2.5, 33),
    (2, 2, 24, 24, 0.2, 24, 100.0, 1.0, 0),           # no chunks
    (12, 3, 200, 40, 0.07, 100, 10000.0, 8.0, 128),
]


def att_of(heads, kv, dim, vdim, scale, rot, base, factor, size):
    return att(heads, kv, dim, vdim, scale, rot if rot else None, base, factor, size)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ATT_CASES)
def test_attention_alone_whole_in_portions_and_batched(case, dtype):
    m = att_of(*case)
    rig = MixerRig("attention", att_params(48, m), dtype, seed=3)
    whole_portions_and_batches(rig, lambda h: P.chunked_attention(h, rig.plain, m, 1e-5), (150, 1, 67), 21,
                               [0, 2, 3, 8, 9, 21], TOL[dtype], dtype == "bfloat16")


def test_the_norm_runs_over_the_whole_row_and_the_gate_over_every_number():
    """Head 0's queries and keys are much larger than the others': a norm over every head, one factor of a head's gate
    for all its numbers, split-half pairs, or positions that are not scaled give another result."""
    m = att(4, 2, 16, 16, 0.4, 16, 100.0, 2.0, 30)

    def edit(t):
        t["q"][:16] *= 5.0
        t["k"][:16] *= 5.0
    rig = MixerRig("attention", att_params(32, m), "float32", seed=4, edit=edit)
    h = inputs(70, 32, 1, False)
    want = P.chunked_attention(h, rig.plain, m, 1e-5)
    assert err(rig.alone(h), want) < H.TOL_F32
    w = rig.plain

    def variant(**swap):
        saved = {n: getattr(P, n) for n in swap}
        try:
            for n, f in swap.items():
                setattr(P, n, f)
            return P.chunked_attention(h, w, m, 1e-5)
        finally:
            for n, f in saved.items():
                setattr(P, n, f)
    by_head = variant(over_rms=lambda x, eps: (lambda y: (y / np.sqrt((y * y).mean(-1, keepdims=True) + eps)).reshape(x.shape))
                      (x.reshape(x.shape[0], -1, 16)))
    assert err(by_head, want) > 0.02
    assert err(variant(rotate_neighbours=P.rotate_halves), want) > 0.02
    assert err(variant(seen_in_chunk=P.seen_in_window), want) > 0.02
    unscaled = dict(m, rot={"dims": 16, "base": 100.0})
    assert err(P.chunked_attention(h, w, unscaled, 1e-5), want) > 0.02
    one_gate = dict(w, g=np.repeat(w["g"][::16], 16, axis=0))
    assert err(P.chunked_attention(h, one_gate, m, 1e-5), want) > 0.02


def flag_attention(D, m, dtype, seed, max_tokens=2048):
    """An attention whose scores are decided by two input channels: channel 0 of a row drives the last even number of its
    queries, channel 1 that of its key, both in a pair that hardly turns.  A key with a large channel 1 takes all the
    weight of every row that sees it and has a large channel 0."""
    dim = m["dim"]

    def edit(t):
        for n in ("q", "k"):
            t[n][:, :2] = 0.0
        t["q"][dim - 2::dim, 0] = 4.0
        t["k"][dim - 2::dim, 1] = 4.0
        t["v"][:, :2] = 0.0
        t["g"][:, :2] = 0.0
        t["q.norm"][:] = 1.0
        t["k.norm"][:] = 1.0
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


FLAG_HEADS = {   # the kernels a head size runs: tcgen05 / mma prompts, the two decode kernels, the general kernel
    "64": (4, 2, 64, 64), "128": (2, 1, 128, 128), "96": (2, 2, 96, 96), "64-narrow-values": (2, 1, 64, 32), "20": (2, 1, 20, 20)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size,at", [(5, 70), (64, 64), (65, 129), (33, 98), (128, 130), (96, 95), (40, 79), (7, 63)])
@pytest.mark.parametrize("heads", list(FLAG_HEADS))
def test_a_key_is_seen_to_the_end_of_its_chunk_and_not_beyond(heads, size, at, dtype):
    """A flagged key at position `at` holds nearly all the weight of every later row of its chunk, and none of the
    next chunk's rows: in whole prompts, in portions cut next to the border and token by token.  With another value
    under the flag the rows of its chunk change, and every other row stays the same bit for bit."""
    nh, nkv, dim, vdim = FLAG_HEADS[heads]
    D, bf = 24, dtype == "bfloat16"
    m = att(nh, nkv, dim, vdim, 0.3, dim, 1e30, None, size)
    rig = flag_attention(D, m, dtype, 7)
    end = (at // size + 1) * size           # the next chunk's first position
    T = end + 9
    h = flag_rows(T, D, bf, slice(None), at)
    moved = h.copy()
    moved[at, 2:] += 2.0
    want, other = (P.chunked_attention(x, rig.plain, m, 1e-5) for x in (h, moved))
    inside = np.arange(T)
    inside = (inside >= at) & (inside < end)
    assert np.abs(other[~inside] - want[~inside]).max() < 1e-12
    assert np.abs(other[inside] - want[inside]).max(-1).min() > 0.05 * np.abs(want).max()
    runs = [lambda x: rig.alone(x), lambda x: token_by_token(rig, x, max(1, end - 12))]

    def portions(x):
        s = rig.cache.alloc_seq()
        cuts = sorted({0, max(1, at - 1), at + 1, end - 1, end, end + 2, T})
        out = [rig.step([s], [x[a:b]])[0] for a, b in zip(cuts[:-1], cuts[1:])]
        rig.cache.free_seq(s)
        return np.concatenate(out)
    runs.append(portions)
    for run in runs:
        a, b = run(h), run(moved)
        assert err(a, want) < TOL[dtype] and err(b, other) < TOL[dtype]
        assert np.array_equal(a[~inside], b[~inside])
        assert np.all(np.abs(a[inside] - b[inside]).max(-1) > 0.03 * np.abs(want).max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [0, 640])
@pytest.mark.parametrize("heads", ["64", "128", "20"])
def test_a_far_key_among_hundreds_is_found_in_a_prompt_and_while_decoding(heads, size, dtype):
    """Position 2 carries the key that only the last rows look for, so those rows put nearly all their weight 600
    positions back: a key lost at a page border, or a split of the key range merged wrongly, changes their result."""
    nh, nkv, dim, vdim = FLAG_HEADS[heads]
    D, bf = 32, dtype == "bfloat16"
    m = att(nh, nkv, dim, vdim, 0.3, dim, 1e30, None, size)
    rig = flag_attention(D, m, dtype, 6, max_tokens=4096)
    h = flag_rows(638, D, bf, slice(600, None), 2)
    want = P.chunked_attention(h, rig.plain, m, 1e-5)
    lost = P.chunked_attention(np.delete(h, 2, 0), rig.plain, m, 1e-5)
    assert err(lost[599:], want[600:]) > 0.1
    assert err(rig.alone(h), want) < TOL[dtype]
    assert err(token_by_token(rig, h, 598), want) < TOL[dtype]


def test_the_softmax_weights_keep_sixteen_bits_in_the_bfloat16_kernels():
    """Two keys share a row's weight as 257 : 255 (half a bfloat16 step from even) and their values are +1 and -1 times
    the same vector: with weights rounded to eight bits the difference of the two would be lost or doubled.  The gate is
    one half everywhere and the output projection keeps the numbers apart."""
    for dim, kernel in ((64, "tcgen05 and decode"), (96, "mma")):
        D = 16
        m = att(1, 1, dim, dim, 1.0, dim, 1e30, None, 0)

        def edit(t):
            for n in ("q", "k", "v", "g", "o"):
                t[n][:] = 0.0
            t["q"][dim - 2, 0] = 1.0
            t["k"][dim - 2, 1] = 1.0
            t["k"][dim - 4, 2] = 1.0
            t["v"][0, 3] = 1.0
            t["o"][0, 0] = 1.0
            t["q.norm"][:] = 1.0 / dim ** 0.5      # a row with one number comes out of the norm as that number's sign
            t["k.norm"][:] = 1.0 / dim ** 0.5
        rig = MixerRig("attention", att_params(D, m), "bfloat16", seed=2, edit=edit)
        h = np.zeros((40, D))
        h[:, 0] = 1.0
        h[:, 1] = -20.0                            # the filler keys
        h[4, 1:4] = [1.0, 32.0, 1.0]               # a key whose share of the row in the query's direction is 1/32
        h[5, 1:4] = [1.0, 64.0, -1.0]              # and 1/64
        want = P.chunked_attention(h, rig.plain, m, 1e-5)
        got = rig.alone(h)
        dec = token_by_token(rig, h, 30)
        assert err(got[6:], want[6:]) < 6e-3, kernel
        assert err(dec[6:], want[6:]) < 6e-3, kernel


@pytest.mark.parametrize("nh,nkv,hd,hin,vin,rot,neox", [
    (4, 2, 64, 64, 64, 64, False), (4, 2, 64, 64, 64, 24, False), (3, 1, 128, 128, 128, 128, False), (40, 8, 128, 128, 128, 128, False),
    (4, 2, 64, 64, 64, 64, True), (5, 5, 12, 12, 20, 8, False), (2, 2, 64, 48, 64, 48, False), (2, 1, 20, 20, 6, 0, False),
    (100, 2, 96, 96, 96, 96, False), (3, 3, 10, 7, 9, 6, True)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_rows_are_normed_turned_and_stored(nh, nkv, hd, hin, vin, rot, neox, dtype):
    """The launch alone: norm of whole rows, both pairings, heads stored wider than they come, every path of the kernel;
    keys and values land at their positions' places in the pages, a padding sequence's row nowhere."""
    from lastengine_b200.engine.batch import BatchBuilder
    dt, bf, page, vd = DT[dtype], dtype == "bfloat16", 64, max(hd, vin) if hin != hd else vin
    lens, pos0, slots = [70, 1, 3], [5, 130, 0], [0, 1, -1]
    table = np.array([[3, 1, -1], [7, 5, 2], [-1, -1, -1]], dtype=np.int32)
    b = BatchBuilder(torch.device(DEV)).build(slots, [[0] * n for n in lens], pos0, [], {0: table})
    M = sum(lens)
    C = (nh + nkv) * hin + nkv * vin
    C += -C % 8                                                   # rows on the 16-byte grid, as a gate behind them leaves them
    x = inputs(M, C, 1, bf, 2.0)
    wq, wk = 1 + 0.2 * inputs(1, nh * hin, 2, False)[0], 1 + 0.2 * inputs(1, nkv * hin, 3, False)[0]
    proj = torch.from_numpy(x).to(DEV, dt)
    kp = torch.full((8, nkv, page, hd), 9.0, dtype=dt, device=DEV)
    vp = torch.full((8, nkv, vd, page), 9.0, dtype=dt, device=DEV)
    q = torch.zeros(M, nh * hd, dtype=dt, device=DEV)
    freq = None
    if rot:
        freq = (100.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)).float().to(DEV)
    K().qk_row_norm_rope_store(q, proj[:, :nh * hin], proj[:, nh * hin:(nh + nkv) * hin],
                               proj[:, (nh + nkv) * hin:(nh + nkv) * hin + nkv * vin], kp, vp, b.tables[0], b,
                               torch.from_numpy(wq).float().to(DEV), torch.from_numpy(wk).float().to(DEV), 1e-3, freq, rot, neox,
                               nh, nkv, hd, page, vd=vd, hd_in=hin, vd_in=vin)
    pos = np.concatenate([np.arange(p, p + n) for p, n in zip(pos0, lens)])
    turn = P.rotate_halves if neox else P.rotate_neighbours
    angle = P.angles(pos, rot, 100.0) if rot else np.zeros((M, 0))

    def rows(cols, w, heads):
        y = (P.over_rms(cols, 1e-3) * w).reshape(M, heads, hin)
        y = turn(y, angle) if rot else y
        return np.pad(y, ((0, 0), (0, 0), (0, hd - hin)))
    tol = 2e-5 if not bf else 8e-3
    assert err(q.double().cpu().numpy(), rows(x[:, :nh * hin], wq, nh).reshape(M, -1)) < tol
    kw, vw = rows(x[:, nh * hin:(nh + nkv) * hin], wk, nkv), x[:, (nh + nkv) * hin:(nh + nkv) * hin + nkv * vin].reshape(M, nkv, vin)
    kd, vdv = kp.double().cpu().numpy(), vp.double().cpu().numpy()
    written = np.zeros((8, page), dtype=bool)
    for i in range(lens[0] + lens[1]):
        s = 0 if i < lens[0] else 1
        pg = table[s, pos[i] // page]
        written[pg, pos[i] % page] = True
        assert np.abs(kd[pg, :, pos[i] % page] - kw[i]).max() < tol * np.abs(kw).max()
        assert np.abs(vdv[pg, :, :vin, pos[i] % page] - vw[i]).max() < 1e-6 * np.abs(vw).max()
        assert np.all(vdv[pg, :, vin:, pos[i] % page] == 0)
    assert np.all(kd.transpose(0, 2, 1, 3)[~written] == 9.0) and np.all(vdv.transpose(0, 3, 1, 2)[~written] == 9.0)


# ---- latent attention in a window ------------------------------------------------------------------------------
LAT_CASES = [  # heads, dim, rot_dim, vdim, rank, scale, base, window, rotated dims, factor
    (5, 24, 16, 40, 64, 0.15, 5000.0, 70, 16, None),      # sizes of the tensor-core kernel
    (2, 32, 32, 64, 128, 0.2, 20000.0, 9, 32, 2.0),
    (8, 64, 64, 64, 256, 0.1, 1e5, 0, 64, None),
    (3, 16, 48, 24, 288, 0.2, 700.0, 65, 20, 2.0),        # tiles of 32 cached rows, a part that passes unturned
    (70, 8, 16, 8, 32, 0.3, 100.0, 33, 16, None),         # more heads than a block takes
    (2, 16, 256, 16, 256, 0.1, 1e4, 40, 256, None),       # rows too wide for tiles of 64
    (3, 10, 6, 14, 20, 0.3, 100.0, 1, 6, None),           # off the 16-byte grid, a window of one position
    (2, 18, 4, 9, 33, 0.22, 900.0, 50, 4, 3.0),
    (4, 16, 0, 16, 96, 0.3, 1.0, 64, 0, None),            # nothing rotated
]


def lat_of(heads, dim, rd, vdim, rank, scale, base, size, dims, factor):
    return lat(heads, dim, rd, vdim, rank, scale, base, size, rot_dims=dims, factor=factor)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", LAT_CASES)
def test_latent_attention_alone_whole_in_portions_and_batched(case, dtype):
    m = lat_of(*case)
    rig = MixerRig("latent_attention", lat_params(48, m), dtype, seed=8, std=0.2)
    whole_portions_and_batches(rig, lambda h: P.latent_attention(h, rig.plain, m, 1e-5), (150, 1, 67), 21,
                               [0, 2, 3, 8, 9, 21], TOL[dtype], dtype == "bfloat16")


@pytest.mark.parametrize("case", [c for c in LAT_CASES if c[4] % 32 == 0])
def test_tensor_core_latent_attention_against_the_general_kernel(case):
    m = lat_of(*case)
    h = inputs(200, 48, 9, True)
    outs = {}
    for mma in (True, False):
        K().set_latent_mma(mma)
        try:
            rig = MixerRig("latent_attention", lat_params(48, m), "bfloat16", seed=8, std=0.2)
            outs[mma] = np.concatenate([rig.alone(h), token_by_token(rig, h, 170)])
        finally:
            K().set_latent_mma(True)
    want = P.latent_attention(h, rig.plain, m, 1e-5)
    assert err(outs[True], outs[False]) < H.TOL_BF16 / 2 and err(outs[True], np.concatenate([want, want])) < H.TOL_BF16


def flag_latent(D, m, dtype, seed, max_tokens=2048):
    """A latent attention whose scores are decided by two input channels, as flag_attention: channel 1 of a row is the
    latent's first number, which alone makes the first number of every head's key; channel 0 that of the queries."""
    dim, rd = m["dim"], m["rot_dim"]

    def edit(t):
        t["q"][:, :2] = 0.0
        t["q"][::dim + rd, :] = 0.0
        t["q"][::dim + rd, 0] = 0.25
        t["dkv"][:, :2] = 0.0
        t["dkv"][0, :] = 0.0
        t["dkv"][0, 1] = 1.0
        t["uk"][:, 0] = 0.0
        t["uk"][::dim, 0] = 1.0
        t["uv"][:, 0] = 0.0
        t["dkv.norm"][:] = 1.0
    # keys and values of about unit size whatever the latent's: larger scores would turn bfloat16 rounding into other weights
    return MixerRig("latent_attention", lat_params(D, m), dtype, seed=seed, std=min(0.3, 2.0 * m["kv_rank"] ** -0.5), edit=edit,
                    max_tokens=max_tokens)


FLAG_LATENTS = {"64": (2, 16, 16, 16, 64), "256": (3, 32, 32, 16, 256), "320": (2, 16, 16, 16, 320), "36": (2, 12, 6, 10, 36)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size,at", [(5, 70), (64, 64), (65, 100), (33, 127), (128, 130), (72, 191), (1, 63)])
@pytest.mark.parametrize("sizes", list(FLAG_LATENTS))
def test_a_latent_row_just_inside_and_just_outside_the_window(sizes, size, at, dtype):
    """A flagged row at position `at` holds the weight of every later row whose window keeps it: the row `size - 1`
    positions later still sees it, the next does not.  Whole prompts and token by token (where the cache gives pages
    back as the window moves on); rows that do not see it stay the same bit for bit when its value changes."""
    H_, dim, rd, vdim, rank = FLAG_LATENTS[sizes]
    D, bf = 24, dtype == "bfloat16"
    m = lat(H_, dim, rd, vdim, rank, 0.3, 100.0, size)
    rig = flag_latent(D, m, dtype, 11)
    T = at + size + 6
    h = flag_rows(T, D, bf, slice(None), at, seed=6)
    moved = h.copy()
    moved[at, 2:] *= -4.0
    want, other = (P.latent_attention(x, rig.plain, m, 1e-5) for x in (h, moved))
    inside = np.arange(T)
    inside = (inside >= at) & (inside < at + size)
    assert np.abs(other[~inside] - want[~inside]).max() < 1e-12
    change = np.abs(other[inside] - want[inside]).max(-1).min()
    assert change > 1e-3 * np.abs(want).max()
    for run in (lambda x: rig.alone(x), lambda x: token_by_token(rig, x, at + 2)):
        a, b = run(h), run(moved)
        assert err(a, want) < TOL[dtype] and err(b, other) < TOL[dtype]
        assert np.array_equal(a[~inside], b[~inside])
        assert np.all(np.abs(a[inside] - b[inside]).max(-1) > 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", ["64", "320", "36"])
@pytest.mark.parametrize("size", [0, 700])
def test_a_far_latent_row_is_found_in_a_prompt_and_while_decoding(sizes, size, dtype):
    H_, dim, rd, vdim, rank = FLAG_LATENTS[sizes]
    D, bf = 32, dtype == "bfloat16"
    m = lat(H_, dim, rd, vdim, rank, 0.3, 1e4, size)
    rig = flag_latent(D, m, dtype, 12, max_tokens=4096)
    h = flag_rows(638, D, bf, slice(600, None), 2, seed=7)
    want = P.latent_attention(h, rig.plain, m, 1e-5)
    lost = P.latent_attention(np.delete(h, 2, 0), rig.plain, m, 1e-5)
    assert err(lost[599:], want[600:]) > 0.1
    assert err(rig.alone(h), want) < TOL[dtype]
    assert err(token_by_token(rig, h, 598), want) < TOL[dtype]


def test_latent_rows_in_chunks_and_neighbouring_pairs():
    """The part's options beyond this design: chunks instead of a window, and neighbouring pairs without a query latent."""
    m = lat(3, 16, 16, 24, 64, 0.2, 300.0, 0)
    for dtype in ("float32", "bfloat16"):
        params = dict(lat_params(40, m), window=0, chunk=37, position=rope(m["rot"], "adjacent"))
        rig = MixerRig("latent_attention", params, dtype, seed=13, std=0.2)
        saved = P.seen_in_window, P.rotate_halves
        P.seen_in_window, P.rotate_halves = (lambda T, size: P.seen_in_chunk(T, 37)), P.rotate_neighbours
        try:
            whole_portions_and_batches(rig, lambda h: P.latent_attention(h, rig.plain, m, 1e-5), (100, 1, 67), 21,
                                       [0, 2, 3, 8, 9, 21], TOL[dtype], dtype == "bfloat16")
        finally:
            P.seen_in_window, P.rotate_halves = saved


# ---- feed-forward, sums, head -----------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,D,F", [(1, 64, 48), (5, 42, 30), (16, 96, 160), (40, 128, 256), (100, 64, 4096), (128, 256, 2048), (300, 64, 96),
                                      (200, 4096, 512), (700, 512, 1024), (1100, 256, 4096)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_squared_relu_in_the_epilogue_of_every_product(rows, D, F, dtype):
    """Rows from one to over a thousand reach the weight stream, the sliced and the tiled tensor-core products and the
    one on pairs of SMs, each of which applies the activation where it stores."""
    from lastengine_b200.engine.workspace import Workspace
    from lastengine_b200.parts.base import BuildEnv
    from lastengine_b200.registry import FEED_FORWARDS
    if dtype == "float32" and rows * D * F > 5e8:
        pytest.skip("the 32-bit path has one product kernel; the small sizes cover it")
    bf = dtype == "bfloat16"
    part = FEED_FORWARDS.get("dense")(hidden_size=D, intermediate_size=F, activation="relu_squared")
    env = BuildEnv(device=torch.device(DEV), dtype=DT[dtype], workspace=Workspace(torch.device(DEV)))
    w = {n: H.bf16_round_np(inputs(s.shape[0], s.shape[1], i, True) * s.shape[1] ** -0.5) for i, (n, s) in enumerate(part.tensors().items())}
    part.load({n: torch.from_numpy(v).to(DEV, DT[dtype]) for n, v in w.items()}, env)
    h = inputs(rows, D, 5, bf)
    out = torch.zeros(rows, D, dtype=torch.float32, device=DEV)
    with K().KernelTimer() as timer:
        part.forward(torch.from_numpy(h).to(DEV, DT[dtype]), out, False, None, env)
    K().check_device_status()
    assert ("leb_activation" in timer.summary()) == (not bf or D % 8 != 0)
    assert err(out.double().cpu().numpy(), P.squared_relu_ff(h, w)) < TOL[dtype]


@pytest.mark.parametrize("act", ["gelu", "relu_squared", "gelu_tanh", "silu"])
@pytest.mark.parametrize("rows,Kd,N", [(3, 64, 96), (50, 128, 256), (200, 4096, 512), (400, 64, 640), (1100, 256, 4096)])
def test_an_activation_in_a_storing_epilogue_gives_the_launch_s_numbers(act, rows, Kd, N):
    kk = K()
    x = torch.from_numpy(inputs(rows, Kd, 1, True)).to(DEV, torch.bfloat16)
    w = torch.from_numpy(inputs(N, Kd, 2, True, Kd ** -0.5)).to(DEV, torch.bfloat16)
    a, b = torch.empty(rows, N, dtype=torch.bfloat16, device=DEV), torch.empty(rows, N, dtype=torch.bfloat16, device=DEV)
    u = torch.empty(rows, N, dtype=torch.float32, device=DEV)
    code = kk.PLAIN_ACTIVATIONS[act]
    kk.linear(a, x, w, kk.plain_act_epilogue(code))
    kk.linear(u, x, w)
    kk.activation(b, u, code)
    kk.check_device_status()
    assert torch.equal(a, b)


@pytest.mark.parametrize("M,D", [(1, 40), (7, 42), (5, 64), (3, 1000), (9, 2048), (2, 4096), (2, 5000)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16", None])
def test_a_result_is_normed_on_its_way_into_the_stream(M, D, dtype):
    x, y = inputs(M, D, 1, False, 3.0), inputs(M, D, 2, False, 0.5)
    w = 0.3 * inputs(1, D, 3, False)[0]
    xd, yd = torch.from_numpy(x).float().to(DEV), torch.from_numpy(y).float().to(DEV)
    h = None if dtype is None else torch.zeros(M, D, dtype=DT[dtype], device=DEV)
    want = xd.double().cpu().numpy() + P.norm_around_one(yd.double().cpu().numpy(), w, 1e-2)
    K().outnorm_residual(xd, yd, torch.from_numpy(1 + w).float().to(DEV), 1e-2, h=h)
    assert err(xd.double().cpu().numpy(), want) < 1e-6
    if h is not None:
        assert torch.equal(h, xd.to(DT[dtype]))


@pytest.mark.parametrize("n", [1, 3, 4, 1000, 4099])
@pytest.mark.parametrize("a,cap", [(0.5, 4.0), (1.0, 20.0), (3.0, 0.0), (1.0, 0.5)])
def test_logits_are_scaled_and_capped(n, a, cap):
    z = inputs(1, n, 3, False, 6.0)[0]
    t = torch.from_numpy(z).float().to(DEV)
    K().softcap(t, a, cap)
    want = cap * np.tanh(a * z / cap) if cap else a * z
    assert err(t.double().cpu().numpy(), want) < 1e-6


# ---- whole models --------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    from lastengine_b200.weights import write_model_dir
    return {n: write_model_dir(cfg, str(tmp_path_factory.mktemp("z" + n)), seed=71 + i, norm_init="random")
            for i, (n, cfg) in enumerate(ALL.items())}


_tensors, _plain = {}, {}


def tensors_of(name, dirs):
    if name not in _tensors:
        _tensors[name] = P.read_safetensors(os.path.join(dirs[name], "model.safetensors"))
    return _tensors[name]


def plain(name, dirs, tokens):
    key = (name, tuple(tokens))
    if key not in _plain:
        _plain[key] = P.forward(ALL[name], tensors_of(name, dirs), tokens)
    return _plain[key]


def close(got, want, dtype) -> bool:
    """32-bit: every position within the tolerance.  bfloat16: the plain implementation does not round, and the norms on
    the sublayers' results amplify rounding where a result is small, so single positions may leave the tolerance: nine
    in ten within it, half of them within half of it, none beyond three times it."""
    got = got.double().cpu().numpy() if isinstance(got, torch.Tensor) else np.asarray(got)
    e = np.abs(got - want).max(-1) / np.abs(want).max()
    if dtype == "float32":
        return bool(np.all(e < H.TOL_F32))
    if e.max() > 3 * H.TOL_BF16:
        return False
    return bool(e.size < 8 or (np.median(e) < H.TOL_BF16 / 2 and np.quantile(e, 0.9) < H.TOL_BF16))


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
    assert close(H.run_tail(eng, reqs[0], tail=90), want[0], dtype)          # decoding across page, chunk and window borders
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


@pytest.mark.parametrize("name", ["A", "C", "E"])
def test_stream_after_every_layer_run(name, dirs):
    """The stream after the first 1, 2, ... layers, seen through the final norm and the head: models whose later layers
    are cut off against the plain implementation."""
    from lastengine_b200 import Engine
    from lastengine_b200.weights.safetensors_io import SafetensorsFile, save_file
    cfg = ALL[name]
    toks = reqs_for(name, [60], 47)[0]
    src = dirs[name]
    sf = SafetensorsFile(os.path.join(src, "model.safetensors"))
    for n_layers in range(1, len(cfg["layers"])):
        cut = dict(cfg, layers=cfg["layers"][:n_layers])
        d = os.path.join(src, f"cut{n_layers}")
        os.makedirs(d, exist_ok=True)
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cut, f)
        keep = {n: sf.tensor(n).clone() for n in sf.names() if not n.startswith("l") or int(n.split(".")[0][1:]) < n_layers}
        save_file(keep, os.path.join(d, "model.safetensors"))
        eng = Engine.from_pretrained(d, dtype="float32", max_tokens=256, max_seqs=2)
        w = P.read_safetensors(os.path.join(d, "model.safetensors"))
        assert close(H.run_whole(eng, toks), P.forward(cut, w, toks), "float32"), f"after {n_layers} layers"


def test_a_layer_that_borrows_tensors_has_a_memory_of_its_own(dirs):
    """The same folder with every borrowed layer written out as a layer of its own gives the same numbers, and a
    borrowing layer that read the owner's cache would not: the two runs see different streams."""
    from lastengine_b200 import Engine
    cfg, w = ALL["A"], tensors_of("A", dirs)
    toks = reqs_for("A", [90], 48)[0]
    want = plain("A", dirs, toks)
    streams = []
    P.forward(cfg, w, toks, streams)
    assert err(streams[1], streams[0]) > 0.05
    spread = {"layers": [{k: v for k, v in l.items() if k != "weights_of"} for l in cfg["layers"]]}
    full = dict(cfg, **spread)
    wf = {k: v for k, v in w.items() if not (k.startswith("l") and k[1].isdigit())}
    for i in range(len(cfg["layers"])):
        wf.update({f"l{i}.{n}": v for n, v in P.sub(w, f"l{P.owner_of(cfg, i)}").items()})
    assert np.abs(P.forward(full, wf, toks) - want).max() < 1e-9
    eng = Engine.from_pretrained(dirs["A"], dtype="float32", max_tokens=512, max_seqs=2)
    assert len(eng.model.blocks) == 3 and len(eng.cache._where) == 5
    assert close(H.run_tail(eng, toks, tail=60), want, "float32")


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_logits_do_not_depend_on_the_cut_or_the_batch_beyond_rounding(name, dirs):
    from lastengine_b200 import Engine
    eng = Engine.from_pretrained(dirs[name], dtype="float32", max_tokens=1024, max_seqs=6)
    reqs = reqs_for(name, [140, 9], 41)
    whole = H.run_whole(eng, reqs[0])
    tail = H.run_tail(eng, reqs[0], tail=80)
    batched = H.run_batch(eng, reqs, [61, 4])[0]
    assert H.rel_err(tail, whole) < 5e-6 and H.rel_err(batched, whole) < 5e-6


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("D", "float32"), ("B", "bfloat16"), ("C", "float32"), ("E", "bfloat16")])
def test_long_decoding_from_a_short_prompt(name, dtype, dirs):
    """Several chunks and windows pass while decoding; pages behind them are given back on the way."""
    from lastengine_b200 import Engine
    eng = Engine.from_pretrained(dirs[name], dtype=dtype, max_tokens=512, max_seqs=2)
    r = reqs_for(name, [330], 42)[0]
    got = H.run_tail(eng, r, tail=326)
    assert close(got, plain(name, dirs, r), dtype)
    eng.cache.check()


@pytest.mark.parametrize("seed", list(range(301, 313)))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layer order, sizes, chunks, windows and borrowed tensors drawn at random: whole prompts, a tail token by token and
    an unequal batch in 32-bit against the plain implementation, every position held; bfloat16 over the positions."""
    from lastengine_b200 import Engine
    from lastengine_b200.weights import write_model_dir
    rng = np.random.default_rng(seed)
    cfg = random_config(rng)
    d = write_model_dir(cfg, str(tmp_path / "m"), seed=seed, norm_init="random")
    w = P.read_safetensors(os.path.join(d, "model.safetensors"))
    reqs = [rng.integers(0, cfg["vocab"], size=n).tolist() for n in (210, 40)]
    want = [P.forward(cfg, w, r) for r in reqs]
    eng = Engine.from_pretrained(d, dtype="float32", max_tokens=1024, max_seqs=4)
    for r, wv in zip(reqs, want):
        assert close(H.run_whole(eng, r), wv, "float32"), cfg
    assert close(H.run_tail(eng, reqs[0], tail=90), want[0], "float32"), cfg
    for g, wv in zip(H.run_batch(eng, reqs, [130, 9]), want):
        assert close(g, wv, "float32"), cfg
    eng.cache.check()
    eng16 = Engine.from_pretrained(d, dtype="bfloat16", max_tokens=1024, max_seqs=4)
    for got in (H.run_whole(eng16, reqs[0]), H.run_tail(eng16, reqs[0], tail=90)):
        e = np.abs(got.double().numpy() - want[0]).max(-1) / np.abs(want[0]).max()
        assert np.median(e) < H.TOL_BF16, cfg


def test_a_step_longer_than_a_pass_runs_in_pieces(dirs):
    """A prompt step of more rows than a pass takes is cut where the pass ends, inside chunks and windows."""
    from lastengine_b200 import Engine
    reqs = reqs_for("A", [150, 40], 49)
    eng = Engine.from_pretrained(dirs["A"], dtype="float32", max_tokens=512, max_seqs=4, max_batch_tokens=47)
    seqs = [eng.new_sequence() for _ in reqs]
    got = H.to_host(eng.step(seqs, reqs, [list(range(len(r))) for r in reqs]))
    eng.release(seqs)
    assert close(got[:150], plain("A", dirs, reqs[0]), "float32") and close(got[150:], plain("A", dirs, reqs[1]), "float32")
    eng.cache.check()


def plain_greedy(name, dirs, prompt, n):
    """Greedy tokens of the plain implementation, and per token the gap between the two best logits."""
    toks, out, margins = list(prompt), [], []
    for _ in range(n):
        row = plain(name, dirs, toks)[-1]
        top = np.sort(row)[-2:]
        margins.append(float((top[1] - top[0]) / np.abs(row).max()))
        out.append(int(np.argmax(row)))
        toks.append(out[-1])
    return out, margins


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("A", "bfloat16"), ("B", "bfloat16"), ("C", "float32"), ("D", "float32")])
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
            if margins[i] < 2 * TOL[dtype]:
                break
            assert got[i] == want[i], f"{name} {dtype}: prompt of {len(p)}, token {i}"
            compared += 1
    assert compared >= (steps * len(prompts) // 2 if dtype == "float32" else 2)
    assert eng.cache.slots.n_held == 0
    eng.cache.check()


def test_graphs_and_plain_steps_generate_the_same_over_several_chunks(dirs):
    """Greedy generation over more than two chunks and a window, replayed and not: the same tokens (the split of a
    decode step's key range is chosen for the table's width in one and for the length in the other)."""
    from lastengine_b200 import Engine, SamplingParams
    out = []
    for graphs in (True, False):
        eng = Engine.from_pretrained(dirs["E"], dtype="float32", max_tokens=1024, use_graphs=graphs)
        res = eng.generate(reqs_for("E", [30, 61, 2], 44), SamplingParams(temperature=0.0), max_new_tokens=180, stop_token_ids=[])
        out.append([list(t) for t in res.tokens])
        eng.cache.check()
    assert out[0] == out[1]


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "bfloat16"), ("D", "float32")])
def test_a_sequence_written_out_and_read_back_goes_on_where_it_stood(name, dtype, dirs):
    """Keys and values of a chunk and latent rows of a window go out as bytes and come back into other pages."""
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
    if margins[0] > 1e-4:
        assert rows[0]["tokens"][0] == want[0]
    sampled = [subprocess.run(base + ["--temperature", "0.9", "--top-k", "20", "--seed", "5"], capture_output=True, text=True, timeout=600)
               for _ in range(2)]
    assert sampled[0].returncode == 0, sampled[0].stderr[-1500:]
    assert sampled[0].stdout == sampled[1].stdout
    p2 = subprocess.run([sys.executable, exe, "inspect", d], capture_output=True, text=True, timeout=600)
    assert p2.returncode == 0, p2.stderr[-1500:]
    assert "latent_attention" in p2.stdout and "output_norm_residual" in p2.stdout or "Zafilix" in p2.stdout
