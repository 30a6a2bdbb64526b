"""The Zafilix decoder on the CPU: reading of config.json, the plan, cache needs and what the cache gives back, random
weights and the loader's names, and the plain implementation's own pieces."""
import copy
import os

import numpy as np
import pytest
import torch

import harness  # noqa: F401  (puts the repository and tests/ on the path)
import plain_zafilix as P
from zafilix_configs import ALL, Z_A, Z_B, Z_C, Z_D, Z_E


def plan_of(cfg):
    from lastengine_b200.registry import plan_from_config
    return plan_from_config(cfg)


def model_of(cfg):
    from lastengine_b200.engine.model import Model
    from lastengine_b200.parts.base import BuildEnv
    return Model(plan_of(cfg), BuildEnv(torch.device("cpu"), torch.float32))


def test_every_size_and_constant_comes_from_the_file():
    from lastengine_b200.config import ZafilixConfig
    c = ZafilixConfig.from_dict(Z_A)
    assert (c.vocab, c.width, c.eps, c.embedding_scale, c.logit_scale, c.logit_softcap) == (210, 80, 1e-5, 7.0, 0.4, 11.0)
    assert [l.type for l in c.layers] == ["attention", "latent_attention"] * 2 + ["attention"]
    a = c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk) == (4, 2, 64, 64, 0.11, 40)
    assert (a.rot.dims, a.rot.base, a.rot.factor) == (64, 10000.0, 3.0)
    m = c.layers[1].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.window) == (5, 24, 16, 40, 64, 0.15, 70)
    assert (m.rot.dims, m.rot.base, m.rot.factor) == (16, 5000.0, 1.0)
    assert [l.ff for l in c.layers] == [112, 112, 112, 72, 112]
    assert [l.owner for l in c.layers] == [0, 1, 0, 3, 0] and c.owners() == [0, 1, 3]        # the last one through layer 2


def test_what_may_be_absent_has_the_design_s_defaults():
    from lastengine_b200.config import ZafilixConfig
    c = ZafilixConfig.from_dict(Z_C)
    assert (c.embedding_scale, c.logit_scale, c.logit_softcap) == (1.0, 1.0, 0.0)
    assert c.layers[0].mixer.rot.dims == 0 and c.layers[0].mixer.chunk == 1
    assert c.layers[4].mixer.chunk == 0 and c.layers[4].mixer.rot.dims == 0 and c.layers[2].ff is None
    assert ZafilixConfig.from_dict(Z_D).layers[3].mixer.window == 0
    assert ZafilixConfig.from_dict(Z_B).layers[3].mixer.rot.factor == 1.0
    assert [l.owner for l in ZafilixConfig.from_dict(Z_D).layers] == [3, 1, 1, 3, 4]
    e = ZafilixConfig.from_dict(Z_E).layers[0].mixer
    assert (e.rot_dim, e.rot.dims, e.rot.factor) == (48, 20, 2.0)
    null = copy.deepcopy(Z_A)
    null["layers"][1]["weights_of"] = None
    assert ZafilixConfig.from_dict(null) == ZafilixConfig.from_dict(Z_A)


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "rot", "dims"), 15, "even"),
    (("layers", 3, "mixer", "rot", "dims"), 18, "rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 18, "rot.dims"),
    (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0, "positive"),
    (("layers", 1, "mixer", "mask", "size"), 0, "size"),
    (("layers", 0, "type"), "conv", "unknown layer type"),
    (("layers", 1, "mlp", "kind"), "gated", "unknown mlp kind"),
    (("layers", 2, "weights_of"), 9, "weights_of"),
    (("layers", 0, "weights_of"), 4, "circle"),
    (("layers", 2, "mlp", "ff"), 64, "sizes"),
    (("layers", 2, "weights_of"), 1, "sizes"),
    (("logit_softcap",), -3.0, "logit_softcap"),
])
def test_errors_name_the_key(path, value, word):
    from lastengine_b200.config import ConfigError, ZafilixConfig
    cfg = copy.deepcopy(Z_A)
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        ZafilixConfig.from_dict(cfg)


@pytest.mark.parametrize("path", [("layers", 0, "mixer", "scale"), ("layers", 1, "mixer", "kv_rank"), ("layers", 1, "mixer", "rot_dim"),
                                  ("layers", 0, "mixer", "mask", "size"), ("layers", 0, "mlp", "ff"), ("norm", "eps"), ("width",)])
def test_a_missing_key_is_named(path):
    from lastengine_b200.config import ConfigError, ZafilixConfig
    cfg = copy.deepcopy(Z_A)
    at = cfg
    for k in path[:-1]:
        at = at[k]
    del at[path[-1]]
    with pytest.raises(ConfigError, match=path[-1]):
        ZafilixConfig.from_dict(cfg)


def test_plan_schedule_cache_needs_and_names():
    from lastengine_b200.parts.base import KVSpec, LatentSpec
    plan = plan_of(Z_A)
    assert plan.architecture == "Zafilix" and [e.layer for e in plan.schedule] == [0, 1, 0, 2, 0]
    assert [l.prefix for l in plan.layers] == ["l0", "l1", "l3"]
    model = model_of(Z_A)
    specs = model.cache_specs()
    assert len(specs) == 5                                        # a layer that borrows tensors keeps a memory of its own
    assert specs[0] == specs[2] == specs[4] == KVSpec(2, 64, chunk=40)
    assert specs[1] == specs[3] == LatentSpec(64, 16, window=70)
    names = {plan.checkpoint_names(n): tuple(s.shape) for n, s in model.tensor_specs().items()}
    assert {k: names[k] for k in ("embed", "head", "final.norm", "l0.norm1", "l0.mix.q", "l0.mix.q.norm", "l0.mix.k.norm",
                                  "l0.mix.g", "l0.mix.o", "l1.mix.q", "l1.mix.dkv", "l1.mix.dkv.norm", "l1.mix.uk", "l1.mix.uv",
                                  "l1.mix.o", "l3.mlp.up", "l3.mlp.down")} == {
        "embed": (210, 80), "head": (210, 80), "final.norm": (80,), "l0.norm1": (80,), "l0.mix.q": (256, 80),
        "l0.mix.q.norm": (256,), "l0.mix.k.norm": (128,), "l0.mix.g": (256, 80), "l0.mix.o": (80, 256), "l1.mix.q": (200, 80),
        "l1.mix.dkv": (80, 80), "l1.mix.dkv.norm": (64,), "l1.mix.uk": (120, 64), "l1.mix.uv": (200, 64), "l1.mix.o": (80, 200),
        "l3.mlp.up": (72, 80), "l3.mlp.down": (80, 72)}
    assert not any(n.startswith(("l2.", "l4.")) for n in names) and "l1.mix.dq" not in names
    assert "l0.norm2" not in {plan_of(Z_B).checkpoint_names(n) for n in model_of(Z_B).tensor_specs()}
    # heads of unequal sizes are cached at the wider one where the fast kernels take it
    d = model_of(Z_D).cache_specs()
    assert d[1] == d[2] == KVSpec(4, 64, chunk=150) and d[4] == KVSpec(1, 96, chunk=130) and d[0] == LatentSpec(256, 64)
    assert model_of(Z_C).cache_specs()[2] == KVSpec(1, 22, 0, 10, chunk=33)


def test_chunked_and_windowed_pages_are_given_back_and_go_out_and_in():
    """A sequence grows token by token: what is held is what the next position still reads, for chunks of one position,
    of less than a page, of exactly one and of more, and for latent rows in a window.  What goes out as bytes comes back."""
    from lastengine_b200.cache import Cache
    from lastengine_b200.parts.base import KVSpec, LatentSpec
    for chunk in (1, 20, 32, 45, 70):
        specs = {0: KVSpec(1, 4, chunk=chunk), 1: LatentSpec(6, 2, window=chunk), 2: LatentSpec(6, 2, chunk=chunk), 3: KVSpec(1, 4)}
        c = Cache(specs, max_tokens=32 * 16, max_seqs=2, dtype=torch.float32, device=torch.device("cpu"), page_size=32)
        a = c.alloc_seq()
        for n in range(200):
            c.reserve({a: 1})
            c.commit({a: 1})
            length = n + 1
            for g in c.kv_groups:
                first = max(length + 1 - g.spec.window if g.spec.window else 0, length // chunk * chunk if g.spec.chunk else 0, 0)
                held = [j for j, p in enumerate(g.seq_pages[a]) if p >= 0]
                # every page that still holds a position from `first` on, and no other
                assert held == [j for j in range(len(g.seq_pages[a])) if (j + 1) * 32 - 1 >= first], (chunk, length, g.spec)
        c.check()
        for g in c.kv_groups:
            g.k_pool.normal_()
        data = c.export_seq(a)
        b = c.import_seq(data)
        assert c.length(b) == 200 and c.export_seq(b) == data
        c.free_seq(a)
        c.free_seq(b)
        c.check()
        assert all(g.pages.n_free == g.pages.n for g in c.kv_groups)


def test_random_folder_goes_through_the_loader(tmp_path):
    from lastengine_b200.weights import write_model_dir
    from lastengine_b200.weights.safetensors_io import SafetensorsFile
    d = write_model_dir(Z_D, str(tmp_path / "m"), seed=3, norm_init="random")
    sf = SafetensorsFile(os.path.join(d, "model.safetensors"))
    w = P.read_safetensors(os.path.join(d, "model.safetensors"))
    assert set(sf.names()) == set(w)
    assert w["l1.mix.q.norm"].shape == (512,) and w["l3.mix.dkv"].shape == (320, 96) and "l0.mix.q" not in w and "l2.norm1" not in w
    assert np.abs(w["l1.norm1"]).max() < 0.9 and np.abs(w["l1.norm1"]).max() > 0          # stored around zero
    lg = P.forward(Z_D, w, [1, 2, 3, 4])
    assert lg.shape == (4, 300) and np.all(np.isfinite(lg)) and np.abs(lg).max() < 30.0
    for n, cfg in ALL.items():
        assert [P.owner_of(cfg, i) for i in range(len(cfg["layers"]))] is not None and plan_of(cfg).schedule, n


def test_plain_chunks_windows_pairs_and_caps():
    s = P.seen_in_chunk(7, 3)
    assert [int(r.sum()) for r in s] == [1, 2, 3, 1, 2, 3, 1] and s[4].tolist() == [False] * 3 + [True, True, False, False]
    w = P.seen_in_window(5, 3)
    assert [int(r.sum()) for r in w] == [1, 2, 3, 3, 3] and w[4].tolist() == [False, False, True, True, True]
    a = P.angles(np.array([0, 2]), 4, 100.0, 4.0)
    assert np.allclose(a, [[0, 0], [0.5, 0.05]])
    x = np.arange(1.0, 7.0)[None, None, :].repeat(2, 0)
    n, h = P.rotate_neighbours(x, a), P.rotate_halves(x, a)
    assert np.allclose(n[0], x[0]) and np.allclose(h[0], x[0]) and np.allclose(n[1, 0, 4:], [5, 6]) and np.allclose(h[1, 0, 4:], [5, 6])
    assert np.allclose(n[1, 0, :2], [np.cos(.5) - 2 * np.sin(.5), 2 * np.cos(.5) + np.sin(.5)])
    assert np.allclose(h[1, 0, [0, 2]], [np.cos(.5) - 3 * np.sin(.5), 3 * np.cos(.5) + np.sin(.5)])
    assert np.allclose(P.head(np.array([[2.0]]), np.array([[3.0]]), 0.5, 4.0), 4.0 * np.tanh(0.75))
    assert np.allclose(P.head(np.array([[2.0]]), np.array([[3.0]]), 0.5, 0.0), 3.0)
    assert np.allclose(P.norm_around_one(np.array([[3.0, 4.0]]), np.array([0.0, 1.0]), 0.0), np.array([[3, 8]]) / np.sqrt(12.5))
