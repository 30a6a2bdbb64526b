"""The Nolapel decoder on the CPU: reading of config.json, the plan, cache needs, random weights and the loader's names, the
embedding's state among the cache's, and the plain implementation's own pieces."""
import copy
import os

import numpy as np
import pytest
import torch

import harness  # noqa: F401  (puts the repository and tests/ on the path)
import plain_nolapel as P
from nolapel_configs import ALL, N_A, N_B, N_C, N_D, N_E, random_config


def plan_of(cfg):
    from lastengine_b200.registry import plan_from_config
    return plan_from_config(cfg)


def model_of(cfg):
    from lastengine_b200.engine.model import Model
    from lastengine_b200.parts.base import BuildEnv
    return Model(plan_of(cfg), BuildEnv(torch.device("cpu"), torch.float32))


def test_every_size_and_constant_comes_from_the_file():
    from lastengine_b200.config import NolapelConfig
    c = NolapelConfig.from_dict(N_A)
    assert (c.vocab, c.width, c.eps, c.logit_softcap) == (220, 80, 1e-5, 9.0)
    assert (c.bigram.buckets, c.bigram.mul_prev, c.bigram.mul_cur) == (97, 31, 5)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (0, 2, 2)
    assert [l.type for l in c.layers] == ["attention", "parallel", "mamba2"]
    a = c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.conv, a.scale, a.window, a.temperature) == (8, 2, 64, 4, 0.12, 40, (0.4, 16.0))
    p = c.layers[1].mixer
    assert (p.left.heads, p.left.kv_heads, p.left.dim, p.left.vdim, p.left.scale, p.left.rot.dims, p.left.rot.base) \
        == (4, 2, 64, 64, 0.13, 64, 10000.0)
    assert (p.left_scale, p.right_heads, p.right_dim, p.right_scale) == (0.7, 3, 16, 1.3)
    s = c.layers[2].mixer
    assert (s.heads, s.vdim, s.state, s.groups, s.norm_groups, s.conv) == (6, 16, 24, 3, 2, 3)
    assert [(l.mlp.experts, l.mlp.top, l.mlp.ff, l.mlp.shared_ff) for l in c.layers] == [(6, 2, 48, 32), (5, 1, 40, 24), (4, 3, 32, 56)]
    assert c.runs() == [(0, 0), (1, None), (0, 1), (1, None), (2, None)]


def test_what_may_be_absent_has_the_design_s_defaults():
    from lastengine_b200.config import NolapelConfig
    c = NolapelConfig.from_dict(N_C)
    assert c.bigram is None and c.loop is None and c.logit_softcap == 0.0
    assert (c.layers[0].mixer.left_scale, c.layers[0].mixer.right_scale, c.layers[0].mixer.left.rot.dims) == (1.0, 1.0, 0)
    assert c.layers[1].mixer.temperature is None and c.layers[1].mlp.shared_ff == 0 and c.layers[3].mlp is None
    assert NolapelConfig.from_dict(N_E).layers[0].mixer.window == 0
    null = copy.deepcopy(N_C)
    null.update(loop=None, embedding=None, logit_softcap=None)
    null["layers"][1]["mixer"].update(q_temp=None, mask={"size": 1})
    assert NolapelConfig.from_dict(null) == c
    idle = dict(copy.deepcopy(N_A), loop={"start": 1, "stop": 1, "times": 4})
    assert [r for r, _ in NolapelConfig.from_dict(idle).runs()] == [0, 1, 2]
    assert plan_of(idle).unused_tensors == ("loop.step", "loop.in") and not plan_of(idle).stream_adds


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"),
    (("layers", 1, "mixer", "left", "kv_heads"), 3, "kv_heads"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 15, "even"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 66, "rot.dims"),
    (("layers", 0, "mixer", "mask", "size"), 0, "size"),
    (("layers", 0, "mixer", "q_temp", "every"), 0, "every"),
    (("layers", 0, "mixer", "vdim"), 32, "vdim"),
    (("layers", 0, "type"), "conv", "unknown layer type"),
    (("layers", 1, "mlp", "kind"), "dense", "unknown mlp kind"),
    (("layers", 1, "mlp", "router", "top"), 6, "top"),
    (("layers", 2, "mixer", "groups"), 4, "groups"),
    (("layers", 2, "mixer", "norm_groups"), 7, "norm_groups"),
    (("loop", "stop"), 4, "loop"),
    (("loop", "times"), 0, "times"),
    (("embedding", "bigram", "buckets"), 0, "buckets"),
    (("logit_softcap",), -3.0, "logit_softcap"),
])
def test_errors_name_the_key(path, value, word):
    from lastengine_b200.config import ConfigError, NolapelConfig
    cfg = copy.deepcopy(N_A)
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        NolapelConfig.from_dict(cfg)


@pytest.mark.parametrize("path", [("layers", 0, "mixer", "scale"), ("layers", 0, "mixer", "conv"), ("layers", 1, "mixer", "right", "dim"),
                                  ("layers", 1, "mixer", "left", "vdim"), ("layers", 2, "mixer", "state"), ("layers", 0, "mlp", "router", "top"),
                                  ("layers", 0, "mlp", "expert", "ff"), ("layers", 0, "mixer", "q_temp", "every"), ("norm", "eps"), ("width",),
                                  ("embedding", "bigram", "mul_cur")])
def test_a_missing_key_is_named(path):
    from lastengine_b200.config import ConfigError, NolapelConfig
    cfg = copy.deepcopy(N_A)
    at = cfg
    for k in path[:-1]:
        at = at[k]
    del at[path[-1]]
    with pytest.raises(ConfigError, match=path[-1]):
        NolapelConfig.from_dict(cfg)


def test_plan_schedule_cache_needs_and_names():
    from lastengine_b200.engine.model import EMBEDDING_ENTRY
    from lastengine_b200.parts.base import KVSpec, StateSpec
    plan = plan_of(N_A)
    assert plan.architecture == "Nolapel" and [e.layer for e in plan.schedule] == [0, 1, 0, 1, 2]
    assert [(a.before, a.matrix, a.row, a.embedding) for a in plan.stream_adds] == [(0, "loop.in", 0, False), (2, "loop.in", 1, False)]
    model = model_of(N_A)
    specs = model.cache_specs()
    assert specs[EMBEDDING_ENTRY] == StateSpec((1,), torch.int32)
    assert specs[0] == specs[2] == (KVSpec(2, 64, window=40), StateSpec((640, 3)))            # every pass has its own
    assert specs[1] == specs[3] == (KVSpec(2, 64), StateSpec((3, 16, 16)), StateSpec((80,)))
    assert specs[4] == (StateSpec((6, 16, 24)), StateSpec((240, 2)))
    names = {plan.checkpoint_names(n): tuple(s.shape) for n, s in model.tensor_specs().items()}
    want = {"embed": (220, 80), "bigram": (98, 80), "head": (220, 80), "final.norm": (80,), "final.norm.alpha": (), "final.norm.b": (80,),
            "loop.in": (80, 160), "loop.step": (2, 80), "l0.norm1": (80,), "l0.norm1.alpha": (), "l0.norm1b.b": (80,), "l0.norm2b": (80,),
            "l0.mix.q": (512, 80), "l0.mix.k": (128, 80), "l0.mix.q.conv": (512, 4), "l0.mix.k.conv": (128, 4), "l0.mix.q.norm": (64,),
            "l0.mix.k.norm": (64,), "l0.mix.o": (80, 512), "l1.mix.left.q": (256, 80), "l1.mix.left.v": (128, 80), "l1.mix.left.sink": (4,),
            "l1.mix.left.o": (80, 256), "l1.mix.right.mu.w": (80,), "l1.mix.right.r": (48, 80), "l1.mix.right.w1": (-1, 80),
            "l1.mix.right.w2": (48, -1), "l1.mix.right.w0": (48,), "l1.mix.right.u": (3, 16), "l1.mix.right.norm": (48,),
            "l1.mix.right.o": (80, 48), "l2.mix.in": (96 + 240 + 6, 80), "l2.mix.conv.b": (240,), "l2.mix.D": (6,), "l0.mlp.router": (6, 80),
            "l0.mlp.e5.down": (80, 48), "l0.mlp.shared.gate": (32, 80)}
    assert {k: names.get(k) for k in want} == want
    assert not any(n.endswith((".mix.v", ".v.conv", ".correction")) for n in names)
    assert "l3.norm2" not in {plan_of(N_C).checkpoint_names(n) for n in model_of(N_C).tensor_specs()}
    # heads of up to 128 are stored at a width the fast kernels take, wider ones as they are
    d = model_of(N_D).cache_specs()
    assert d[0][0] == KVSpec(4, 64, window=130) and d[2][0] == KVSpec(4, 96)
    assert model_of(N_E).cache_specs()[0][0] == KVSpec(2, 200) and EMBEDDING_ENTRY not in model_of(N_C).cache_specs()


def test_the_embedding_s_state_is_a_slot_s_and_goes_out_and_in():
    """The last token of a sequence lies among the cache's states: zeroed when a slot is given out, written out first."""
    from lastengine_b200.cache import Cache
    model = model_of(N_A)
    c = Cache(model.cache_specs(), max_tokens=640, max_seqs=3, dtype=torch.float32, device=torch.device("cpu"))
    a = c.alloc_seq()
    c.reserve({a: 70})
    c.commit({a: 70})
    view = c.view(-1, True, {})
    assert view.state.shape == (3, 1) and view.state.dtype == torch.int32 and view.k is None
    view.state[a, 0] = 123456
    for g in c.state_groups:
        if g.spec.dtype == torch.float32:
            g.data.normal_()
    data = c.export_seq(a)
    b = c.import_seq(data)
    assert int(c.view(-1, True, {}).state[b, 0]) == 123456 and c.export_seq(b) == data
    c.free_seq(a)
    c.free_seq(b)
    e = c.alloc_seq()
    assert int(c.view(-1, True, {}).state[e, 0]) == 0
    c.free_seq(e)
    c.check()


def test_random_folder_goes_through_the_loader(tmp_path):
    from lastengine_b200.weights import write_model_dir
    from lastengine_b200.weights.loader import load_model_dir
    d = write_model_dir(N_A, str(tmp_path / "m"), seed=3, norm_init="random")
    w = P.read_safetensors(os.path.join(d, "model.safetensors"))
    assert w["bigram"].shape == (98, 80) and w["final.norm.alpha"].shape == () and w["l1.mix.right.w1"].shape[0] == w["l1.mix.right.w2"].shape[1]
    m = model_of(N_A)
    load_model_dir(m, d)
    assert m.stream_matrices["loop.in"].shape == (80, 160) and np.allclose(m.final_norm.alpha, w["final.norm.alpha"])
    assert np.allclose(m.blocks[1].mixer.right.w2.numpy(), w["l1.mix.right.w2"].T)
    lg = P.forward(N_A, w, [1, 2, 3, 4])
    assert lg.shape == (4, 220) and np.all(np.isfinite(lg)) and np.abs(lg).max() < 9.0
    for n, cfg in ALL.items():
        assert plan_of(cfg).schedule and model_of(cfg).tensor_specs(), n
    for seed in range(40):
        assert plan_of(random_config(np.random.default_rng(seed))).schedule


def test_parts_refuse_what_they_cannot_do():
    from lastengine_b200.registry import BLOCKS, EMBEDDINGS, MIXERS, NORMS
    base = dict(hidden_size=16, num_heads=2, num_kv_heads=1, head_dim=8, norm_eps=1e-5)
    for bad in (dict(values="keys", v_head_dim=4), dict(values="both"), dict(sink="one"), dict(slopes=[0.1]), dict(query_temperature=(0.1, 0.0))):
        with pytest.raises(ValueError):
            MIXERS.get("attention")(**base, **bad)
    with pytest.raises(ValueError):
        MIXERS.get("time_mixing")(hidden_size=16, num_heads=1, head_dim=300, norm_eps=1e-5)
    with pytest.raises(ValueError):
        EMBEDDINGS.get("token_pair_embedding")(8, 4, 0, 1, 1)
    rms, dyt = NORMS.get("rmsnorm")(8, 1e-5), NORMS.get("dynamic_tanh")(8)
    for args in ((rms, None, dyt, None), (dyt, None, None, None), (dyt, dyt, dyt, dyt)):
        with pytest.raises(ValueError):
            BLOCKS.get("sandwich_norm_residual")(None, None, args[0], args[1], args[2], args[3])


def test_plain_pairs_slopes_temperatures_and_sinks():
    assert P.pair_rows([4, 7, 2], {"buckets": 10, "mul_prev": 3, "mul_cur": 5}).tolist() == [10, (12 + 35) % 10, (21 + 10) % 10]
    assert np.allclose(P.slopes(2), [2.0 ** -4, 2.0 ** -8]) and np.allclose(P.slopes(3)[2], 2.0 ** -8)
    t = P.query_temperature(np.array([0, 2, 3, 6, 7]), {"coef": 0.5, "every": 4})
    assert np.allclose(t, [1, 1, 1 + .5 * np.log(2), 1 + .5 * np.log(2), 1 + .5 * np.log(3)])
    assert np.all(P.query_temperature(np.arange(4), None) == 1)
    p = P.softmax_with_sink(np.array([[1.0, 2.0, 9.0]]), np.array([[True, True, False]]), 0.0)
    assert np.allclose(p, np.array([[np.e, np.e ** 2, 0]]) / (1 + np.e + np.e ** 2))
    assert np.allclose(P.softmax_with_sink(np.array([[1.0, 1.0]]), np.ones((1, 2), bool), None), 0.5)
    assert np.allclose(P.softmax_with_sink(np.array([[-900.0]]), np.ones((1, 1), bool), 0.0), 0.0)
    s = P.seen(5, 3)
    assert [int(r.sum()) for r in s] == [1, 2, 3, 3, 3] and int(P.seen(4, 0).sum()) == 10
    # a bias of distance and one of the position alone differ as soon as a sink has its share
    q, k, v = np.zeros((3, 1, 2)), np.zeros((3, 1, 2)), np.ones((3, 1, 1))
    o = P.weighted_values(q, k, v, 1.0, P.seen(3, 0), [1.0], [0.0])
    assert np.allclose(o[:, 0], [n / (1 + n) for n in (1, 1 + np.exp(-1), 1 + np.exp(-1) + np.exp(-2))])


def test_plain_recurrence_reads_before_it_decays():
    """One number per head: o_t = r_t (S + u k_t v_t), S <- w_t S + k_t v_t."""
    r, k, v, w = (np.array(x, dtype=np.float64).reshape(3, 1, 1) for x in ([1, 2, 3], [1, 1, 2], [5, 7, 1], [0.5, 0.25, 1.0]))
    o = P.bonus_recurrence(r, k, v, w, np.array([[10.0]]))
    assert np.allclose(o.ravel(), [50.0, 2 * (5 + 70), 3 * (0.25 * 5 + 7 + 20)])
    h = np.arange(6.0).reshape(3, 2)
    assert np.array_equal(P.row_before(h), [[0, 0], [0, 1], [2, 3]])


def test_plain_experts_see_their_weighted_rows():
    """A gated expert is not linear in its input: a weight on the row and one on the result differ."""
    rng = np.random.default_rng(0)
    h = rng.standard_normal((4, 6))
    f = {"router": {"experts": 3, "top": 2}}
    w = {"router": rng.standard_normal((3, 6)), **{f"e{e}.{n}": rng.standard_normal(s) for e in range(3)
                                                   for n, s in (("gate", (5, 6)), ("up", (5, 6)), ("down", (6, 5)))}}
    ids, s, gap = P.route(h, w, f)
    assert np.all(s > 0) and np.all(s < 1) and np.all(gap >= 0) and np.all(s[:, 0] >= s[:, 1])
    y = P.expert_mixture(h, w, f)
    late = sum(s[:, j:j + 1] * np.stack([P.gated(h[t:t + 1], *(w[f"e{ids[t, j]}.{n}"] for n in ("gate", "up", "down")))[0] for t in range(4)])
               for j in range(2))
    assert np.abs(y - late).max() > 0.05
