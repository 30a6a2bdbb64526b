"""The Nolapel decoder as a plan.

x = embed[token] + bigram[hash of the previous token and this one] (parts.embedding, token_pair_embedding).  A layer is the
sandwich arrangement (parts.block): x <- x + n1b(mixer(n1(x))), x <- x + n2b(ff(n2(x))) with pointwise norms
tanh(alpha x) w + b (parts.norm, dynamic_tanh).  Mixers, chosen layer by layer: grouped-query attention (parts.attention)
whose q and k go through a short causal convolution and a weighted norm per head, whose values are the convolved keys, with a
query temperature, a distance bias per head, a window and a constant sink in the softmax; two mixers side by side
(parts.composite), causal attention with rotations and a learned sink per head beside time mixing (parts.time_mixing); or the
state-space layer (parts.recurrent).  Feed-forward: silu-gated experts chosen by the largest sigmoids, each on its weight
times the input, plus a shared expert; a layer may lack it.  A range of layers may run several times in a row with the
same weights, every run with a cache entry of its own; before every pass the stream becomes W [stream ; embedding output]
plus the pass's row of a table.  The model's norm, the head's own matrix, logits soft-capped.

Tensor names: embed, bigram, head, final.norm, loop.in, loop.step, and per layer l<i>.norm1, .norm1b, .norm2, .norm2b (a norm n
is the three tensors n, n.alpha and n.b), l<i>.mix.* (left.* and right.* of the parallel mixer) and
l<i>.mlp.{router, e<j>.gate/up/down, shared.gate/up/down}.
"""
from __future__ import annotations

import re

from ..config.nolapel import ATTENTION, MAMBA2, PARALLEL, NolapelConfig
from ..parts.base import LayerSpec, ModelPlan, PartSpec, ScheduleEntry, StreamAdd
from ..registry import ARCHITECTURES

NAMES = ("Nolapel", "nolapel")
PAIR_TABLE, LOOP_MATRIX, LOOP_TABLE = "bigram", "loop.in", "loop.step"

# names that are a part's prefix in the plan and a tensor in the checkpoint
_BARE = re.compile(r"^(embed|head)$")


def distance_slopes(heads: int) -> list[float]:
    """What the score of a key loses per position of distance, head by head."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def _alias(name: str) -> str:
    return name + ".weight" if _BARE.match(name) else name


def _checkpoint_name(canonical: str) -> str:
    return canonical[: -len(".weight")] if canonical.endswith(".weight") and _BARE.match(canonical[: -len(".weight")]) \
        else canonical


def _mixer(lay, W: int, eps: float) -> PartSpec:
    m = lay.mixer
    if lay.type == ATTENTION:
        return PartSpec("attention", {
            "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "norm_eps": eps,
            "qk_norm": True, "scale": m.scale, "window": m.window, "conv_taps": m.conv, "values": "keys",
            "slopes": distance_slopes(m.heads), "sink": "zero", "query_temperature": m.temperature,
            "wide_weights": True, "widen": True,
            "names": {"q": "q", "k": "k", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "q_conv": "q.conv", "k_conv": "k.conv"}})
    if lay.type == MAMBA2:
        return PartSpec("state_space", {
            "hidden_size": W, "num_heads": m.heads, "v_head_dim": m.vdim, "state_size": m.state, "num_groups": m.groups,
            "norm_groups": m.norm_groups, "conv_taps": m.conv, "norm_eps": eps})
    assert lay.type == PARALLEL
    a = m.left
    position = PartSpec("rope", {"rope_dim": a.rot.dims, "theta": a.rot.base, "style": "neox"}) if a.rot.dims else PartSpec("none")
    return PartSpec("parallel_mixers", {
        "left": PartSpec("attention", {
            "hidden_size": W, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim, "v_head_dim": a.vdim,
            "norm_eps": eps, "qk_norm": False, "scale": a.scale, "position": position, "sink": "learned",
            "wide_weights": True, "widen": True, "names": {"q": "q", "k": "k", "v": "v", "o": "o", "sink": "sink"}}),
        "right": PartSpec("time_mixing", {"hidden_size": W, "num_heads": m.right_heads, "head_dim": m.right_dim, "norm_eps": eps}),
        "left_scale": m.left_scale, "right_scale": m.right_scale})


def nolapel_plan(cfg: NolapelConfig) -> ModelPlan:
    W = cfg.width
    norm = PartSpec("dynamic_tanh", {"size": W, "tensor": ""})
    layers: list[LayerSpec] = []
    for i, lay in enumerate(cfg.layers):
        f = lay.mlp
        ffn = None if f is None else PartSpec("topk_moe", {
            "hidden_size": W, "num_experts": f.experts, "top_k": f.top, "expert_size": f.ff, "router": "sigmoid",
            "norm_topk": False, "use_bias": False, "activation": "silu", "weight_input": True, "shared_size": f.shared_ff,
            "names": {"router": "router", "gate": "e{e}.gate", "up": "e{e}.up", "down": "e{e}.down"}})
        layers.append(LayerSpec(
            prefix=f"l{i}", mixer=_mixer(lay, W, cfg.eps), ffn=ffn, mixer_norm=norm, post_mixer_norm=norm,
            ffn_norm=None if ffn is None else norm, post_ffn_norm=None if ffn is None else norm, block="sandwich_norm_residual",
            names={"mixer": "mix", "ffn": "mlp", "mixer_norm": "norm1", "post_mixer_norm": "norm1b", "ffn_norm": "norm2",
                   "post_ffn_norm": "norm2b"}))
    schedule, adds = [], []
    for at, (layer, opens) in enumerate(cfg.runs()):
        schedule.append(ScheduleEntry(layer))
        if opens is not None:
            adds.append(StreamAdd(before=at, table=LOOP_TABLE, row=opens, matrix=LOOP_MATRIX))
    embedding = PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": W})
    if cfg.bigram is not None:
        g = cfg.bigram
        embedding = PartSpec("token_pair_embedding", {
            "vocab_size": cfg.vocab, "hidden_size": W, "buckets": g.buckets, "mul_prev": g.mul_prev, "mul_cur": g.mul_cur,
            "pair_tensor": PAIR_TABLE})
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=W, vocab_size=cfg.vocab, embedding=embedding, final_norm=norm,
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tied": False, "softcap": cfg.logit_softcap}),
        layers=layers, schedule=schedule,
        names={"embedding": "embed", "final_norm": "final.norm", "head": "head"},
        tensor_aliases=_alias, checkpoint_names=_checkpoint_name,
        stream_adds=tuple(adds), stream_tables={LOOP_TABLE: (cfg.loop.times, W)} if adds else {},
        stream_matrices={LOOP_MATRIX: (W, 2 * W)} if adds else {},
        unused_tensors=() if adds else (LOOP_TABLE, LOOP_MATRIX),      # a checkpoint may carry those of a loop over no layers
        # sizes that keep the signal of random weights alive through the sums of a looped model
        init_std=0.05, init_stds={".router": 0.3, ".conv": 0.5, LOOP_TABLE: 0.3, "embed.weight": 0.5, PAIR_TABLE: 0.5,
                                  ".w2": 0.3})


@ARCHITECTURES.register(*NAMES)
def build_nolapel(raw: dict) -> ModelPlan:
    return nolapel_plan(NolapelConfig.from_dict(raw))
