"""The Zafilix decoder as a plan.

x = embed[token] * scale.  A layer norms what its sublayers give, not what they read (parts.block,
output_norm_residual): x <- x + N1(mixer(x)), x <- x + N2(ff(x)), RMS norms whose weights are stored around zero.
Mixers, chosen layer by layer: grouped-query attention (parts.attention) with q and k normed over their whole
projected row, a rotation of neighbouring pairs with linear position scaling, positions cut into chunks, and an
output gate per number of every head; or latent attention (parts.latent_attention) with q straight from its
projection, a split-half rotation of the rotated part and a sliding window.  Feed-forward: dense down(relu(up x)^2),
which a layer may lack.  A layer may run another layer's tensors with a cache entry of its own: the plan holds every
set of tensors once and a schedule entry per layer run.  Final RMS norm, the head's own matrix, logits times a
constant and soft-capped.

Tensor names: embed, head, final.norm, and per layer with tensors of its own l<i>.norm1, l<i>.norm2,
l<i>.mix.{q, k, v, q.norm, k.norm, g, o} or l<i>.mix.{q, dkv, dkv.norm, uk, uv, o}, and l<i>.mlp.{up, down}.
"""
from __future__ import annotations

import re

from ..config.zafilix import ATTENTION, LATENT, ZafilixConfig
from ..parts.base import LayerSpec, ModelPlan, PartSpec, ScheduleEntry
from ..registry import ARCHITECTURES

NAMES = ("Zafilix", "zafilix")

# names that are a part's prefix in the plan and a tensor in the checkpoint
_BARE = re.compile(r"^(embed|head)$")


def _alias(name: str) -> str:
    return name + ".weight" if _BARE.match(name) else name


def _checkpoint_name(canonical: str) -> str:
    return canonical[: -len(".weight")] if canonical.endswith(".weight") and _BARE.match(canonical[: -len(".weight")]) \
        else canonical


def zafilix_plan(cfg: ZafilixConfig) -> ModelPlan:
    W = cfg.width
    norm = PartSpec("rmsnorm", {"size": W, "eps": cfg.eps, "offset": 1.0, "tensor": ""})
    layers: list[LayerSpec] = []
    place: dict[int, int] = {}       # layer of the configuration -> its place among the layers with tensors
    for i in cfg.owners():
        lay, m = cfg.layers[i], cfg.layers[i].mixer
        position = PartSpec("rope", {"rope_dim": m.rot.dims, "theta": m.rot.base, "scaling_factor": m.rot.factor,
                                     "style": "adjacent" if lay.type == ATTENTION else "neox"}) \
            if m.rot.dims else PartSpec("none")
        if lay.type == ATTENTION:
            mixer = PartSpec("attention", {
                "hidden_size": W, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
                "norm_eps": cfg.eps, "qk_norm": "row", "position": position, "scale": m.scale, "chunk": m.chunk,
                "output_gate": "numbers", "wide_weights": True,
                "names": {"q": "q", "k": "k", "v": "v", "o": "o", "gate": "g", "q_norm": "q.norm", "k_norm": "k.norm"}})
        else:
            assert lay.type == LATENT
            mixer = PartSpec("latent_attention", {
                "hidden_size": W, "num_heads": m.heads, "head_dim": m.dim, "rope_dim": m.rot_dim, "v_head_dim": m.vdim,
                "q_rank": 0, "kv_rank": m.kv_rank, "norm_eps": cfg.eps, "scale": m.scale, "position": position,
                "window": m.window, "wide_weights": True})
        ffn = None if lay.ff is None else PartSpec("dense", {"hidden_size": W, "intermediate_size": lay.ff,
                                                             "activation": "relu_squared"})
        place[i] = len(layers)
        layers.append(LayerSpec(
            prefix=f"l{i}", mixer=mixer, ffn=ffn, mixer_norm=norm, ffn_norm=None if ffn is None else norm,
            block="output_norm_residual",
            names={"mixer": "mix", "ffn": "mlp", "mixer_norm": "norm1", "ffn_norm": "norm2"}))
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=W, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": W, "scale": cfg.embedding_scale}),
        final_norm=norm,
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": W, "tied": False, "scale": cfg.logit_scale,
                                      "softcap": cfg.logit_softcap}),
        layers=layers, schedule=[ScheduleEntry(place[lay.owner]) for lay in cfg.layers],
        names={"embedding": "embed", "final_norm": "final.norm", "head": "head"},
        tensor_aliases=_alias, checkpoint_names=_checkpoint_name,
        # sizes that keep the signal of random weights alive through stream and norms
        init_std=0.05)


@ARCHITECTURES.register(*NAMES)
def build_zafilix(raw: dict) -> ModelPlan:
    return zafilix_plan(ZafilixConfig.from_dict(raw))
