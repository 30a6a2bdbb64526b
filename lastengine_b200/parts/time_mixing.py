"""Time mixing: a recurrent mixer with a matrix state per head whose decay depends on the token, channel by channel.

Every projection reads its own mix of a row and the row before it (zeros before a sequence's first row):
    x_s = h + (h_before - h) mu_s,   s in r, k, v, g, w
    r = W_r x_r,  k = W_k x_k,  v = W_v x_v   (heads x dim),   gate = silu(W_g x_g)
    decay = exp(-exp(W_2 tanh(W_1 x_w) + w_0))   per head and key channel
Per head, with a weight u per key channel for the row's own write,
    o = (S + diag(u) k v^T)^T r,   then   S <- diag(decay) S + k v^T
o is divided by its root mean square per head (eps of the norm); the heads side by side are multiplied by a weight over all
of them and by the gate; out = W_o o.

State per sequence: S [heads, dim, dim] (a column contiguous) and the last row's h, both zero at its start.  The mixes of
r, k, v and g are four buffers of one grouped product; the projections run in the activation type with float results, and
everything between them and the output projection (the decay's tanh, its second product and exponentials, the recurrence,
the norm and the gate) is float.  The inner size of W_1 and W_2 is whatever the checkpoint's tensors have.
"""
from __future__ import annotations

import torch

from ..ops import kernels
from ..registry import MIXERS
from .base import MATRIX, NORM, VECTOR, BuildEnv, Mixer, StateSpec, TensorSpec

_MIXES = ("r", "k", "v", "g", "w")       # in the order the mixes lie in memory: the first four feed one grouped product


@MIXERS.register("time_mixing")
class TimeMixingMixer(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, norm_eps: float, decay_rank: int | None = None,
                 names: dict[str, str] | None = None):
        """`decay_rank`: the inner size of the decay's low-rank pair; None: the checkpoint's (random weights then take a
        quarter of head_dim, at least 8)."""
        if head_dim > kernels.RECURRENCE_MAX_ROWS:
            raise ValueError(f"head_dim {head_dim} is larger than the recurrence kernel takes ({kernels.RECURRENCE_MAX_ROWS})")
        self.D, self.H, self.d = int(hidden_size), int(num_heads), int(head_dim)
        self.eps, self.rank = float(norm_eps), decay_rank
        self.n = {"r": "r", "k": "k", "v": "v", "g": "g", "o": "o", "decay_down": "w1", "decay_up": "w2", "decay_base": "w0",
                  "bonus": "u", "norm": "norm", **{f"mu_{s}": f"mu.{s}" for s in _MIXES}}
        self.n.update(names or {})
        self.w_in = self.w_low = self.w_out = self.mu = self.w2 = self.w0 = self.bonus = self.norm_w = None

    def tensors(self) -> dict[str, TensorSpec]:
        D, C, n = self.D, self.H * self.d, self.n
        rank, free = (-1 if self.rank is None else int(self.rank)), max(8, self.d // 4)
        t = {n[f"mu_{s}"]: TensorSpec((D,), VECTOR, std=0.5) for s in _MIXES}
        t.update({n[s]: TensorSpec((C, D), MATRIX) for s in _MIXES[:4]})
        t.update({n["o"]: TensorSpec((D, C), MATRIX), n["decay_down"]: TensorSpec((rank, D), MATRIX, free=free),
                  n["decay_up"]: TensorSpec((C, rank), VECTOR, free=free), n["decay_base"]: TensorSpec((C,), VECTOR, std=1.0),
                  n["bonus"]: TensorSpec((self.H, self.d), VECTOR, std=0.5), n["norm"]: TensorSpec((C,), NORM)})
        return t

    def cache_spec(self):
        return StateSpec((self.H, self.d, self.d), torch.float32), StateSpec((self.D,), torch.float32)

    def load(self, tensors, env: BuildEnv) -> None:
        n, f32 = self.n, torch.float32
        low, up = tensors[n["decay_down"]], tensors[n["decay_up"]]
        if low.shape[0] != up.shape[1]:
            raise ValueError(f"the decay's low-rank pair does not fit: {tuple(low.shape)} with {tuple(up.shape)}")
        self.rank = int(low.shape[0])
        self.w_in = torch.stack([tensors[n[s]] for s in _MIXES[:4]]).contiguous()
        self.w_low, self.w_out = low.contiguous(), tensors[n["o"]].contiguous()
        self.mu = torch.stack([tensors[n[f"mu_{s}"]].to(f32) for s in _MIXES]).contiguous()
        self.w2 = up.to(f32).t().contiguous()
        self.w0 = tensors[n["decay_base"]].to(f32).reshape(-1).contiguous()
        self.bonus = tensors[n["bonus"]].to(f32).reshape(-1).contiguous()
        self.norm_w = tensors[n["norm"]].to(f32).contiguous()

    def flops_per_row(self) -> int:
        # the products, the low rank's second one, and per head the state's read-out, decay and write
        return super().flops_per_row() + 2 * self.H * self.d * int(self.rank or 0) + 8 * self.H * self.d * self.d

    def forward(self, h, out, accumulate, batch, cache, env) -> None:
        H, d, C = self.H, self.d, self.H * self.d
        M = h.shape[0]
        ws, f32 = env.workspace, torch.float32
        mix = ws.get("tmix.mix", (5, M, self.D), env.dtype)
        kernels.row_shift_mix(mix, h, self.mu, cache.states[1], batch)
        proj = ws.get("tmix.proj", (4, M, C), f32)
        kernels.linear(proj.view(4 * M, C), mix[:4].view(4 * M, self.D), self.w_in,
                       group_offsets=kernels.equal_group_offsets(4, M, h.device), rows_hint=4 * M)
        low = ws.get("tmix.low", (M, self.rank), f32)
        kernels.linear(low, mix[4], self.w_low)
        decay = ws.get("tmix.decay", (M, C), f32)
        kernels.low_rank_decay(decay, low, self.w2, self.w0)
        o = ws.get("tmix.o", (M, C), f32)
        kernels.gated_recurrence(o, proj[1], proj[0], proj[2], None, decay, cache.states[0], batch, H, H, d, d, delta=False,
                                 bonus=self.bonus)
        on = ws.get("tmix.on", (M, C), env.dtype)
        kernels.group_norm_gate(on, o, proj[3], self.norm_w, d, self.eps, gate_first=False, silu_after=True)
        kernels.linear(out, on, self.w_out, kernels.ACCUMULATE if accumulate else kernels.STORE)
