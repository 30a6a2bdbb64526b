"""A plain, slow implementation of the Nolapel decoder, for tests only.

Whole sequences, no cache, no batching, one function per mechanism, numpy in double precision.
It shares no code with the library.

The design in this file's notation.  x0[t] = E[c_t] + B[(a c_(t-1) + b c_t) mod n] with a table B of n + 1 rows whose
last one stands before a sequence's first token.  A range of layers may run n times in a row with the same weights;
before every pass x <- U [x; x0] + s_pass.  A layer norms what its sublayers read and what they give:
    x <- x + N1'(mixer(N1(x))),   x <- x + N2'(ff(N2(x)))      (the second only with a feed-forward)
with the pointwise N(x) = tanh(alpha x) w + b.  Mixers:

* attention: q and k through a short causal convolution per channel; the value of a position is its convolved key;
  RMS norm with a weight on every q and k head; q at position p times 1 + c ln(floor((p + 1) / m) + 1);
  s_ij = scale q_i . k_j - 2^(-8 (h + 1) / H) (i - j) over the last `size` positions; p = exp(s) / (1 + sum exp(s)).
* parallel: a left(h) + b right(h).  Left: plain causal attention, the first rot.dims numbers of q and k heads turned
  (pairs i, i + dims/2), one more logit per head in the denominator.  Right: every projection reads its own mix
  h_t + (h_(t-1) - h_t) mu; per head o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T with
  w = exp(-exp(W2 tanh(W1 mix) + w0)); o over its root mean square per head, times a weight, times silu(G mix).
* mamba2: W_in h = [z | x | B | C | dt]; x, B, C through a causal convolution with bias and silu;
  dt = softplus(dt + dt_bias); per head S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x; y silu(z) over its
  root mean square in equal parts, times a weight.

Feed-forward: experts D_e (silu(G_e u) * U_e u) of u = s_e h for the experts with the largest sigmoid scores s_e, plus a
shared expert of h.  Logits = cap tanh(H N(x) / cap).
"""
from __future__ import annotations

import json
import struct

import numpy as np


def read_safetensors(path: str) -> dict[str, np.ndarray]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        b, t = e["data_offsets"]
        if e["dtype"] == "BF16":
            arr = np.frombuffer(data[b:t], dtype=np.uint16).reshape(e["shape"])
            out[name] = (arr.astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif e["dtype"] == "F32":
            out[name] = np.frombuffer(data[b:t], dtype=np.float32).reshape(e["shape"]).astype(np.float64)
        elif e["dtype"] == "I32":
            out[name] = np.frombuffer(data[b:t], dtype=np.int32).reshape(e["shape"]).copy()
        else:
            raise ValueError(f"{name}: dtype {e['dtype']}")
    return out


# ---- small functions ---------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def over_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def pointwise_tanh(x, w, alpha, b):
    return np.tanh(alpha * x) * w + b


def norm_named(x, tensors, name):
    return pointwise_tanh(x, tensors[name], tensors[name + ".alpha"], tensors[name + ".b"])


def causal_conv(u, taps, bias=None):
    """u [T, C], taps [C, K] with the last column on the current row; zeros before the start."""
    T, C = u.shape
    K = taps.shape[1]
    padded = np.concatenate([np.zeros((K - 1, C)), u], axis=0)
    y = np.zeros((T, C))
    for j in range(K):
        y += padded[j: j + T] * taps[:, j]
    return y if bias is None else y + bias


# ---- embedding ------------------------------------------------------------------------------------------
def pair_rows(tokens, g):
    """Rows of the pair table: the previous token and this one hashed; the last row for the first token."""
    rows = [g["buckets"]]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * g["mul_prev"] + int(cur) * g["mul_cur"]) % g["buckets"])
    return np.asarray(rows)


def embedding(cfg, tensors, tokens):
    x = tensors["embed"][np.asarray(tokens)]
    g = (cfg.get("embedding") or {}).get("bigram")
    return x + tensors["bigram"][pair_rows(tokens, g)] if g else x


# ---- attention --------------------------------------------------------------------------------------------
def seen(T, size):
    """[T, T]: row i sees j <= i, and with size > 0 only the last `size` positions."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & ((d < size) if size else True)


def slopes(H):
    return 2.0 ** (-8.0 * (np.arange(H) + 1) / H)


def query_temperature(pos, t):
    """A factor per position that grows with the logarithm of how many times `every` positions have passed."""
    if not t:
        return np.ones(len(pos))
    return 1.0 + t["coef"] * np.log(np.floor((pos + 1) / t["every"]) + 1.0)


def rotate_halves(x, dims, base):
    """The first `dims` numbers of the last axis, pairs (i, i + dims/2), turned by the row's position times
    base^(-2i/dims); x [T, heads, n].  Angles are formed in 32-bit."""
    if not dims:
        return x
    half = dims // 2
    f = (np.float64(base) ** (-2.0 * np.arange(half) / dims)).astype(np.float32)
    a = (np.arange(x.shape[0], dtype=np.float32)[:, None] * f[None, :]).astype(np.float64)
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def softmax_with_sink(s, mask, sink):
    """Rows of s over the seen columns with one more logit `sink` in the denominator (None: none)."""
    s = np.where(mask, s, -np.inf)
    m = s.max(-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    p = np.exp(s - m)
    return p / (p.sum(-1, keepdims=True) + (0.0 if sink is None else np.exp(sink - m)))


def weighted_values(q, k, v, scale, mask, slope, sink):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H e]; slope and sink per head, or None."""
    T, H = q.shape[:2]
    G = k.shape[1]
    dist = np.arange(T)[:, None] - np.arange(T)[None, :]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        if slope is not None:
            s = s - slope[h] * dist
        out[:, h] = softmax_with_sink(s, mask, None if sink is None else sink[h]) @ v[:, g]
    return out.reshape(T, -1)


def biased_attention(h, w, m, eps):
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = causal_conv(h @ w["q"].T, w["q.conv"]).reshape(T, H, d)
    k = causal_conv(h @ w["k"].T, w["k.conv"]).reshape(T, G, d)
    v = k
    q = over_rms(q, eps) * w["q.norm"]
    k = over_rms(k, eps) * w["k.norm"]
    q = q * query_temperature(np.arange(T), m.get("q_temp"))[:, None, None]
    size = (m.get("mask") or {}).get("size", 0)
    return weighted_values(q, k, v, m["scale"], seen(T, size), slopes(H), np.zeros(H)) @ w["o"].T


def sink_attention(h, w, m):
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).reshape(T, H, d)
    k = (h @ w["k"].T).reshape(T, G, d)
    v = (h @ w["v"].T).reshape(T, G, e)
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q, k = rotate_halves(q, rot["dims"], rot["base"]), rotate_halves(k, rot["dims"], rot["base"])
    return weighted_values(q, k, v, m["scale"], seen(T, 0), None, w["sink"]) @ w["o"].T


# ---- recurrent mixers ---------------------------------------------------------------------------------------
def row_before(h):
    return np.concatenate([np.zeros((1, h.shape[1])), h[:-1]], axis=0)


def low_rank_decay(mix, w):
    return np.exp(-np.exp(np.tanh(mix @ w["w1"].T) @ w["w2"].T + w["w0"]))


def bonus_recurrence(r, k, v, decay, u):
    """r, k, v, decay [T, H, d], u [H, d]: the read-out sees the state before the row and the row's own write times u."""
    T, H, d = r.shape
    S = np.zeros((H, d, d))
    o = np.zeros((T, H, d))
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hij,hi->hj", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return o


def time_mixing(h, w, m, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    step = row_before(h) - h
    mix = {n: h + step * w["mu." + n] for n in "rkvgw"}
    r, k, v = ((mix[n] @ w[n].T).reshape(T, H, d) for n in "rkv")
    o = bonus_recurrence(r, k, v, low_rank_decay(mix["w"], w).reshape(T, H, d), w["u"])
    return (over_rms(o, eps).reshape(T, H * d) * w["norm"] * silu(mix["g"] @ w["g"].T)) @ w["o"].T


def side_by_side(h, w, m, eps):
    left = sink_attention(h, sub(w, "left."), m["left"])
    right = time_mixing(h, sub(w, "right."), m["right"], eps)
    return m.get("left_scale", 1.0) * left + m.get("right_scale", 1.0) * right


def mamba2(h, w, m, eps):
    T = h.shape[0]
    H, e, N, G, parts = m["heads"], m["vdim"], m["state"], m["groups"], m["norm_groups"]
    inner = H * e
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner: 2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    xs = xbc[:, :inner].reshape(T, H, e)
    B = np.repeat(xbc[:, inner: inner + G * N].reshape(T, G, N), H // G, axis=1)
    C = np.repeat(xbc[:, inner + G * N:].reshape(T, G, N), H // G, axis=1)
    dt = softplus(dt + w["dt_bias"])
    decay = np.exp(-np.exp(w["A_log"]) * dt)
    S = np.zeros((H, N, e))
    y = np.zeros((T, H, e))
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * xs[t][:, None, :]
        y[t] = np.einsum("hne,hn->he", S, C[t]) + w["D"][:, None] * xs[t]
    y = y.reshape(T, inner) * silu(z)
    return (over_rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * w["norm"]) @ w["o"].T


def mixer(kind, h, w, m, eps):
    return {"attention": biased_attention, "parallel": side_by_side, "mamba2": mamba2}[kind](h, w, m, eps)


# ---- feed-forward -----------------------------------------------------------------------------------------
def gated(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, w, f):
    """(chosen experts [T, top], their scores [T, top], gap between the last chosen and the first rejected score [T])."""
    E, top = f["router"]["experts"], f["router"]["top"]
    s = sigmoid(h @ w["router"].T)
    order = np.argsort(-s, axis=-1, kind="stable")
    ids = order[:, :top]
    gap = np.full(h.shape[0], np.inf)
    if top < E:
        gap = np.take_along_axis(s, order[:, top - 1: top], 1)[:, 0] - np.take_along_axis(s, order[:, top: top + 1], 1)[:, 0]
    return ids, np.take_along_axis(s, ids, 1), gap


def expert_mixture(h, w, f, gaps=None):
    ids, scores, gap = route(h, w, f)
    if gaps is not None:
        gaps.append(gap)
    y = np.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, j = np.nonzero(ids == e)
        if len(t):
            y[t] += gated(scores[t, j][:, None] * h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    if f.get("shared"):
        y = y + gated(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return y


# ---- the model ----------------------------------------------------------------------------------------
def sub(tensors, prefix):
    return {n[len(prefix):]: t for n, t in tensors.items() if n.startswith(prefix)}


def running_order(cfg):
    """(layer, number of the pass it opens or None) in running order."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop or loop["start"] == loop["stop"]:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


def enter_pass(x, x0, t, tensors):
    return np.concatenate([x, x0], axis=-1) @ tensors["loop.in"].T + tensors["loop.step"][t]


def forward(cfg, tensors, tokens, streams=None, gaps=None):
    """Logits [T, vocab] of one sequence; `streams` takes the stream after every layer run, `gaps` every routed layer
    run's distance to another choice of experts."""
    eps = cfg["norm"]["eps"]
    x0 = embedding(cfg, tensors, tokens)
    x = x0
    for i, opens in running_order(cfg):
        lay, p = cfg["layers"][i], f"l{i}."
        if opens is not None:
            x = enter_pass(x, x0, opens, tensors)
        y = mixer(lay["type"], norm_named(x, tensors, p + "norm1"), sub(tensors, p + "mix."), lay["mixer"], eps)
        x = x + norm_named(y, tensors, p + "norm1b")
        if lay.get("mlp"):
            y = expert_mixture(norm_named(x, tensors, p + "norm2"), sub(tensors, p + "mlp."), lay["mlp"], gaps)
            x = x + norm_named(y, tensors, p + "norm2b")
        if streams is not None:
            streams.append(x.copy())
    z = norm_named(x, tensors, "final.norm") @ tensors["head"].T
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(z / cap) if cap else z
