"""A plain, slow implementation of the Zafilix decoder, for tests only.

Whole sequences, no cache, no batching, one function per mechanism, numpy in double precision.
It shares no code with the library.

The design in this file's notation.  x[t] = E[token_t] * s_e.  Every layer run adds two normed results to the
stream; what the sublayers read is the stream as it stands:
    x <- x + N1(M(x));   x <- x + N2(F(x))      (F absent: the first sum alone)
N(y) = y / rms(y) * (1 + w) with rms(y) = sqrt(mean(y^2) + eps).  A layer that borrows another layer's weights
runs them again with a memory of its own.  M is one of two mixers:

* chunked attention: Q = Wq x, K = Wk x, V = Wv x.  The whole row Q is divided by its rms and multiplied by a weight
  over the row, K likewise; then heads are cut out of them.  The first `dims` numbers of a q or k head turn by
  the token's position, neighbours (2i, 2i+1) by the angle t * base^(-2i/dims) / factor.  Token t reads the
  tokens of its own chunk up to itself: floor(j / size) = floor(t / size), j <= t.  softmax(scale q.k), the heads
  side by side times sigmoid(Wg x), then Wo.
* latent attention in a window: q = Wq x per head [n | r] with n unrotated and r rotated numbers;
  [a | b] = Wdkv x, c = a / rms(a) * w; one rotated key part b for all heads, halves (i, i + dims/2) paired;
  keys Wuk c, values Wuv c per head; score (n.k + r.b) * scale over 0 <= t - j < size; softmax; Wo.

F(x) = D relu(U x)^2.  Logits: z = H N_final(x) * a, then cap * tanh(z / cap).
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
        else:
            raise ValueError(f"{name}: dtype {e['dtype']}")
    return out


# ---- small functions ---------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def over_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm_around_one(x, w, eps):
    """x over its root mean square times (1 + w)."""
    return over_rms(x, eps) * (1.0 + w)


def softmax_over(s, seen):
    """Softmax along the last axis over the places where `seen`."""
    s = np.where(seen, s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


def sub(w: dict, prefix: str) -> dict:
    """The tensors under `prefix.`, by the rest of their names."""
    p = prefix + "."
    return {k[len(p):]: v for k, v in w.items() if k.startswith(p)}


# ---- rotations --------------------------------------------------------------------------------------
def angles(pos, dims, base, factor=1.0):
    f = float(base) ** (-2.0 * np.arange(dims // 2) / dims) / factor
    return pos[:, None].astype(np.float64) * f[None, :]                                # [T, dims/2]


def rotate_neighbours(x, a):
    """x [T, heads, d]: numbers 2i and 2i + 1 turned by a[:, i]."""
    n = 2 * a.shape[1]
    y = x.copy()
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2] = u * c - v * s
    y[..., 1:n:2] = v * c + u * s
    return y


def rotate_halves(x, a):
    """x [T, heads, d]: numbers i and i + n/2 turned by a[:, i], n = twice the angles' number."""
    h = a.shape[1]
    y = x.copy()
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :h], x[..., h:2 * h]
    y[..., :h] = u * c - v * s
    y[..., h:2 * h] = v * c + u * s
    return y


# ---- what a token sees -----------------------------------------------------------------------------------
def seen_in_chunk(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i // size == j // size) if size else j <= i


def seen_in_window(T, size):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i - j < size) if size else j <= i


# ---- mixers -----------------------------------------------------------------------------------------
def chunked_attention(x, w, m, eps):
    T = x.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (over_rms(x @ w["q"].T, eps) * w["q.norm"]).reshape(T, H, d)
    k = (over_rms(x @ w["k"].T, eps) * w["k.norm"]).reshape(T, G, d)
    v = (x @ w["v"].T).reshape(T, G, e)
    rot = m.get("rot") or {}
    if rot.get("dims"):
        a = angles(np.arange(T), rot["dims"], rot["base"], float((rot.get("scaling") or {}).get("factor", 1.0)))
        q, k = rotate_neighbours(q, a), rotate_neighbours(k, a)
    kv_of = np.arange(H) // (H // G)
    s = np.einsum("ihd,jhd->hij", q, k[:, kv_of]) * m["scale"]
    p = softmax_over(s, seen_in_chunk(T, int((m.get("mask") or {}).get("size", 0)))[None])
    o = np.einsum("hij,jhe->ihe", p, v[:, kv_of]).reshape(T, H * e)
    return (o * sigmoid(x @ w["g"].T)) @ w["o"].T


def latent_attention(x, w, m, eps):
    T = x.shape[0]
    H, d, r, e, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (x @ w["q"].T).reshape(T, H, d + r)
    down = x @ w["dkv"].T
    c = over_rms(down[:, :rank], eps) * w["dkv.norm"]
    qn, qr, kr = q[..., :d], q[..., d:], down[:, None, rank:]
    rot = m.get("rot") or {}
    if rot.get("dims"):
        a = angles(np.arange(T), rot["dims"], rot["base"], float((rot.get("scaling") or {}).get("factor", 1.0)))
        qr, kr = rotate_halves(qr, a), rotate_halves(kr, a)
    kn = (c @ w["uk"].T).reshape(T, H, d)
    v = (c @ w["uv"].T).reshape(T, H, e)
    s = (np.einsum("ihd,jhd->hij", qn, kn) + np.einsum("ihd,jd->hij", qr, kr[:, 0])) * m["scale"]
    p = softmax_over(s, seen_in_window(T, int((m.get("mask") or {}).get("size", 0)))[None])
    return np.einsum("hij,jhe->ihe", p, v).reshape(T, H * e) @ w["o"].T


# ---- feed-forward --------------------------------------------------------------------------------------
def squared_relu_ff(x, w):
    u = np.maximum(x @ w["up"].T, 0.0)
    return (u * u) @ w["down"].T


# ---- the model ---------------------------------------------------------------------------------------
def owner_of(cfg: dict, i: int) -> int:
    """The layer whose tensors layer i runs."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = int(cfg["layers"][i]["weights_of"])
    return i


def run_layer(x, w, spec, eps):
    mix = {"attention": chunked_attention, "latent_attention": latent_attention}[spec["type"]]
    x = x + norm_around_one(mix(x, sub(w, "mix"), spec["mixer"], eps), w["norm1"], eps)
    if spec.get("mlp") is not None:
        x = x + norm_around_one(squared_relu_ff(x, sub(w, "mlp")), w["norm2"], eps)
    return x


def head(xn, w, a, cap):
    z = xn @ w.T * a
    return cap * np.tanh(z / cap) if cap else z


def forward(cfg: dict, w: dict, tokens, streams: list | None = None) -> np.ndarray:
    """Logits [T, vocab] of one sequence; `streams` collects the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i in range(len(cfg["layers"])):
        j = owner_of(cfg, i)
        x = run_layer(x, sub(w, f"l{j}"), cfg["layers"][j], eps)
        if streams is not None:
            streams.append(x.copy())
    return head(norm_around_one(x, w["final.norm"], eps), w["head"], float(cfg.get("logit_scale", 1.0)),
                float(cfg.get("logit_softcap") or 0.0))
