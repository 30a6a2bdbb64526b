"""Small Zafilix configurations for the tests.  They differ from one another in every size and constant: width,
vocabulary, eps, embedding scale, logit scale and cap (also absent), the order of the layers, which layers run another
layer's tensors (a neighbour's, a far one's, one that borrows itself), which have a feed-forward, head counts and
grouping (one key head for all, a key head per head), key and value sizes (equal, smaller, larger, no multiples of 8),
the rotated part of a head (none, part, all), the positions' scaling (also 1 and absent), chunks and windows (one
position, a few, a cache page, more than one, none), latents (multiples of 32, others) and their rotated parts."""


def rotation(dims, base, factor):
    r = {"dims": dims, "base": base}
    if factor is not None:
        r["scaling"] = {"factor": factor}
    return r


def att(heads, kv_heads, dim, vdim, scale, rot_dims, base, factor, size):
    a = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot_dims is not None:
        a["rot"] = rotation(rot_dims, base, factor)
    if size:
        a["mask"] = {"size": size}
    return a


def lat(heads, dim, rot_dim, vdim, kv_rank, scale, base, size, rot_dims=None, factor=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": rotation(rot_dim if rot_dims is None else rot_dims, base, factor)}
    if size:
        m["mask"] = {"size": size}
    return m


def layer(mixer, ff, weights_of=None):
    e = {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer,
         "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def model(vocab, width, eps, layers, emb=None, a=None, cap=None):
    c = {"architecture": "Zafilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if emb is not None:
        c["embedding"] = {"scale": emb}
    if a is not None:
        c["logit_scale"] = a
    if cap is not None:
        c["logit_softcap"] = cap
    return c


# heads of 64 (the tcgen05 prompt attention, the decode attention that prepares its own rows), a chunk shorter than a
# page and one that is no divisor of a page; one layer borrowed twice, once through a layer that borrows itself
_A0 = att(4, 2, 64, 64, 0.11, 64, 10000.0, 3.0, 40)
_A1 = lat(5, 24, 16, 40, 64, 0.15, 5000.0, 70)
Z_A = model(210, 80, 1e-5, [layer(_A0, 112), layer(_A1, 112), layer(_A0, 112, 0), layer(_A1, 72), layer(_A0, 112, 2)], 7.0, 0.4, 11.0)

# the latent layer first, no feed-forward in one layer, heads of 128 on one key head, a chunk of exactly a page
_B0 = lat(3, 32, 32, 64, 128, 0.2, 20000.0, 9)
_B1 = att(3, 1, 128, 128, 0.07, 128, 1e6, 1.0, 64)
Z_B = model(140, 72, 1e-6, [layer(_B0, None), layer(_B1, 96), layer(_B0, None, 0), layer(att(6, 6, 32, 32, 0.2, 16, 300.0, None, 100), 40)],
            4.0, 1.5, 6.0)

# no size on the 16-byte grid, no rotation in one layer, a chunk of one position, a window of one, no cap
Z_C = model(97, 42, 1e-4, [layer(att(5, 5, 12, 20, 0.3, None, None, None, 1), 30), layer(lat(3, 10, 6, 14, 20, 0.3, 100.0, 1), 26),
                           layer(att(3, 1, 22, 10, 0.25, 10, 5000.0, 2.5, 33), None), layer(lat(2, 18, 4, 9, 33, 0.22, 900.0, 50), 18),
                           layer(att(2, 2, 26, 26, 0.2, 0, 10000.0, 2.0, 0), 22)])

# unequal head sizes that are cached at the wider one, partial rotation, chunks of several pages, no windows; a
# borrowed neighbour, and a layer that comes before the one whose tensors it runs
_D1 = att(8, 4, 64, 32, 0.13, 32, 50000.0, 2.0, 150)
_D3 = lat(6, 48, 64, 32, 256, 0.1, 1e5, 0)
Z_D = model(300, 96, 1e-5, [layer(_D3, 88, 3), layer(_D1, 64), layer(_D1, 64, 1), layer(_D3, 88),
                            layer(att(4, 1, 48, 96, 0.16, 48, 1000.0, 1.5, 130), 120)], 9.5, 1.0, 30.0)

# more latent numbers than a tile of 64 rows takes, an odd rotated tail that passes unchanged, four heads a key head of 64
Z_E = model(64, 64, 1e-5, [layer(lat(2, 16, 48, 24, 288, 0.2, 700.0, 65, rot_dims=20, factor=2.0), 48),
                           layer(att(8, 2, 64, 64, 0.1, 64, 10000.0, None, 96), 56),
                           layer(att(2, 2, 64, 64, 0.1, 24, 400.0, 5.0, 7), 56)], 3.0, 0.7, 9.0)

ALL = {"A": Z_A, "B": Z_B, "C": Z_C, "D": Z_D, "E": Z_E}


def random_config(rng) -> dict:
    """A configuration drawn at random: layer count and order, borrowed tensors, every size (also off the 8-number grid),
    chunks and windows around the page and tile borders or none, the rotated part, which layers have a feed-forward."""
    def pick(xs):
        return xs[int(rng.integers(0, len(xs)))]

    def reach():
        return 0 if rng.random() < 0.1 else pick([1, 2, 7, 31, 32, 33, 63, 64, 65, 100, 127, 128, 129, 200])

    def attention():
        kv = pick([1, 1, 2, 2, 3, 4])
        d = pick([8, 16, 24, 32, 48, 64, 96, 128, 20, 36, 64, 128])
        return att(kv * pick([1, 2, 3, 4]), kv, d, pick([d, d, 16, 32, 40, 64, 128, 12]), float(rng.uniform(0.05, 0.4)),
                   None if rng.random() < 0.1 else pick([d, d, d // 2, d // 4]) // 2 * 2, pick([100.0, 10000.0, 5e5]),
                   pick([None, 1.0, 2.0, 1.5]), reach())

    def latent():
        r = pick([16, 16, 32, 64, 8, 10, 6])
        return lat(pick([1, 2, 3, 6, 10]), pick([8, 16, 32, 64, 20, 100]), r, pick([8, 16, 32, 64, 33]),
                   pick([32, 64, 96, 128, 256, 20, 50]), float(rng.uniform(0.05, 0.4)), pick([100.0, 10000.0, 5e5]), reach(),
                   rot_dims=pick([r, r, r, r // 2]) // 2 * 2, factor=pick([None, None, 2.0]))

    layers = []
    for i in range(int(rng.integers(1, 6))):
        if i and rng.random() < 0.35:
            j = int(rng.integers(0, i))
            layers.append(dict(layers[j], weights_of=j))
        else:
            layers.append(layer(attention() if rng.random() < 0.5 else latent(), pick([24, 64, 100, 256, 30, None])))
    return model(pick([64, 101, 500]), pick([32, 40, 48, 64, 72, 96, 128, 192, 50, 84]), pick([1e-5, 1e-6]), layers,
                 pick([None, 4.0, 9.0]), pick([None, 0.5, 2.0]), pick([None, 5.0, 30.0]))
