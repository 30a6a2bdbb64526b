"""Small Nolapel configurations for the tests.  They differ from one another in every size and constant: width,
vocabulary, eps, the pair table's buckets and factors (also absent), the cap on the logits (also absent), the order of the
layers, the looped range (the first layers, the last, one layer, all, none; one pass and several), which layers have
a feed-forward, experts, choices and shared expert (also absent), head counts and grouping (one key head for all, a key
head per head, counts that are no power of two), key and value sizes (equal, unequal, no multiples of 8), the rotated part
of a head (none, part, all), taps (also one), windows (one position, a few, a cache page, more than one, none), query
temperatures (also absent), scales of the two mixers side by side (also 1), groups of the state-space layer."""


def att(heads, kv_heads, dim, conv, scale, size=0, temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def left(heads, kv_heads, dim, vdim, scale, rot_dims=None, base=10000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot_dims is not None:
        m["rot"] = {"dims": rot_dims, "base": base}
    return m


def par(left_mixer, heads, dim, a=None, b=None):
    m = {"left": left_mixer, "right": {"heads": heads, "dim": dim}}
    if a is not None:
        m["left_scale"] = a
    if b is not None:
        m["right_scale"] = b
    return m


def ssm(heads, vdim, state, groups, norm_groups, conv):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp):
    return {"type": "parallel" if "left" in mixer else ("mamba2" if "state" in mixer else "attention"), "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, layers, pairs=None, loop=None, cap=None):
    c = {"architecture": "Nolapel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if pairs is not None:
        c["embedding"] = {"bigram": {"buckets": pairs[0], "mul_prev": pairs[1], "mul_cur": pairs[2]}}
    if loop is not None:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    if cap is not None:
        c["logit_softcap"] = cap
    return c


# heads of 64 (the tcgen05 prompt attention, the decode attention that prepares its own rows), the first two layers looped
N_A = model(220, 80, 1e-5, [
    layer(att(8, 2, 64, 4, 0.12, 40, (0.4, 16)), moe(6, 2, 48, 32)),
    layer(par(left(4, 2, 64, 64, 0.13, 64), 3, 16, 0.7, 1.3), moe(5, 1, 40, 24)),
    layer(ssm(6, 16, 24, 3, 2, 3), moe(4, 3, 32, 56))], (97, 31, 5), (0, 2, 2), 9.0)

# heads of 128 and 32, three heads on one key head, no feed-forward in one layer, one layer looped three times
N_B = model(150, 72, 1e-6, [
    layer(ssm(4, 24, 16, 1, 4, 4), None),
    layer(par(left(3, 1, 128, 128, 0.08, 32, 500.0), 2, 32, 1.0, 0.5), moe(9, 4, 24)),
    layer(att(6, 6, 32, 2, 0.2, 64, (0.2, 50)), moe(8, 1, 64, 48)),
    layer(att(2, 1, 128, 5, 0.09, 100), moe(4, 2, 16, 16))], (1009, 7, 1), (1, 2, 3), 20.0)

# no size on the 16-byte grid, five heads, one tap, a window of one position, no rotation, no pair table, no cap
N_C = model(101, 42, 1e-4, [
    layer(par(left(5, 5, 12, 20, 0.3), 3, 10), moe(3, 3, 10, 14)),
    layer(att(5, 1, 22, 1, 0.25, 1), moe(7, 2, 18)),
    layer(ssm(5, 6, 10, 5, 3, 2), moe(2, 1, 22, 6)),
    layer(att(3, 3, 18, 3, 0.25, 33, (1.0, 7)), None)])

# unequal head sizes stored at a wider one, part of a head rotated, every layer looped, heads of 48 and 80 widened
N_D = model(300, 96, 1e-5, [
    layer(att(4, 4, 48, 3, 0.15, 130, (0.25, 33)), moe(16, 5, 24, 40)),
    layer(ssm(8, 20, 32, 4, 1, 5), moe(4, 4, 48)),
    layer(par(left(8, 4, 80, 48, 0.1, 20, 1000.0), 4, 24, 1.2, 0.6), moe(12, 1, 56, 72))], (12, 3, 2), (0, 3, 2), 30.0)

# no window, heads of 200, a pair table of one bucket, the last layer looped once, no feed-forward anywhere
N_E = model(64, 64, 1e-5, [
    layer(att(4, 2, 200, 4, 0.07, 0, (0.5, 3)), None),
    layer(par(left(16, 1, 64, 64, 0.12, 64, 1e6), 1, 64, 0.4, 0.9), None),
    layer(att(12, 3, 64, 3, 0.12, 7), None)], (1, 0, 1), (2, 3, 1), 4.0)

ALL = {"A": N_A, "B": N_B, "C": N_C, "D": N_D, "E": N_E}


def random_config(rng) -> dict:
    """A configuration drawn at random: layer count and order, the looped range, every size (also off the 8-number grid),
    windows around the page and tile borders or none, taps, temperatures, which layers have a feed-forward."""
    def pick(xs):
        return xs[int(rng.integers(0, len(xs)))]

    def attention():
        kv = pick([1, 1, 2, 2, 3, 4])
        size = 0 if rng.random() < 0.1 else pick([1, 2, 7, 31, 32, 33, 63, 64, 65, 100, 127, 128, 129, 200])
        return att(kv * pick([1, 2, 3, 4]), kv, pick([8, 16, 24, 32, 48, 64, 96, 128, 20, 36, 64, 130]), pick([1, 2, 3, 4, 5, 7]),
                   float(rng.uniform(0.05, 0.3)), size, None if rng.random() < 0.2 else (float(rng.uniform(0.05, 0.6)), pick([1, 5, 16, 64, 100])))

    def side_by_side():
        kv, d = pick([1, 1, 2, 3, 4]), pick([8, 16, 24, 32, 48, 64, 96, 128, 20, 64, 136])
        lm = left(kv * pick([1, 2, 3, 4]), kv, d, pick([d, d, d, 16, 40, 64]), float(rng.uniform(0.05, 0.3)),
                  None if rng.random() < 0.1 else pick([d, d, d // 2]) // 2 * 2, pick([100.0, 10000.0, 5e5]))
        return par(lm, pick([1, 2, 3, 4]), pick([8, 16, 32, 64, 12, 10]), pick([None, 0.7, 1.2]), pick([None, 0.5, 1.1]))

    def state_space():
        g, e = pick([1, 2, 3]), pick([8, 16, 32, 20])
        h = g * pick([1, 2, 4])
        return ssm(h, e, pick([8, 16, 32, 64, 20]), g, pick([1, h]), pick([1, 2, 3, 4, 6]))

    def experts():
        if rng.random() < 0.2:
            return None
        n = pick([2, 4, 7, 12])
        return moe(n, int(rng.integers(1, min(n, 4) + 1)), pick([16, 32, 40, 18]), pick([None, 24, 48, 20]))

    layers = [layer(pick([attention, side_by_side, state_space])(), experts()) for _ in range(int(rng.integers(1, 5)))]
    loop = None
    if rng.random() < 0.7:
        a = int(rng.integers(0, len(layers)))
        loop = (a, int(rng.integers(a, len(layers))) + 1, pick([1, 2, 3]))
    return model(pick([64, 101, 500]), pick([32, 40, 48, 64, 72, 96, 128, 192, 50, 84]), pick([1e-5, 1e-6]), layers,
                 None if rng.random() < 0.15 else (pick([1, 13, 211, 4096]), pick([0, 3, 131]), pick([1, 17, 0])), loop, pick([None, 5.0, 30.0]))
