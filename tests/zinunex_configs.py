"""Tiny Zinunex configurations for tests.  They differ in every size and option: the order of layer types, heads and key heads
(one head, all heads on one key head, as many key heads as heads), head sizes that are multiples of 16 or not, value sizes of
the latent layers equal to the key's or not, rotated parts with and without scaled frequencies, cached rows of 64 and 128, rows
that are padded to those, and rows the tensor-core kernels decline, windows shorter and longer than a page or none, layers that
read an earlier layer's cache with a window shorter than, longer than and equal to its own (several readers of one source, a reader
right behind it or far behind), partial and whole half-split rotations, groups or none, one expert per token or many, groups of one
expert, a shared expert of the experts' size, of another size or none, layers without feed-forward, side inputs of 1 to 40 entries or
none, widths and vocabularies that are no power of two and no multiple of 8."""


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, window=None, base=10000.0, scaling=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def attention(heads, kv, dim, scale, rot_dims=None, base=10000.0, factor=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}
    if rot_dims != 0:
        m["rot"] = {"base": base, "dims": dim if rot_dims is None else rot_dims}
        if factor is not None:
            m["rot"]["scaling"] = {"factor": factor}
    return {"type": "attention", "mixer": m}


def moe(experts, top, ff, scale=1.0, groups=None, shared=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def with_mlp(layer, mlp):
    return dict(layer, mlp=mlp)


YARN = (4.0, 64, 8.0, 1.0)

ZIN_A = {
    "architecture": "Zinunex", "vocab": 211, "width": 64, "norm": {"eps": 1e-5}, "token_side": {"dim": 12},
    "layers": [
        with_mlp(attention(4, 2, 16, 0.3, factor=3.0), moe(6, 2, 24, 1.7, groups=(3, 2), shared=24)),
        with_mlp(latent(3, 16, 8, 12, 24, 0.25, window=9, base=300.0, scaling=YARN), moe(4, 1, 16, shared=20)),
        with_mlp(latent(2, 8, 8, 20, 24, 0.4, window=21, base=300.0, scaling=YARN, kv_from=1), None),
        with_mlp(attention(3, 3, 8, 0.5, rot_dims=4, base=50.0), moe(8, 3, 16, 2.5, groups=(4, 2))),
        with_mlp(latent(5, 12, 8, 8, 24, 0.3, window=4, base=300.0, scaling=YARN, kv_from=1), moe(3, 3, 8, 0.5, groups=(3, 3), shared=30)),
    ]}

ZIN_B = {
    "architecture": "Zinunex", "vocab": 301, "width": 52, "norm": {"eps": 1e-6}, "token_side": {"dim": 7},
    "layers": [
        with_mlp(latent(5, 12, 12, 20, 28, 0.2, window=70, base=500000.0), moe(5, 5, 12, 2.0)),
        with_mlp(attention(6, 1, 24, 0.2, rot_dims=10, base=1000.0, factor=0.5), moe(10, 4, 20, 1.0, groups=(2, 1), shared=36)),
        with_mlp(latent(1, 7, 12, 5, 28, 0.5, base=500000.0, kv_from=0), None),
    ]}

ZIN_C = {
    "architecture": "Zinunex", "vocab": 512, "width": 128, "norm": {"eps": 1e-6}, "token_side": {"dim": 40},
    "layers": [
        with_mlp(latent(4, 32, 16, 32, 48, 0.14, window=48, base=10000.0, scaling=(8.0, 512, 32.0, 1.0)), moe(8, 2, 64, 1.5, groups=(2, 1), shared=64)),
        with_mlp(attention(4, 2, 64, 0.125, base=20000.0, factor=4.0), moe(12, 3, 32, 1.0, groups=(4, 3), shared=128)),
        with_mlp(latent(8, 32, 16, 48, 48, 0.14, window=48, base=10000.0, scaling=(8.0, 512, 32.0, 1.0), kv_from=0), moe(8, 3, 32, 2.0)),
        with_mlp(attention(8, 1, 128, 0.09, rot_dims=64, base=500000.0), moe(8, 2, 64, 1.0, groups=(4, 2), shared=40)),
    ]}

ZIN_D = {
    "architecture": "Zinunex", "vocab": 500, "width": 128, "norm": {"eps": 1e-5}, "token_side": {"dim": 16},
    "layers": [
        with_mlp(latent(16, 16, 32, 16, 60, 0.14, window=33, base=1000.0, scaling=(2.0, 100, 4.0, 0.5)), moe(16, 4, 24, 1.0, groups=(8, 3), shared=64)),
        with_mlp(latent(12, 24, 8, 40, 32, 0.2, window=130, base=80.0), moe(4, 2, 48, 1.0, shared=48)),
        with_mlp(latent(6, 20, 32, 24, 60, 0.14, window=150, base=1000.0, scaling=(2.0, 100, 4.0, 0.5), kv_from=0), None),
        with_mlp(attention(2, 2, 64, 0.125), moe(8, 2, 64, 1.0, groups=(2, 2), shared=16)),
        with_mlp(latent(12, 8, 8, 8, 32, 0.3, window=20, base=80.0, kv_from=1), moe(8, 1, 64, 3.0, groups=(4, 1), shared=64)),
    ]}

ZIN_E = {
    "architecture": "Zinunex", "vocab": 97, "width": 40, "norm": {"eps": 3e-6},
    "layers": [
        with_mlp(attention(1, 1, 12, 0.4, rot_dims=0), None),
        with_mlp(latent(1, 7, 0, 5, 9, 0.5, window=1), moe(3, 2, 8, 3.0, groups=(1, 1), shared=11)),
        with_mlp(attention(10, 1, 20, 0.3, base=30.0, factor=2.0), moe(1, 1, 16, 1.0, shared=16)),
    ]}

ALL = {"A": ZIN_A, "B": ZIN_B, "C": ZIN_C, "D": ZIN_D, "E": ZIN_E}
PAGE = {"A": 4, "B": 8, "C": 16, "D": 16, "E": 16}
