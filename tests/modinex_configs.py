"""Tiny Modinex configurations for tests.  They differ in every size and option: the order of layer types, feed-forwards on either
type or none, heads and key heads, head sizes that are multiples of 16 or not, value sizes equal to the key size, larger and
smaller, rotation over the whole head, a part of it or none, stretches shorter and longer than a page, of one position, or no
mask, decay powers 1 and others, decay inner sizes that are no multiple of 8, norms in one group, in a few and in many, widths
and vocabularies that are no power of two and no multiple of 8."""


def attention(heads, kv, dim, vdim, scale, size=None, rot=None, base=10000.0):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size}
    if rot is not None:
        m["rot"] = {"base": base, "dims": rot}
    return {"type": "attention", "mixer": m}


def gla(heads, dim, vdim, tau, rank):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}}


def with_mlp(layer, ff):
    return dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


MOD_A = {
    "architecture": "Modinex", "vocab": 211, "width": 72, "max_positions": 700, "norm": {"eps": 1e-5, "groups": 3},
    "layers": [
        with_mlp(attention(6, 2, 12, 20, 0.35, size=9, rot=8, base=300.0), 40),
        with_mlp(gla(3, 8, 24, 4.0, 5), None),
        with_mlp(attention(2, 1, 16, 16, 0.25, size=21, rot=16), None),
        with_mlp(gla(2, 20, 12, 1.0, 12), 30),
    ]}

MOD_B = {
    "architecture": "Modinex", "vocab": 301, "width": 52, "max_positions": 900, "norm": {"eps": 1e-6},
    "layers": [
        with_mlp(gla(2, 24, 33, 9.0, 3), 44),
        with_mlp({"type": "attention", "mixer": {"heads": 3, "dim": 24, "scale": 0.2, "mask": {"size": 70}}}, 64),
        with_mlp(gla(1, 40, 70, 30.0, 20), None),
        with_mlp(attention(4, 4, 8, 12, 0.4), 20),
    ]}

MOD_C = {
    "architecture": "Modinex", "vocab": 480, "width": 128, "max_positions": 1200, "norm": {"eps": 1e-6, "groups": 8},
    "layers": [
        with_mlp(attention(4, 2, 48, 96, 0.14, size=48, rot=32, base=500000.0), 160),
        with_mlp(gla(2, 64, 96, 12.0, 8), 96),
        with_mlp(attention(8, 1, 32, 16, 0.2, size=200, rot=32), None),
        with_mlp(gla(3, 16, 48, 5.0, 16), None),
    ]}

MOD_D = {
    "architecture": "Modinex", "vocab": 500, "width": 192, "max_positions": 1100, "norm": {"eps": 1e-5, "groups": 2},
    "layers": [
        with_mlp(gla(4, 128, 32, 16.0, 24), None),
        with_mlp(attention(16, 2, 64, 128, 0.125, size=128, rot=64), 256),
        with_mlp(gla(1, 32, 208, 2.0, 16), None),
        with_mlp(attention(12, 1, 112, 64, 0.1, size=75, rot=48), None),
    ]}

MOD_E = {
    "architecture": "Modinex", "vocab": 97, "width": 40, "max_positions": 600, "norm": {"eps": 3e-6, "groups": 5},
    "layers": [
        with_mlp(attention(1, 1, 7, 5, 0.5, size=1), 16),
        with_mlp(gla(1, 7, 5, 1.0, 1), 24),
        with_mlp(gla(2, 136, 20, 3.0, 4), None),
        with_mlp(attention(5, 5, 10, 3, 0.6, size=17, rot=10, base=50.0), 8),
    ]}

ALL = {"A": MOD_A, "B": MOD_B, "C": MOD_C, "D": MOD_D, "E": MOD_E}
PAGE = {"A": 4, "B": 8, "C": 16, "D": 32, "E": 16}
