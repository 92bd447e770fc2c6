"""Modinex: which parts each layer has, from its typed config.

Embedding "embed" plus the position's row of "pos".  Layer i (tensors "l<i>."): the sandwich arrangement (norms "norm1" /
"norm2" before the sublayers, "norm1b" / "norm2b" on their outputs, all in groups) around a mixer "mix." and, where the layer
has one, a feed-forward "mlp.".  Mixers: "attention" (chunked attention with sigmoid weights: "q", "k", "v", "o", head norms
"q.norm" / "k.norm", a number per head "pb") and "gla" (gated linear attention: "q", "k", "v", "g", "o", "norm", the decay's
"a1", "a2", "a2.b").  Feed-forward "dense" ("up", "up.b", "down", "down.b", tanh gelu).  Final norm "final.norm" (in groups
too), head "head".
"""
from __future__ import annotations

from ..config.modinex import ModinexConfig, parse_modinex_config
from ..config.registry import Architecture, register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 20         # without a position table the design states no limit
DEFAULT_RANK = 16               # inner size of the decay's two-step projection when neither a tensor nor the config gives it


def modinex_model_spec(cfg: ModinexConfig, tensor_shapes=None) -> ModelSpec:
    """tensor_shapes: name -> shape of the model folder's tensors, when known: the position table has as many rows as the
    stored tensor "pos" (which config.json's max_positions states too), the decay's inner size is that of "<layer>.mix.a1"."""
    W = cfg.width
    shapes = tensor_shapes or {}
    n_positions = cfg.max_positions
    if tensor_shapes is not None:
        stored = tensor_shapes.get("pos")
        n_positions = int(stored[0]) if stored else None

    def norm(name):
        return PartSpec("rmsnorm", {"width": W, "eps": cfg.eps, "name": name, "groups": cfg.groups})

    layers = []
    for i, L in enumerate(cfg.layers):
        prefix = f"l{i}."
        m = L.mixer
        if L.type == "attention":
            position = PartSpec("none")
            if m.rot_dims:
                position = PartSpec("rope_neox", {"head_dim": m.dim, "n_rot": m.rot_dims, "theta": m.rot_base})
            mixer = PartSpec("attention", {
                "hidden": W, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_head_dim": m.vdim,
                "scale": m.scale, "chunk": m.chunk, "weights": "sigmoid", "qk_norm": True, "eps": cfg.eps, "position": position,
                "names": {k: "mix." + v for k, v in {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm",
                                                     "score_bias": "pb"}.items()}})
        else:
            a1 = shapes.get(prefix + "mix.a1")
            mixer = PartSpec("gated_linear_attention", {
                "hidden": W, "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau,
                "decay_rank": int(a1[0]) if a1 else (m.rank or DEFAULT_RANK), "eps": cfg.eps,
                "names": {k: "mix." + v for k, v in {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "a1": "a1",
                                                     "a2": "a2", "a2_bias": "a2.b"}.items()}})
        ff = None
        if L.mlp is not None:
            ff = PartSpec("dense", {"hidden": W, "ff": L.mlp.ff, "act": "gelu_tanh", "bias": True,
                                    "names": {"up": "mlp.up", "down": "mlp.down", "up_bias": "mlp.up.b", "down_bias": "mlp.down.b"}})
        params = {"mixer_out_norm": norm("norm1b")}
        if ff is not None:
            params["feed_forward_out_norm"] = norm("norm2b")
        layers.append(LayerSpec(prefix=prefix, mixer=mixer, feed_forward=ff, mixer_norm=norm("norm1"),
                                feed_forward_norm=norm("norm2") if ff is not None else None, block="sandwich_residual", params=params))
    positions = {"name": "pos", "rows": n_positions} if n_positions else None
    return ModelSpec(
        architecture="Modinex", vocab_size=cfg.vocab, hidden_size=W,
        embedding=PartSpec("token_table", {"vocab": cfg.vocab, "width": W, "name": "embed", "position_table": positions}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm"), head=PartSpec("linear", {"vocab": cfg.vocab, "width": W, "name": "head"}),
        max_positions=n_positions or MAX_POSITIONS, eos_token_ids=())


register_architecture(Architecture(name="Modinex", model_types=("modinex",),
                                   parse_config=parse_modinex_config, model_spec=modinex_model_spec), replace=True)
