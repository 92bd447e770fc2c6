"""Zinunex: which parts each layer has, from its typed config.

Embedding "embed".  Layer i (tensors "l<i>."): the pre-norm arrangement around a mixer "mix." ("norm1") and a routed feed-forward
"mlp." ("norm2"), then the layer's token input ("side.gate", "side.proj", "side.norm"; its columns of the table "side.embed").
Mixers: "latent_attention" ("q", "dkv", "dkv.norm", "uk", "uv", "o"; the cache keeps the normed latent and one rotated key part per
position; a layer with kv_from has no "dkv" and reads the cache of the schedule entry that makes it) and "attention" ("q", "k",
"sink", "o"; keys before the rotation are the values).  Feed-forward: "router", "correction", experts "e<j>.up" / ".down",
"shared.up" / ".down" / ".sg".  Final norm "final.norm", head "head".
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.zinunex import ZinunexConfig, parse_zinunex_config
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

MAX_POSITIONS = 1 << 20         # the design states no limit; rotation angles are 32-bit products


def _latent(W, m, eps):
    position = PartSpec("none")
    if m.rot_dims:
        sc = m.rot_scaling
        position = PartSpec("rope_interleaved", {
            "head_dim": m.rot_dim, "n_rot": m.rot_dims, "theta": m.rot_base,
            "scaling": None if sc is None else {"factor": sc.factor, "original": sc.original, "fast": sc.fast, "slow": sc.slow}})
    return PartSpec("latent_attention", {
        "hidden": W, "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "q_rank": None, "kv_rank": m.kv_rank, "rot_dim": m.rot_dim,
        "position": position, "scale": m.scale, "eps": eps, "window": m.window, "reads": m.kv_from is not None, "pad_row": True,
        "names": {k: "mix." + v for k, v in {"q": "q", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "o": "o"}.items()}})


def _attention(W, m):
    position = PartSpec("none")
    if m.rot_dims:
        position = PartSpec("rope_neox", {"head_dim": m.dim, "n_rot": m.rot_dims, "theta": m.rot_base, "linear_scaling": m.rot_factor})
    return PartSpec("attention", {
        "hidden": W, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "scale": m.scale, "qk_norm": False,
        "v_from_k": True, "sink": "learned", "position": position,
        "names": {"q": "mix.q", "k": "mix.k", "o": "mix.o", "sink": "mix.sink"}})


def _routed(W, r):
    shared = None
    if r.shared_ff is not None:
        shared = {"ff": r.shared_ff, "names": {"up": "mlp.shared.up", "down": "mlp.shared.down"}, "factor": "mlp.shared.sg"}
    return PartSpec("routed_experts", {
        "hidden": W, "ff": r.ff, "experts": r.experts, "top": r.top, "score": "sigmoid", "renormalise": False, "weight_scale": r.scale,
        "groups": r.groups, "keep": r.keep, "group_score": "top2", "correction": True, "weight_on": "output", "gated": False,
        "act": "relu2", "shared": shared,
        "names": {"router": "mlp.router", "correction": "mlp.correction", "up": "mlp.e{e}.up", "down": "mlp.e{e}.down"}})


def zinunex_model_spec(cfg: ZinunexConfig) -> ModelSpec:
    W, n = cfg.width, len(cfg.layers)
    layers, schedule = [], []
    for i, L in enumerate(cfg.layers):
        mixer = _latent(W, L.mixer, cfg.eps) if L.type == "latent_attention" else _attention(W, L.mixer)
        ff = ff_norm = None
        if L.mlp is not None:
            ff = _routed(W, L.mlp)
            ff_norm = PartSpec("rmsnorm", {"width": W, "eps": cfg.eps, "name": "norm2"})
        params = {}
        if cfg.side_dim is not None:
            params["after"] = PartSpec("token_side_input", {
                "width": W, "dim": cfg.side_dim, "index": i, "columns": n * cfg.side_dim, "vocab": cfg.vocab, "eps": cfg.eps,
                "table": "side.embed"})
        layers.append(LayerSpec(prefix=f"l{i}.", mixer=mixer, feed_forward=ff,
                                mixer_norm=PartSpec("rmsnorm", {"width": W, "eps": cfg.eps, "name": "norm1"}),
                                feed_forward_norm=ff_norm, params=params))
        schedule.append(ScheduleEntry(i, cache_from=getattr(L.mixer, "kv_from", None)))
    return ModelSpec(
        architecture="Zinunex", vocab_size=cfg.vocab, hidden_size=W,
        embedding=PartSpec("token_table", {"vocab": cfg.vocab, "width": W, "name": "embed"}),
        layers=tuple(layers), schedule=tuple(schedule),
        final_norm=PartSpec("rmsnorm", {"width": W, "eps": cfg.eps, "name": "final.norm"}),
        head=PartSpec("linear", {"vocab": cfg.vocab, "width": W, "name": "head"}),
        max_positions=MAX_POSITIONS, eos_token_ids=())


register_architecture(Architecture(name="Zinunex", model_types=("zinunex",),
                                   parse_config=parse_zinunex_config, model_spec=zinunex_model_spec), replace=True)
