"""Dinutar as data: which parts, with which constants, under which tensor names.

Tensor names: ``embed`` (which is the output head too), ``bigram``, ``embed.norm``, ``final.norm``, and per layer ``l<i>.``:
``norm1``, ``ls1`` (and with a feed-forward ``norm2``, ``ls2``), ``mix.*`` (q, k, v, g, o of a retention layer; q, dkv,
dkv.norm, uk, uv, o of a latent attention layer) and ``mlp.up``, ``mlp.down``.  A layer that reads another layer's cached rows
has no dkv tensors and runs on that layer's cache lane without writing it; every other layer has a lane of its own, and the
embedding has one for the previous token.
"""
from __future__ import annotations

from ..config.dinutar import DinutarConfig, LatentMixer, RetentionMixer, Rotation
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

LAYER_NAMES = {"mixer_norm": "norm1", "feed_forward_norm": "norm2", "mixer_scale": "ls1", "feed_forward_scale": "ls2",
               "mixer": "mix.", "feed_forward": "mlp."}


def _position(rot: Rotation, head_dim: int) -> PartSpec:
    if not rot.dims:
        return PartSpec("none", {})
    params = {"head_dim": head_dim, "theta": rot.base, "rot_dim": rot.dims}
    if rot.factor is not None:
        params.update({"factor": rot.factor, "original": rot.original, "fast": rot.fast, "slow": rot.slow})
    return PartSpec("yarn_rope", params)


def _mixer(cfg: DinutarConfig, m) -> PartSpec:
    if isinstance(m, RetentionMixer):
        return PartSpec("retention", {"hidden_size": cfg.width, "n_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim,
                                      "decay": tuple(m.decay), "eps": cfg.norm_eps, "position": _position(m.rot, m.dim)})
    if isinstance(m, LatentMixer):
        names = {"q": "q", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "o": "o"}
        return PartSpec("latent_attention", {
            "hidden_size": cfg.width, "n_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "q_rank": 0, "kv_rank": m.kv_rank,
            "softmax_scale": m.scale, "eps": cfg.norm_eps, "rot_dim": m.rot_dim,
            "position": _position(m.rot, m.rot_dim) if m.rot_dim else None, "own_kv": m.kv_from is None, "names": names})
    raise ValueError(f"unknown mixer {type(m).__name__}")


def model_spec(cfg: DinutarConfig) -> ModelSpec:
    norm = PartSpec("rms_norm", {"hidden_size": cfg.width, "eps": cfg.norm_eps, "weight_name": "", "wide": True})
    block = PartSpec("post_norm_residual", {"hidden_size": cfg.width, "alpha": cfg.postln_alpha, "layer_scale": True})
    layers, schedule, lane_of = [], [], {}
    for i, layer in enumerate(cfg.layers):
        src = getattr(layer.mixer, "kv_from", None)
        if src is None:
            lane_of[i] = len(lane_of)
        elif src not in lane_of:
            raise ValueError(f"layer {i} reads the rows of layer {src}, which has none of its own before it")
        schedule.append(ScheduleEntry(layer=i, lane=lane_of[i if src is None else src], writes_cache=src is None))
        ffn = None
        if layer.mlp is not None:
            ffn = PartSpec("plain_ffn", {"hidden_size": cfg.width, "intermediate_size": layer.mlp.ff, "activation": "relu2",
                                         "names": {"up": "up", "down": "down"}})
        layers.append(LayerSpec(block=block, mixer=_mixer(cfg, layer.mixer), feed_forward=ffn, mixer_norm=norm,
                                feed_forward_norm=norm if ffn is not None else None, prefix=f"l{i}.", names=LAYER_NAMES))
    embedding = {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "scale": cfg.embedding_scale, "eps": cfg.norm_eps,
                 "weight_name": "embed", "bigram_name": "bigram", "norm_name": "embed.norm"}
    if cfg.bigram is not None:
        embedding.update({"buckets": cfg.bigram.buckets, "mul_prev": cfg.bigram.mul_prev, "mul_cur": cfg.bigram.mul_cur})
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("bigram_embedding", embedding), layers=layers, schedule=schedule, final_norm=norm,
        head=PartSpec("scaled_lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "scale": 1.0, "tied": True}),
        embedding_name="", final_norm_name="final.norm", head_name="", max_positions=0)
