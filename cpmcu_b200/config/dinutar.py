"""Typed configuration of the Dinutar architecture: a decoder of layers whose norm comes after the sum (the stream times a
constant plus the sublayer's output, scaled channel by channel, is normed), over a token embedding with a second table
that pairs of tokens index; the mixer is retention (a linear recurrence with one fixed decay per head and rotated queries
and keys) or attention over a cached latent with a rotated key part (some layers reading another layer's cached rows); the
feed-forward is dense with a squared relu and no gate, or absent.

``config.json`` is nested; every size and constant is read from it:

    architecture, vocab, width, postln_alpha, norm.eps, embedding = {scale, bigram: {buckets, mul_prev, mul_cur}},
    layers[i] = {type: "retention" | "latent_attention", mixer: {...}, mlp: {kind: "dense", ff} | null}
    retention:        mixer = {heads, dim, vdim, decay: [one number per head], rot: {dims, base}}
    latent_attention: mixer = {heads, dim, rot_dim, vdim, kv_rank, scale, kv_from (absent: a latent of its own),
                               rot: {dims, base, scaling: {factor, original, fast, slow}}}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple, Union

from .base import FieldReader

NAME = "Dinutar"


@dataclass(frozen=True)
class Rotation:
    dims: int                        # 0: no rotation
    base: float = 10000.0
    factor: Optional[float] = None   # None: frequencies as they are; else the slow ones are stretched
    original: float = 8192.0
    fast: float = 32.0
    slow: float = 1.0

    def to_json(self) -> Optional[Dict[str, Any]]:
        if not self.dims:
            return None
        out: Dict[str, Any] = {"dims": self.dims, "base": self.base}
        if self.factor is not None:
            out["scaling"] = {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}
        return out


@dataclass(frozen=True)
class RetentionMixer:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Rotation

    def to_json(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}
        if self.rot.dims:
            out["rot"] = self.rot.to_json()
        return out


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotation
    kv_from: Optional[int] = None    # the layer whose cached rows this one reads; None: its own

    def to_json(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim,
                               "kv_rank": self.kv_rank, "scale": self.scale}
        if self.rot.dims:
            out["rot"] = self.rot.to_json()
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class DenseMlp:
    ff: int

    def to_json(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int

    def to_json(self) -> Dict[str, Any]:
        return {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}


@dataclass(frozen=True)
class DinutarLayer:
    type: str
    mixer: Union[RetentionMixer, LatentMixer]
    mlp: Optional[DenseMlp]

    def to_json(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_json(), "mlp": self.mlp.to_json() if self.mlp else None}


def _rotation(mr: FieldReader, default_dims: int = 0) -> Rotation:
    rot = mr.child("rot")
    if rot is None:
        return Rotation(0)
    dims = rot.integer("dims", default_dims, minimum=0) or 0
    base = rot.number("base", 10000.0, positive=True) or 10000.0
    out = Rotation(dims, base)
    sc = rot.child("scaling")
    if sc is not None:
        out = Rotation(dims, base, sc.number("factor", positive=True), sc.number("original", positive=True),
                       sc.number("fast", 32.0, positive=True), sc.number("slow", 1.0, positive=True))
        sc.check(base != 1.0, "scaled frequencies need a base other than 1")
    rot.absorb(sc)
    rot.check(dims % 2 == 0, "'dims' must be even")
    mr.absorb(rot)
    return out


@dataclass(frozen=True)
class DinutarConfig:
    vocab: int
    width: int
    embedding_scale: float
    bigram: Optional[Bigram]
    postln_alpha: float
    norm_eps: float
    layers: Tuple[DinutarLayer, ...]
    architecture: str = NAME

    MIXER_TYPES = ("retention", "latent_attention")

    @staticmethod
    def _retention(mr: FieldReader) -> RetentionMixer:
        heads, dim = mr.integer("heads", minimum=1), mr.integer("dim", minimum=1)
        decay = mr.numbers("decay")
        rot = _rotation(mr)
        if heads is not None and decay is not None:
            mr.check(len(decay) == heads, f"'decay' must hold one number per head ({heads}), got {len(decay)}")
        if dim is not None:
            mr.check(rot.dims <= dim, f"'rot.dims' must be at most 'dim' {dim}")
        return RetentionMixer(heads, dim, mr.integer("vdim", dim, minimum=1), tuple(decay or ()), rot)

    @staticmethod
    def _latent(mr: FieldReader) -> LatentMixer:
        heads, dim = mr.integer("heads", minimum=1), mr.integer("dim", minimum=1)
        rot_dim = mr.integer("rot_dim", 0, minimum=0) or 0
        rot = _rotation(mr, rot_dim)
        m = LatentMixer(heads, dim, rot_dim, mr.integer("vdim", dim, minimum=1), mr.integer("kv_rank", minimum=1),
                        mr.number("scale"), rot, mr.integer("kv_from", None, minimum=0))
        mr.check(rot_dim % 2 == 0, "'rot_dim' must be even")
        mr.check(rot.dims == rot_dim, f"'rot.dims' {rot.dims} must equal 'rot_dim' {rot_dim}")
        return m

    @classmethod
    def from_dict(cls, data: Dict[str, Any]) -> "DinutarConfig":
        r = FieldReader(data)
        vocab = r.integer("vocab", minimum=1)
        width = r.integer("width", minimum=1)
        alpha = r.number("postln_alpha", 1.0)
        emb = r.child("embedding")
        scale, bigram = 1.0, None
        if emb is not None:
            scale = emb.number("scale", 1.0)
            br = emb.child("bigram")
            if br is not None:
                bigram = Bigram(br.integer("buckets", minimum=1), br.integer("mul_prev"), br.integer("mul_cur"))
            emb.absorb(br)
        r.absorb(emb)
        norm = r.child("norm")
        eps = norm.number("eps", positive=True) if norm is not None else None
        if norm is None:
            r.check(False, "required key 'norm' is missing")
        r.absorb(norm)
        raw_layers = data.get("layers")
        layers: List[DinutarLayer] = []
        if not isinstance(raw_layers, list) or not raw_layers:
            r.check(False, "'layers' must be a non-empty list")
            raw_layers = []
        for i, raw in enumerate(raw_layers):
            lr = FieldReader(raw, f"config.json:layers[{i}]") if isinstance(raw, dict) else None
            if lr is None:
                r.check(False, f"layers[{i}] must be an object")
                continue
            kind = lr.string("type", choices=cls.MIXER_TYPES)
            mr = lr.child("mixer")
            mixer = None
            if mr is None:
                lr.check(False, "required key 'mixer' is missing")
            elif kind == "retention":
                mixer = cls._retention(mr)
            elif kind == "latent_attention":
                mixer = cls._latent(mr)
            lr.absorb(mr)
            pr = lr.child("mlp")
            mlp = None
            if pr is not None:
                pr.string("kind", "dense", choices=("dense",))
                mlp = DenseMlp(pr.integer("ff", minimum=1))
            lr.absorb(pr)
            r.problems.extend(lr.problems)
            if not lr.problems and mixer is not None:
                layers.append(DinutarLayer(kind, mixer, mlp))
        # a layer that reads another's cached rows: that layer is an earlier latent attention with a latent of its own and
        # rows of the same make
        if len(layers) == len(raw_layers):
            for i, layer in enumerate(layers):
                m = layer.mixer
                if not isinstance(m, LatentMixer) or m.kv_from is None:
                    continue
                src = layers[m.kv_from].mixer if m.kv_from < i else None
                where = f"layers[{i}].mixer.kv_from"
                if not isinstance(src, LatentMixer) or src.kv_from is not None:
                    r.check(False, f"{where} must name an earlier latent attention layer that has a latent of its own")
                    continue
                r.check((src.kv_rank, src.rot_dim, src.rot) == (m.kv_rank, m.rot_dim, m.rot),
                        f"{where}: layer {m.kv_from} differs in 'kv_rank', 'rot_dim' or rotation")
        r.finish()
        return cls(vocab, width, float(scale), bigram, float(alpha), float(eps), tuple(layers))

    @classmethod
    def from_json(cls, path: str) -> "DinutarConfig":
        from .base import read_config_json
        return cls.from_dict(read_config_json(path))

    def to_dict(self) -> Dict[str, Any]:
        emb: Dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = self.bigram.to_json()
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": emb,
                "postln_alpha": self.postln_alpha, "norm": {"eps": self.norm_eps},
                "layers": [layer.to_json() for layer in self.layers]}
