"""Small Dinutar configurations and random weights for the tests, and an error measure.

The configurations differ from one another in every size, in the order of the layers and in what is left out (the second
embedding table, the embedding's scale, the rotation and its stretching, a layer's feed-forward, layers that read another
layer's rows).  Values that a given checkpoint might happen to make equal (key and value sizes of a head, head counts of the
mixers, of a layer and of the layer whose rows it reads) or 1 are unequal here, or 1 where a checkpoint would have more.
Weights are rounded to bfloat16 so that both precisions read the same values.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List, Optional

import torch

NAME = "Dinutar"


def _ret(heads, dim, vdim, decay, rot=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "retention", "mixer": m}


def _latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=1000.0, scaling=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"dims": rot_dim, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def _layer(mixer: dict, ff: Optional[int]) -> dict:
    return dict(mixer, mlp={"kind": "dense", "ff": ff} if ff else None)


def _model(vocab, width, alpha, eps, layers, scale=None, bigram=None) -> dict:
    emb = {}
    if scale is not None:
        emb["scale"] = scale
    if bigram:
        emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return {"architecture": NAME, "vocab": vocab, "width": width, "postln_alpha": alpha, "norm": {"eps": eps}, "embedding": emb,
            "layers": layers}


YARN = (4.0, 64, 16.0, 1.0)


def config_a() -> dict:
    """Both mixers with and without a feed-forward; a rotation of part of a retention head; two latents, the first read by
    two later layers with other head counts, head sizes and scales, one of them behind the second latent's layer."""
    return _model(211, 96, 2.5, 1e-5, [
        _layer(_latent(4, 16, 8, 24, 24, 0.3, 5000.0, YARN), 64),
        _layer(_ret(3, 24, 40, [0.5, 0.97, 0.9995], rot=(16, 900.0)), None),
        _layer(_latent(3, 8, 8, 40, 24, 0.45, 5000.0, YARN, kv_from=0), 40),
        _layer(_ret(4, 20, 12, [0.9, 0.99, 0.999, 0.7], rot=(20, 1e5)), 72),
        _layer(_latent(2, 24, 12, 16, 56, 0.2, 300.0), None),
        _layer(_latent(5, 12, 8, 8, 24, 0.25, 5000.0, YARN, kv_from=0), None),
        _layer(_latent(3, 16, 12, 24, 56, 0.35, 300.0, kv_from=4), 56),
    ], scale=0.7, bigram=(101, 37, 11))


def config_b() -> dict:
    """One head everywhere; no second table, no embedding scale, alpha 1; no rotation in a retention layer and in a latent
    layer; a layer of a mixer alone last; a decay of one (nothing is forgotten)."""
    return _model(130, 64, 1.0, 1e-3, [
        _layer(_ret(1, 40, 72, [1.0]), 24),
        _layer(_latent(1, 40, 0, 72, 56, 0.2), 40),
        _layer(_latent(1, 12, 0, 8, 56, 0.5, kv_from=1), 8),
        _layer(_ret(1, 8, 16, [0.9], rot=(2, 10.0)), None),
    ])


def config_c() -> dict:
    """Sizes that fit no kernel's favourite multiple: a width of 100, heads of 12, 13 and 70 with values of 7, 9 and 36, a
    rotation of six dimensions, a latent row of 26 values, feed-forwards of 20 and 9; a table of one hashed row, and
    multipliers whose products exceed 32 bits."""
    return _model(77, 100, 4.0, 1e-4, [
        _layer(_ret(5, 12, 7, [0.6, 0.8, 0.95, 0.99, 0.999], rot=(6, 777.0)), 20),
        _layer(_latent(5, 12, 6, 36, 20, 0.25, 50.0, (1.5, 10, 3.0, 2.0)), None),
        _layer(_ret(2, 70, 9, [0.98, 0.9], rot=(70, 30.0)), 9),
        _layer(_latent(7, 20, 6, 4, 20, 0.4, 50.0, (1.5, 10, 3.0, 2.0), kv_from=1), 36),
        _layer(_ret(1, 13, 36, [0.93]), None),
    ], scale=1.5, bigram=(1, 2_000_000_011, 1_999_999_973))


def config_d() -> dict:
    """Sizes the tensor-core and the vectorised kernels take: latent rows of 64 and 576 values, retention heads of 64 x 64,
    128 x 128 and 200 x 136, more than sixteen heads, a width of 128."""
    return _model(150, 128, 3.5, 1e-6, [
        _layer(_ret(2, 128, 128, [0.99, 0.9999], rot=(128, 10000.0)), 192),
        _layer(_latent(18, 32, 16, 32, 48, 0.35, 1e4, (8.0, 128, 32.0, 1.0)), 96),
        _layer(_ret(1, 200, 136, [0.996], rot=(64, 1e4)), None),
        _layer(_latent(4, 64, 64, 32, 512, 0.1, 1e4), 64),
        _layer(_latent(3, 64, 64, 48, 512, 0.1, 1e4, kv_from=3), None),
        _layer(_ret(4, 64, 64, [0.5, 0.9, 0.99, 0.999], rot=(32, 500.0)), 128),
    ], scale=0.25, bigram=(997, 7, 3))


def only(kind: str) -> dict:
    """Three layers of one kind of mixer and no feed-forward: the mechanism alone."""
    mixers = {
        "retention": [_ret(3, 16, 40, [0.8, 0.98, 0.9999], rot=(8, 50.0)), _ret(6, 40, 8, [0.5, 0.6, 0.9, 0.95, 0.99, 0.995], rot=(40, 900.0)),
                      _ret(2, 70, 20, [0.99, 1.0])],
        "latent_attention": [_latent(3, 8, 8, 16, 32, 0.4, 20.0, YARN), _latent(2, 24, 0, 8, 16, 0.3),
                             _latent(5, 12, 8, 4, 32, 0.5, 20.0, YARN, kv_from=0)],
    }[kind]
    return _model(90, 80, 2.0, 1e-5, [_layer(m, None) for m in mixers], scale=1.0, bigram=(53, 5, 1))


CONFIGS = {"a": config_a, "b": config_b, "c": config_c, "d": config_d, "retention": lambda: only("retention"),
           "latent_attention": lambda: only("latent_attention")}


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "embed.norm": (W,), "final.norm": (W,)}
    if cfg["embedding"].get("bigram"):
        out["bigram"] = (cfg["embedding"]["bigram"]["buckets"] + 1, W)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (W,), p + "ls1": (W,)})
        if layer["type"] == "retention":
            out.update({p + "mix.q": (H * d, W), p + "mix.k": (H * d, W), p + "mix.v": (H * dv, W), p + "mix.g": (H * dv, W)})
        else:
            R, dr = m["kv_rank"], m["rot_dim"]
            out.update({p + "mix.q": (H * (d + dr), W), p + "mix.uk": (H * d, R), p + "mix.uv": (H * dv, R)})
            if "kv_from" not in m:
                out.update({p + "mix.dkv": (R + dr, W), p + "mix.dkv.norm": (R,)})
        out[p + "mix.o"] = (W, H * dv)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "ls2": (W,), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.split(".")[-1]
        if name in ("embed", "bigram"):
            t = torch.randn(shape, generator=g)
        elif last in ("ls1", "ls2"):
            t = 0.6 * torch.randn(shape, generator=g)                  # of both signs
        elif ".mlp." in name:
            t = torch.randn(shape, generator=g) * shape[1] ** -0.5
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) * (1.4 / shape[1] ** 0.5)
        else:
            t = 1.0 + 0.25 * torch.randn(shape, generator=g)           # norm weights
        out[name] = t.to(torch.bfloat16)
    return out


def write_folder(cfg: dict, weights: Dict[str, torch.Tensor], out_dir: str) -> str:
    from cpmcu_b200.weights.safetensors_io import save_file

    os.makedirs(out_dir, exist_ok=True)
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(out_dir, "model.safetensors"))
    return out_dir


def random_ids(vocab: int, n: int, seed: int) -> List[int]:
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


# Largest allowed root mean square of (engine - plain) over the vocabulary, the mean difference taken off, relative to
# the root mean square of the plain logits, for the worst row and for the median row.  float32: summation order only.
# bfloat16: activations between the kernels and the cached rows are rounded to bfloat16 in the engine; single rows react
# strongly to that rounding (a read-out of a retention head is divided by its own size, however small, and squared relus
# follow), so the worst row has a loose bound and the median a tight one, and float32 carries the exact comparison.
TOL = {"float32": 6e-5, "bfloat16": 0.5}
MEDIAN_TOL = {"float32": 4e-6, "bfloat16": 1.5e-2}


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape, (got.shape, want.shape)
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
