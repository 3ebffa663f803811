"""Small Teselix configurations for the tests; they differ from one another in every size, in the order of
their layers, in which layers share weights and in their constants."""
from __future__ import annotations

import tempfile
from pathlib import Path


def _ret(heads, dim, vdim, decay, base, dims, scaling=None):
    rot = {"base": base, "dims": dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": rot}


def _lat(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, scaling=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
            "scale": scale, "rot": rot}


def _moe(experts, top, ff, limit, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def _layer(kind, mixer, mlp=None, weights_of=None):
    out = {"type": kind, "mixer": mixer, "mlp": mlp}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def _model(vocab, width, eps, alpha, layers):
    return {"architecture": "Teselix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "layers": layers}


_A_LAT = _lat(3, 10, 6, 14, 20, 18, 0.3, 300.0, (3.0, 40.0, 8.0, 0.5))
_A_RET = _ret(2, 12, 20, [0.9, 0.97], 50.0, 8)
_A_MOE = _moe(5, 2, 36, 1.5, (40, 0.8))
# odd sizes that no tensor-core kernel takes; a rotation over part of a head; stretched frequencies; a layer
# without a feed-forward; a layer that uses another's weights, and one that uses that one's
TA = _model(211, 72, 1e-5, 1.7, [
    _layer("retention", _A_RET, _A_MOE),
    _layer("latent_attention", _A_LAT, _moe(4, 1, 28, 0.7, (28, 3.0))),
    _layer("latent_attention", _A_LAT, _moe(4, 1, 28, 0.7, (28, 3.0)), weights_of=1),
    _layer("retention", _ret(3, 10, 6, [0.5, 0.8, 0.99], 1000.0, 10)),
    _layer("retention", _A_RET, _A_MOE, weights_of=0),
    _layer("latent_attention", _A_LAT, _moe(4, 1, 28, 0.7, (28, 3.0)), weights_of=2),
])

# sizes the bfloat16 tensor-core kernels take: heads of 64 (the prompt's), cached rows of 128 and of 160; a shared expert
# of twice an expert's size, one of its size, and none; three experts a token
TB = _model(320, 128, 1e-6, 2.5, [
    _layer("latent_attention", _lat(4, 48, 16, 64, 112, 64, 0.125, 5000.0, (8.0, 64.0, 16.0, 1.0)), _moe(6, 3, 64, 2.0, (128, 1.0))),
    _layer("retention", _ret(2, 64, 64, [0.95, 0.995], 10000.0, 64), _moe(8, 2, 64, 1.0, (64, 4.0))),
    _layer("retention", _ret(1, 128, 128, [0.98], 200.0, 32), _moe(8, 1, 96, 7.0)),
    _layer("latent_attention", _lat(6, 96, 32, 128, 128, 96, 0.09, 10000.0)),
    _layer("retention", _ret(2, 64, 64, [0.95, 0.995], 10000.0, 64), _moe(8, 2, 64, 1.0, (64, 4.0)), weights_of=1),
])

# nothing divides by four; every expert chosen; a shared expert that does not come in whole experts; alpha of 1; a
# decay of 1 (nothing is forgotten) and one of 0 (nothing is kept); no rotation at all in one retention
TC = _model(97, 50, 1e-4, 1.0, [
    _layer("retention", _ret(3, 10, 6, [1.0, 0.0, 0.75], 20.0, 6), _moe(3, 3, 22, 1.0, (10, 0.5))),
    _layer("latent_attention", _lat(5, 6, 2, 10, 14, 22, 0.4, 9.0), _moe(2, 1, 18, 0.3)),
    _layer("retention", _ret(1, 14, 22, [0.9], 3.0, 0), _moe(2, 1, 18, 0.3, (18, 0.3))),
])

# every size odd; one head; one expert
TD = _model(31, 51, 1e-5, 3.0, [
    _layer("latent_attention", _lat(1, 7, 4, 9, 11, 5, 0.5, 40.0, (2.0, 16.0, 4.0, 0.25)), _moe(1, 1, 17, 1.0, (17, 2.0))),
    _layer("retention", _ret(1, 5, 3, [0.6], 7.0, 4), _moe(5, 4, 9, 0.9)),
])

# heads beyond the fused output (values of 192), keys of 192, a stretched rotation in a retention; cached rows of 256 and
# of 64, twenty query heads on the latent
TE = _model(260, 192, 1e-5, 1.3, [
    _layer("retention", _ret(1, 192, 192, [0.99], 10000.0, 192, (4.0, 128.0, 8.0, 1.0)), _moe(4, 2, 48, 1.2, (144, 1.5))),
    _layer("latent_attention", _lat(2, 64, 64, 96, 192, 128, 0.1, 10000.0, (16.0, 32.0, 4.0, 1.0)), _moe(4, 2, 48, 1.2, (144, 1.5))),
    _layer("latent_attention", _lat(20, 16, 16, 32, 48, 40, 0.2, 100.0)),
])

CONFIGS = {"A": TA, "B": TB, "C": TC, "D": TD, "E": TE}


def make_folder(cfg_dict, seed=0, store_dtype="bfloat16", root=None, edit=None):
    """Write a random model folder; ``edit(name, tensor) -> tensor`` may change tensors on their way out."""
    import json

    import torch
    from airframe_b200.config import config_from_dict
    from airframe_b200.engine.model import declared_weights
    from airframe_b200.weights.random_init import random_tensor
    from airframe_b200.weights.safetensors_io import write_safetensors
    root = Path(root or tempfile.mkdtemp(prefix="tx_model_"))
    root.mkdir(parents=True, exist_ok=True)
    cfg = config_from_dict(cfg_dict)
    (root / "config.json").write_text(json.dumps(cfg.to_dict()))
    dt = {"bfloat16": torch.bfloat16, "float32": torch.float32}[store_dtype]

    def entries():
        for d in declared_weights(cfg.model_spec()):
            table = d.kind == "choice_table"

            def make(d=d, table=table):
                t = random_tensor(d, seed, torch.float32)
                if table:
                    return t
                # projections large enough that gates, sinks, limits and scores move away from their middles
                if d.kind == "matrix":
                    t = t * (6.0 if ".mlp." in d.name else 3.0)
                if d.kind == "table":
                    t = t * 20.0
                if d.name.endswith(("mix.uq", "mix.uv", "mix.o")):
                    t = t * (6.0 if d.name.endswith("uq") else 3.0)
                if d.kind == "norm":
                    t = t * 8.0 + 2.0 if d.name.endswith("sink") else t * 3.0
                if edit is not None:
                    t = edit(d.name, t)
                return t.to(dt)
            yield d.name, tuple(d.shape), torch.int32 if table else dt, make
    write_safetensors(root / "model.safetensors", entries(), metadata={"format": "pt"})
    return root
