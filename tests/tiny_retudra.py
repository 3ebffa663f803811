"""Small Retudra configurations for the tests; they differ from one another in every size, in the order of
their layers and in their constants."""
from __future__ import annotations

import tempfile
from pathlib import Path


def _delta(heads, kv_heads, dim, vdim, conv, rank, gate_rank=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rank": rank}
    if gate_rank is not None:
        m["gate_rank"] = gate_rank
    return m


def _attn(heads, kv_heads, dim, vdim, scale, base, dims, size=None, keep=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": dims}}
    if size is not None:
        m["mask"] = {"size": size} if keep is None else {"size": size, "keep_first": keep}
    return m


def _lat(heads, dim, rot_dim, vdim, kv_rank, scale, base):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
            "rot": {"base": base, "dims": rot_dim}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, identity, top, ff, groups=None):
    ro = {"experts": experts, "identity": identity, "top": top}
    if groups is not None:
        ro["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": ro}


def _layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _model(vocab, width, eps, mult, cap, side, layers):
    return {"architecture": "Retudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "logit_softcap": cap, "token_side": {"dim": side} if side else None, "layers": layers}


# odd sizes that no tensor-core kernel takes; two value heads on a key head; a window within a page that keeps three
# tokens, and one that keeps more than a page; a layer without a feed-forward; two identity experts in three groups
RA = _model(211, 72, 1e-5, 0.6, 9.0, 12, [
    _layer("channel_delta", _delta(4, 2, 12, 20, 3, 10), _moe(7, 2, 3, 28, (3, 2))),
    _layer("attention", _attn(6, 3, 10, 14, 0.4, 300.0, 6, 9, 3), _dense(52)),
    _layer("latent_attention", _lat(3, 10, 6, 14, 20, 0.3, 50.0)),
    _layer("attention", _attn(4, 1, 18, 18, 0.2, 900.0, 18, 70, 67), _moe(4, 1, 2, 36)),
    _layer("channel_delta", _delta(3, 3, 10, 6, 5, 7, 13), _dense(20)),
])

# sizes the bfloat16 tensor-core kernels take: heads of 64 (mma) and 128 (tcgen05), windows over several pages with kept
# tokens that end inside a page and at its border; cached latent rows of 128; keys and values of 64 and of 128
RB = _model(320, 128, 1e-6, 0.9, 20.0, 16, [
    _layer("attention", _attn(4, 2, 64, 64, 0.125, 5000.0, 32, 100, 70), _moe(6, 2, 3, 64, (2, 1))),
    _layer("channel_delta", _delta(2, 1, 64, 64, 4, 16), _moe(8, 0, 2, 64, (4, 2))),
    _layer("attention", _attn(2, 2, 128, 128, 0.09, 20000.0, 128, 130, 64), _dense(192)),
    _layer("channel_delta", _delta(1, 1, 128, 128, 2, 24, 8), _moe(3, 5, 4, 32, (2, 2))),
    _layer("latent_attention", _lat(4, 48, 16, 64, 112, 0.125, 5000.0), _dense(256)),
])

# nothing divides by four; no convolution at all (one tap); no window, no rotation; no side input; no softcap; every
# expert and identity expert chosen
RC = _model(97, 50, 1e-4, 1.0, None, 0, [
    _layer("channel_delta", _delta(3, 1, 10, 6, 1, 5), _moe(2, 1, 3, 22)),
    _layer("attention", _attn(5, 5, 6, 10, 0.4, 9.0, 0), _moe(3, 0, 1, 18, (3, 1))),
    _layer("latent_attention", _lat(5, 6, 2, 10, 14, 0.4, 9.0), None),
])

# every size odd; one head; a window of one position that keeps one; a convolution longer than the shortest prompts
RD = _model(31, 51, 1e-5, 0.3, 3.0, 5, [
    _layer("attention", _attn(1, 1, 7, 9, 0.5, 40.0, 4, 1, 1), _moe(1, 4, 2, 17)),
    _layer("channel_delta", _delta(1, 1, 5, 3, 9, 3), _dense(11)),
    _layer("latent_attention", _lat(1, 7, 4, 9, 11, 0.5, 40.0), _moe(5, 0, 5, 9)),
])

# values of another size than the keys on the tensor cores (padded heads), twenty query heads on one; cached latent rows of
# 256 and of 64; keys of 192, values of 96
RE = _model(260, 192, 1e-5, 0.7, 12.0, 24, [
    _layer("channel_delta", _delta(2, 2, 192, 96, 4, 20), _moe(4, 2, 2, 48, (3, 2))),
    _layer("attention", _attn(20, 1, 96, 64, 0.1, 1000.0, 48, 200, 5), _moe(4, 2, 2, 48, (3, 2))),
    _layer("latent_attention", _lat(2, 64, 64, 96, 192, 0.1, 10000.0), _dense(144)),
    _layer("latent_attention", _lat(20, 16, 16, 32, 48, 0.2, 100.0)),
])

CONFIGS = {"A": RA, "B": RB, "C": RC, "D": RD, "E": RE}


def make_folder(cfg_dict, seed=0, store_dtype="bfloat16", root=None, edit=None):
    """Write a random model folder; ``edit(name, tensor) -> tensor`` may change tensors on their way out."""
    import json

    import torch
    from airframe_b200.config import config_from_dict
    from airframe_b200.engine.model import declared_weights
    from airframe_b200.weights.random_init import random_tensor
    from airframe_b200.weights.safetensors_io import write_safetensors
    root = Path(root or tempfile.mkdtemp(prefix="rd_model_"))
    root.mkdir(parents=True, exist_ok=True)
    cfg = config_from_dict(cfg_dict)
    (root / "config.json").write_text(json.dumps(cfg.to_dict()))
    dt = {"bfloat16": torch.bfloat16, "float32": torch.float32}[store_dtype]

    def entries():
        for d in declared_weights(cfg.model_spec()):
            def make(d=d):
                t = random_tensor(d, seed, torch.float32)
                # projections large enough that gates, scores and decays move away from their middles
                if d.kind == "matrix":
                    t = t * 5.0
                if d.kind == "table":
                    t = t * 20.0
                if d.name.endswith("router"):          # choices that seldom rest on a close call
                    t = t * 4.0
                if d.name.endswith("correction"):      # (they are at home among softmax scores; some outweigh them)
                    t = t * 1.5
                if d.name.endswith("dt_bias"):         # from channels that keep little to channels that keep nearly all
                    t = t * 20.0 - 2.0
                if d.name.endswith("A_log"):
                    t = t * 5.0
                if d.name.endswith(".b") and ".norm" in d.name:
                    t = t * 3.0
                if edit is not None:
                    t = edit(d.name, t)
                return t.to(dt)
            yield d.name, tuple(d.shape), dt, make
    write_safetensors(root / "model.safetensors", entries(), metadata={"format": "pt"})
    return root
