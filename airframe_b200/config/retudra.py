"""Retudra: a decoder-only model whose only norms stand on the sublayers' outputs and whose
layers mix tokens in one of three ways (``layers[i].type``):

attention          grouped heads, q and k normed over the whole projection, a rotation over part of a
                   head, a sliding window beside which the sequence's first tokens stay visible
                   (``mask.size``, ``mask.keep_first``);
latent_attention   keys and values made from a small latent vector per token, a rotated key part that
                   the heads share, all earlier keys, the heads' outputs times sigmoid(W_g h) element by
                   element;
channel_delta      the delta rule with a decay per key channel: q, k and v through a short causal
                   convolution and silu, unit q and k, S <- diag(g) S, S <- S + beta k (v - S^T k)^T,
                   o = S^T q, each head's o over its root mean square, times a low-rank sigmoid gate.

x <- x + m LN_1(mixer(x)), then x <- x + m LN_2(ff(x)) (layer norms with weight and bias, m =
``residual_mult``), then every layer adds what the token's own id says to it: with e the layer's part of
``side.embed[token]``, x <- x + m RMS(W_p (gelu_tanh(W_s x) * e)).  The feed-forward is absent, dense, or
a mixture of experts: softmax scores, a correction for the choice only, a choice among the best groups
(a group's score its largest), weights as they are, and identity experts behind the others.  The
logits come from a head of their own and pass a softcap.

config.json gives every size and every constant that differs between models.  Tensor names: ``embed``,
``side.embed``, ``l<i>.norm1|norm2`` (each with ``.b``), ``l<i>.mix.*``, ``l<i>.mlp.*``,
``l<i>.side.gate|proj|norm``, ``final.norm`` (with ``.b``), ``head``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Optional

from .base import (ConfigError, KeyReader, LayerSpec, ModelConfig, ModelSpec, PartSpec,
                   ScheduleEntry)

LAYER_TYPES = ("attention", "latent_attention", "channel_delta")

# Angles are worked out in 64 bits from integer positions and the mixers have no bound of their own; a 32-bit
# float holds positions exactly up to here.
MAX_POSITIONS = 1 << 24

KEY_EPS = 1e-6      # under the root of the unit queries and keys of channel_delta


@dataclass
class RetudraConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    logit_softcap: Optional[float]                  # None: the logits as they are
    side_dim: int                                   # 0: no per-layer token input
    layers: list = field(default_factory=list)      # the entries of config.json's "layers", checked

    architecture = "Retudra"

    # ------------------------------------------------------------------ reading

    @staticmethod
    def _check_rot(where: str, m: dict, most: int) -> int:
        rot = KeyReader(m.get("rot"), where + ".rot")
        dims = rot.integer("dims", minimum=0)
        rot.number("base", positive=True)
        if dims % 2 or dims > most:
            raise ConfigError(f"{where}.rot: dims {dims} must be even and at most {most}")
        return dims

    @classmethod
    def _check_mixer(cls, i: int, kind: str, m: dict) -> None:
        where = f"config.json: layers[{i}].mixer"
        r = KeyReader(m, where)
        heads = r.integer("heads", minimum=1)
        dim = r.integer("dim", minimum=1)
        r.integer("vdim", minimum=1)
        if kind != "latent_attention":
            kv = r.integer("kv_heads", minimum=1)
            if heads % kv:
                raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv} kv_heads")
        if kind == "channel_delta":
            r.integer("conv", minimum=1)
            return
        r.number("scale")
        if kind == "attention":
            cls._check_rot(where, m, dim)
            if m.get("mask") is not None:
                mask = KeyReader(m["mask"], where + ".mask")
                mask.integer("size", minimum=1)
                mask.integer("keep_first", 0, minimum=0)
            return
        r.integer("kv_rank", minimum=1)
        rot_dim = r.integer("rot_dim", minimum=0)
        if cls._check_rot(where, m, rot_dim) != rot_dim:
            raise ConfigError(f"{where}: rot.dims {m['rot']['dims']} must be rot_dim {rot_dim}")

    @staticmethod
    def _check_mlp(i: int, mlp: dict) -> None:
        where = f"config.json: layers[{i}].mlp"
        mr = KeyReader(mlp, where)
        kind = mr.string("kind")
        if kind == "dense":
            mr.integer("ff", minimum=1)
            return
        if kind != "moe":
            raise ConfigError(f"{where}.kind '{kind}' is unknown (known: ['dense', 'moe'])")
        KeyReader(mlp.get("expert"), where + ".expert").integer("ff", minimum=1)
        ro = KeyReader(mlp.get("router"), where + ".router")
        n = ro.integer("experts", minimum=1) + ro.integer("identity", 0, minimum=0)
        top = ro.integer("top", minimum=1)
        count = keep = 1
        if ro.data.get("groups") is not None:
            gr = KeyReader(ro.data["groups"], where + ".router.groups")
            count, keep = gr.integer("count", minimum=1), gr.integer("keep", minimum=1)
        if n % count or keep > count:
            raise ConfigError(f"{where}.router: {n} experts in {count} groups of which {keep} are kept")
        if top > keep * (n // count):
            raise ConfigError(f"{where}.router: top {top} of {keep * (n // count)} experts")

    @classmethod
    def from_dict(cls, data: dict) -> "RetudraConfig":
        r = KeyReader(data)
        layers = data.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must list at least one layer")
        checked = []
        for i, layer in enumerate(layers):
            lr = KeyReader(layer, f"config.json: layers[{i}]")
            kind = lr.string("type")
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: layers[{i}].type '{kind}' is unknown (known: {list(LAYER_TYPES)})")
            if not isinstance(layer.get("mixer"), dict):
                raise ConfigError(f"config.json: layers[{i}].mixer must be an object")
            cls._check_mixer(i, kind, layer["mixer"])
            if layer.get("mlp") is not None:
                cls._check_mlp(i, layer["mlp"])
            checked.append(copy.deepcopy({"type": kind, "mixer": layer["mixer"], "mlp": layer.get("mlp")}))
        side = data.get("token_side")
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   norm_eps=KeyReader(data.get("norm"), "config.json: norm").number("eps", positive=True),
                   residual_mult=r.number("residual_mult"),
                   logit_softcap=r.number("logit_softcap", None, positive=True),
                   side_dim=0 if side is None else KeyReader(side, "config.json: token_side").integer("dim", minimum=1),
                   layers=checked)

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "layers": copy.deepcopy(self.layers), "norm": {"eps": self.norm_eps},
                "residual_mult": self.residual_mult, "logit_softcap": self.logit_softcap,
                "token_side": {"dim": self.side_dim} if self.side_dim else None, "vocab": self.vocab, "width": self.width}

    # ------------------------------------------------------------------ the model

    def _mixer(self, p: str, kind: str, m: dict) -> PartSpec:
        h, eps = self.width, self.norm_eps
        if kind == "channel_delta":
            names = {n: p + n for n in ("q", "k", "v", "b", "a1", "a2", "dt_bias", "A_log", "g1", "g2", "norm", "o")}
            names.update({n + "_conv": f"{p}{n}.conv" for n in ("q", "k", "v")})
            return PartSpec("channel_delta", {
                "hidden_size": h, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                "value_dim": m["vdim"], "taps": m["conv"], "eps": eps, "key_eps": KEY_EPS, "weights": names,
                "decay_rank": m.get("rank"), "gate_rank": m.get("gate_rank", m.get("rank"))})
        position = PartSpec("rope", {"theta": float(m["rot"]["base"]), "rotary_dim": m["rot"]["dims"], "pairing": "half",
                                     "precise_angles": True})
        if kind == "attention":
            mask = m.get("mask") or {}
            return PartSpec("attention", {
                "hidden_size": h, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                "value_dim": m["vdim"], "scale": float(m["scale"]), "softcap": 0.0, "window": mask.get("size"),
                "keep_first": mask.get("keep_first") or 0, "position": position,
                **{f"{n}_weight": p + n for n in ("q", "k", "v", "o")},
                "qk_norm": {"whole": True, "q_weight": p + "q.norm", "k_weight": p + "k.norm", "eps": eps},
                "wide_output": True})
        return PartSpec("latent_attention", {
            "hidden_size": h, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"],
            "value_dim": m["vdim"], "kv_rank": m["kv_rank"], "scale": float(m["scale"]), "window": None, "eps": eps,
            "position": position, "dkv_norm_weight": p + "dkv.norm",
            **{f"{n}_weight": p + n for n in ("q", "dkv", "uk", "uv", "o")}, "value_gate_weight": p + "g",
            "wide_output": True})

    def _feed_forward(self, p: str, mlp) -> PartSpec:
        if mlp is None:
            return PartSpec("none")
        if mlp["kind"] == "dense":
            return PartSpec("gated_mlp", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": "silu",
                                          **{f"{n}_weight": p + n for n in ("gate", "up", "down")}, "wide_output": True})
        ro = mlp["router"]
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "num_experts": ro["experts"],
            "top": ro["top"], "expert": "silu_glu", "router_weight": p + "router", "expert_weights": p + "e{e}.{role}",
            "router": {"score": "softmax", "correction_weight": p + "correction", "groups": copy.deepcopy(ro.get("groups")),
                       "group_score": "max", "identity": ro.get("identity") or 0}})

    def model_spec(self) -> ModelSpec:
        h, eps, m = self.width, self.norm_eps, self.residual_mult

        def norm(name: str, scale: float = 1.0) -> PartSpec:
            return PartSpec("layer_norm", {"weight": name, "bias": name + ".b", "size": h, "eps": eps, "scale": scale})

        layers = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            norms = {"post_mixer": norm(p + "norm1", m)}
            if layer["mlp"] is not None:
                norms["post_feed_forward"] = norm(p + "norm2", m)
            block = {}
            if self.side_dim:
                norms["post_side"] = PartSpec("rms_norm", {"weight": p + "side.norm", "size": h, "eps": eps,
                                                           "weight_offset": 0.0, "weight_kind": "gain", "scale": m})
                block["side"] = PartSpec("token_side", {
                    "hidden_size": h, "dim": self.side_dim, "vocab_size": self.vocab, "index": i,
                    "parts": len(self.layers), "activation": "gelu_tanh", "table_weight": "side.embed",
                    "gate_weight": p + "side.gate", "proj_weight": p + "side.proj"})
            layers.append(LayerSpec(prefix=p, block=PartSpec("postnorm", block),
                                    mixer=self._mixer(p + "mix.", layer["type"], layer["mixer"]),
                                    feed_forward=self._feed_forward(p + "mlp.", layer["mlp"]), norms=norms))
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=h, vocab_size=self.vocab, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"weight": "embed", "vocab_size": self.vocab, "hidden_size": h,
                                                   "scale": 1.0}),
            layers=layers, schedule=[ScheduleEntry(i) for i in range(len(layers))], final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": h, "softcap": self.logit_softcap or 0.0,
                                      "weight": "head"}),
            stop_token_ids=[])
        spec.validate()
        return spec
