"""Teselix: a decoder-only model whose norms stand behind the residual sums and whose
layers mix tokens in one of two ways (``layers[i].type``):

retention          linear attention with a fixed decay per head: q and k rotated
                   (half-split pairs), S <- decay S + k v^T, o = S^T q, each head's o over
                   its root mean square, times silu(W_g h);
latent_attention   keys and values made from a small latent vector per token, queries
                   from a latent of their own, a rotated key part that the heads share
                   (neighbouring pairs; frequencies stretched for a longer context when
                   ``rot.scaling`` says so), all earlier keys, a learned sink per head in the
                   softmax's denominator, an output gate per head.

x <- norm1(alpha x + sigmoid(W_1 x + b_1) * mixer(shift(x))), then
x <- norm2(alpha x + sigmoid(W_2 x + b_2) * ff(x)), layer norms with weight and bias; shift
moves each token's row towards the row before it, by a factor per channel.  The
feed-forward is absent or a mixture of clamped gated experts that a table looks up by the
token's id, each with the weight 1 / top, beside a shared one.  A layer may use another
layer's weights (``weights_of``) with a cache and a state of its own.  The embedding
table also makes the logits.

config.json gives every size and every constant that differs between models.
Tensor names: ``embed``, ``l<i>.norm1|norm2`` (each with ``.b``), ``l<i>.shift``, ``l<i>.rg1|rg2``
(each with ``.b``), ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field

from .base import (ConfigError, KeyReader, LayerSpec, ModelConfig, ModelSpec, PartSpec,
                   ScheduleEntry)

LAYER_TYPES = ("retention", "latent_attention")

# Angles are worked out in 64 bits from integer positions and the mixers have no bound of their own; a 32-bit
# float holds positions exactly up to here.
MAX_POSITIONS = 1 << 24


@dataclass
class TeselixConfig(ModelConfig):
    vocab: int
    width: int
    alpha: float
    norm_eps: float
    layers: list = field(default_factory=list)      # the entries of config.json's "layers", checked

    architecture = "Teselix"

    # ------------------------------------------------------------------ reading

    @staticmethod
    def _check_rot(where: str, m: dict, most: int) -> None:
        rot = KeyReader(m.get("rot"), where + ".rot")
        dims = rot.integer("dims", minimum=0)
        base = rot.number("base", positive=True)
        if dims % 2 or dims > most:
            raise ConfigError(f"{where}.rot: dims {dims} must be even and at most {most}")
        sc = rot.data.get("scaling")
        if sc is not None:
            sr = KeyReader(sc, where + ".rot.scaling")
            for key in ("factor", "original", "fast", "slow"):
                sr.number(key, positive=True)
            if not base > 1:
                raise ConfigError(f"{where}.rot: scaling needs a base above 1")

    @classmethod
    def _check_mixer(cls, i: int, kind: str, m: dict) -> None:
        where = f"config.json: layers[{i}].mixer"
        r = KeyReader(m, where)
        heads = r.integer("heads", minimum=1)
        dim = r.integer("dim", minimum=1)
        r.integer("vdim", minimum=1)
        if kind == "retention":
            decay = m.get("decay")
            if not isinstance(decay, list) or len(decay) != heads \
                    or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in decay):
                raise ConfigError(f"{where}.decay must list one number for each of the {heads} heads")
            cls._check_rot(where, m, dim)
            return
        r.number("scale")
        r.integer("kv_rank", minimum=1)
        r.integer("q_rank", minimum=1)
        rot_dim = r.integer("rot_dim", minimum=0)
        cls._check_rot(where, m, rot_dim)
        if m["rot"]["dims"] != rot_dim:
            raise ConfigError(f"{where}: rot.dims {m['rot']['dims']} must be rot_dim {rot_dim}")

    @staticmethod
    def _check_mlp(i: int, mlp: dict) -> None:
        where = f"config.json: layers[{i}].mlp"
        mr = KeyReader(mlp, where)
        if mr.string("kind") != "moe":
            raise ConfigError(f"{where}.kind '{mlp['kind']}' is unknown (known: ['moe'])")
        experts = [("expert", mlp.get("expert"))]
        if mlp.get("shared") is not None:
            experts.append(("shared", mlp["shared"]))
        for name, e in experts:
            er = KeyReader(e, f"{where}.{name}")
            er.integer("ff", minimum=1)
            er.number("limit", positive=True)
        ro = KeyReader(mlp.get("router"), where + ".router")
        n, top = ro.integer("experts", minimum=1), ro.integer("top", minimum=1)
        if top > n:
            raise ConfigError(f"{where}.router: top {top} of {n} experts")

    @classmethod
    def from_dict(cls, data: dict) -> "TeselixConfig":
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
            mlp = layer.get("mlp")
            if mlp is not None:
                cls._check_mlp(i, mlp)
            entry = {"type": kind, "mixer": layer["mixer"], "mlp": mlp}
            if layer.get("weights_of") is not None:
                entry["weights_of"] = lr.integer("weights_of", minimum=0)
            checked.append(copy.deepcopy(entry))
        config = cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                     alpha=r.number("postln_alpha"),
                     norm_eps=KeyReader(data.get("norm"), "config.json: norm").number("eps", positive=True), layers=checked)
        for i, layer in enumerate(checked):
            j = config.owner(i)
            if any(layer[key] != checked[j][key] for key in ("type", "mixer", "mlp")):
                raise ConfigError(f"config.json: layers[{i}] uses the weights of layer {j} but differs from it")
        return config

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "layers": copy.deepcopy(self.layers), "norm": {"eps": self.norm_eps},
                "postln_alpha": self.alpha, "vocab": self.vocab, "width": self.width}

    # ------------------------------------------------------------------ the model

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses (its own number without ``weights_of``)."""
        seen = [i]
        while self.layers[seen[-1]].get("weights_of") is not None:
            j = self.layers[seen[-1]]["weights_of"]
            if j >= len(self.layers) or j in seen:
                raise ConfigError(f"config.json: layers[{i}].weights_of leads to no layer with weights of its own")
            seen.append(j)
        return seen[-1]

    def _mixer(self, p: str, kind: str, m: dict) -> PartSpec:
        h, eps, rot = self.width, self.norm_eps, m["rot"]
        position = PartSpec("rope", {"theta": float(rot["base"]), "rotary_dim": rot["dims"], "precise_angles": True,
                                     "pairing": "half" if kind == "retention" else "adjacent",
                                     "scaling": copy.deepcopy(rot.get("scaling"))})
        if kind == "retention":
            return PartSpec("retention", {
                "hidden_size": h, "num_heads": m["heads"], "head_dim": m["dim"], "value_dim": m["vdim"],
                "decay": [float(d) for d in m["decay"]], "eps": eps, "position": position,
                "weights": {n: p + n for n in ("q", "k", "v", "g", "o")}})
        return PartSpec("latent_attention", {
            "hidden_size": h, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"],
            "value_dim": m["vdim"], "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "scale": float(m["scale"]),
            "window": None, "eps": eps, "position": position, "dq_weight": p + "dq", "dq_norm_weight": p + "dq.norm",
            "uq_weight": p + "uq", "dkv_weight": p + "dkv", "dkv_norm_weight": p + "dkv.norm", "uk_weight": p + "uk",
            "uv_weight": p + "uv", "o_weight": p + "o", "sink_weight": p + "sink", "gate_weight": p + "g",
            "wide_output": True})

    def _feed_forward(self, p: str, mlp) -> PartSpec:
        if mlp is None:
            return PartSpec("none")
        params = {"hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "limit": float(mlp["expert"]["limit"]),
                  "num_experts": mlp["router"]["experts"], "top": mlp["router"]["top"], "table_weight": p + "table",
                  "vocab_size": self.vocab, "expert_weights": p + "e{e}.{role}"}
        if mlp.get("shared") is not None:
            params["shared"] = {"intermediate_size": mlp["shared"]["ff"], "limit": float(mlp["shared"]["limit"]),
                                "gate_weight": p + "shared.gate", "up_weight": p + "shared.up",
                                "down_weight": p + "shared.down"}
        return PartSpec("routed_experts", params)

    def model_spec(self) -> ModelSpec:
        h = self.width

        def norm(name: str) -> PartSpec:
            return PartSpec("layer_norm", {"weight": name, "bias": name + ".b", "size": h, "eps": self.norm_eps})

        layers, place = [], {}
        for i, layer in enumerate(self.layers):
            if self.owner(i) != i:
                continue
            p = f"l{i}."
            gates = [{"weight": f"{p}rg{q}", "bias": f"{p}rg{q}.b"} for q in (1, 2)]
            norms = {"mixer_sum": norm(p + "norm1")}
            if layer["mlp"] is not None:
                norms["feed_forward_sum"] = norm(p + "norm2")
            place[i] = len(layers)
            layers.append(LayerSpec(prefix=p, block=PartSpec("normed_sum", {"hidden_size": h, "alpha": self.alpha,
                                                                            "shift_weight": p + "shift", "gates": gates}),
                                    mixer=self._mixer(p + "mix.", layer["type"], layer["mixer"]),
                                    feed_forward=self._feed_forward(p + "mlp.", layer["mlp"]), norms=norms))
        # every run keeps a cache and states of its own: layers that share weights share nothing else
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=h, vocab_size=self.vocab, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"weight": "embed", "vocab_size": self.vocab, "hidden_size": h,
                                                   "scale": 1.0}),
            layers=layers, schedule=[ScheduleEntry(place[self.owner(i)]) for i in range(len(self.layers))],
            final_norm=norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": h, "softcap": 0.0, "tied_to": "embed"}),
            stop_token_ids=[])
        spec.validate()
        return spec
