"""Attention whose keys and values are made from one small latent vector per
token, which is all the cache keeps.

Per token: [c' | r'] = W_dkv h with c' of ``kv_rank`` and r' of ``rot_dim``
elements; c = c' / rms(c') * w_norm is the latent, r = rotate(r') one rotated
key part that all heads share.  Head a has the key [W_uk,a c | r] and the value
W_uv,a c; its query q_a = W_q,a h is [``head_dim`` plain | ``rot_dim`` rotated]
elements; the queries may be made from a latent of their own (``q_rank``:
q = W_uq (W_dq h / rms * w_q)).  score = (q_plain . k_plain + q_rot . r) * scale
over all earlier keys or a sliding window, softmax (with a learned sink per head in
the denominator when the model has one), each head's output times a gate
sigmoid(W_g h) when the model has one (a factor per head, or one per element of the heads' values), output projection over the concatenated heads.

The products with W_uk and W_uv are moved to the query's side, where they
cost one small product per new token instead of one per cached token:
q_plain . (W_uk,a c) = (W_uk,a^T q_plain) . c and sum_j p_j W_uv,a c_j =
W_uv,a (sum_j p_j c_j).  The attention itself then runs over one shared
key/value head whose key row is the cached [c | r] (``kv_rank + rot_dim``
elements) and whose value is the first ``kv_rank`` elements of the same row;
the cache holds no value pages.

A prompt in bfloat16 goes the other way round where the head sizes allow: one
product turns the step's rows [c | r] into every head's key [W_uk,a c | r] and
value W_uv,a c (the weight holds W_uk, W_uv and an identity for r, heads padded
with zeros up to a size the tensor-core attention kernels take), and those
kernels run as for ordinary heads; per token that costs a product with W_uk and
W_uv once, not once per key it sees.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..config.base import ConfigError, PartSpec
from ..weights.loader import WeightDecl
from .base import KVNeed, Mixer, build_part, register_part
from .linear import PartialSums, linear, linear_split
from .rope import Rope


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    """Parameters: ``hidden_size``, ``num_heads``, ``head_dim`` (the plain part of a query/key head), ``rot_dim``
    (its rotated part), ``value_dim``, ``kv_rank``, ``scale``, ``window`` (None = all keys), ``mask`` ("window" or
    "chunk"), ``eps`` (of the latents' norms), ``position`` (a ``rope`` PartSpec with ``rotary_dim`` = ``rot_dim``),
    tensor names ``q_weight`` [heads (head_dim + rot_dim), hidden], or with ``q_rank`` ``dq_weight`` [q_rank, hidden],
    ``dq_norm_weight`` [q_rank] and ``uq_weight`` [heads (head_dim + rot_dim), q_rank]; ``dkv_weight``
    [kv_rank + rot_dim, hidden], ``dkv_norm_weight`` [kv_rank], ``uk_weight`` [heads head_dim, kv_rank],
    ``uv_weight`` [heads value_dim, kv_rank], ``o_weight`` [hidden, heads value_dim]; optional ``sink_weight``
    [heads]; optional ``gate_weight`` [heads, hidden] or ``value_gate_weight`` [heads value_dim, hidden]; optional
    ``wide_output``."""
    graph_safe = True

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden = int(self.param("hidden_size"))
        self.heads = int(self.param("num_heads"))
        self.dim = int(self.param("head_dim"))
        self.rot = int(self.param("rot_dim"))
        self.dv = int(self.param("value_dim"))
        self.rank = int(self.param("kv_rank"))
        self.scale = float(self.param("scale"))
        self.eps = float(self.param("eps"))
        w = self.params.get("window")
        self.window = int(w) if w else None
        self.mask = self.params.get("mask") or "window"
        if self.mask not in kernels.MASKS:
            raise ConfigError(f"latent_attention: unknown mask '{self.mask}'")
        if self.dim < 1 or self.rot % 2:
            raise ConfigError(f"latent_attention: head_dim {self.dim} must be positive and rot_dim {self.rot} even")
        self.position = build_part("position", self.param("position"), ctx)
        if not isinstance(self.position, Rope) or self.position.rotary_dim != self.rot:
            raise ConfigError("latent_attention: the position encoding is a rotation over rot_dim")
        self.q_rank = int(self.params.get("q_rank") or 0)
        q_names = ("dq_weight", "dq_norm_weight", "uq_weight") if self.q_rank else ("q_weight",)
        self.names = {k: self.param(k) for k in (*q_names, "dkv_weight", "dkv_norm_weight", "uk_weight", "uv_weight",
                                                 "o_weight")}
        self.sink_name = self.params.get("sink_weight")
        self.gate_name = self.params.get("gate_weight")
        self.value_gate_name = self.params.get("value_gate_weight")
        if self.gate_name and self.value_gate_name:
            raise ConfigError("latent_attention: a gate per head or per value, not both")
        self.w_in = self.w_uq = self.w_uk = self.w_uv = self.w_o = self.norm_w = self.q_norm_w = self.sinks = None
        self.off_kv = self.off_gate = 0      # where the sections of a projection row begin (the queries' part first)
        self.fast_hd = 0            # head size of the prompt's tensor-core path (0: there is none)
        self.w_up = self.w_o_fast = None

    def kv_need(self):
        return KVNeed(1, self.rank + self.rot, self.window, 0)       # (values: the latent part of the key row)

    def weight_decls(self):
        n, H, h = self.names, self.heads, self.hidden
        if self.q_rank:
            decls = [WeightDecl(n["dq_weight"], (self.q_rank, h)), WeightDecl(n["dq_norm_weight"], (self.q_rank,), "gain"),
                     WeightDecl(n["uq_weight"], (H * (self.dim + self.rot), self.q_rank))]
        else:
            decls = [WeightDecl(n["q_weight"], (H * (self.dim + self.rot), h))]
        decls = [*decls,
                 WeightDecl(n["dkv_weight"], (self.rank + self.rot, h)),
                 WeightDecl(n["dkv_norm_weight"], (self.rank,), "norm"),
                 WeightDecl(n["uk_weight"], (H * self.dim, self.rank)),
                 WeightDecl(n["uv_weight"], (H * self.dv, self.rank)),
                 WeightDecl(n["o_weight"], (h, H * self.dv))]
        if self.sink_name:
            decls.append(WeightDecl(self.sink_name, (H,), "norm"))
        if self.gate_name:
            decls.append(WeightDecl(self.gate_name, (H, h)))
        if self.value_gate_name:
            decls.append(WeightDecl(self.value_gate_name, (H * self.dv, h)))
        return [*decls, *self.position.weight_decls()]

    def load(self, weights):
        n, dt, H = self.names, self.ctx.compute_dtype, self.heads
        # one product for all that reads the input: rows [q heads, or the queries' latent | latent | shared key part | gate]
        rows = [weights[n["dq_weight" if self.q_rank else "q_weight"]], weights[n["dkv_weight"]]]
        self.off_kv = rows[0].shape[0]
        self.off_gate = self.off_kv + rows[1].shape[0]
        if self.gate_name or self.value_gate_name:
            rows.append(weights[self.gate_name or self.value_gate_name])
        self.w_in = torch.cat(rows, dim=0).to(dt).contiguous()
        if self.q_rank:
            self.w_uq = weights[n["uq_weight"]].to(dt).contiguous()
            self.q_norm_w = weights[n["dq_norm_weight"]].to(torch.float32).contiguous()
        # per head: q_plain [dim] -> rank (W_uk as it lies), weighted latent [rank] -> value_dim (W_uv transposed)
        self.w_uk = weights[n["uk_weight"]].to(dt).reshape(H, self.dim, self.rank).contiguous()
        self.w_uv = weights[n["uv_weight"]].to(dt).reshape(H, self.dv, self.rank).transpose(1, 2).contiguous()
        self.w_o = weights[n["o_weight"]].to(dt).contiguous()
        self.norm_w = weights[n["dkv_norm_weight"]].to(torch.float32).contiguous()
        if self.sink_name:
            self.sinks = weights[self.sink_name].to(torch.float32).contiguous()
        self.position.load(weights)
        # a prompt's path over the tensor-core attention kernels: keys and values of every head out of one product
        hd = 0
        if dt == torch.bfloat16 and self.w_o.is_cuda and (self.rank + self.rot) % 8 == 0 and self.mask == "window":
            hd = kernels.attn_prefill_fast_head(max(self.dim + self.rot, self.dv))
        if hd:
            up = torch.zeros(2 * H * hd, self.rank + self.rot, dtype=dt, device=self.w_o.device)
            k_rows, v_rows = up[: H * hd].view(H, hd, -1), up[H * hd:].view(H, hd, -1)
            k_rows[:, : self.dim, : self.rank] = weights[n["uk_weight"]].to(dt).view(H, self.dim, self.rank)
            k_rows[:, self.dim: self.dim + self.rot, self.rank:] = torch.eye(self.rot, dtype=dt, device=up.device)
            v_rows[:, : self.dv, : self.rank] = weights[n["uv_weight"]].to(dt).view(H, self.dv, self.rank)
            self.w_up = up
            if hd == self.dv:
                self.w_o_fast = self.w_o
            else:
                wide = torch.zeros(self.hidden, H, hd, dtype=dt, device=up.device)
                wide[:, :, : self.dv] = self.w_o.view(self.hidden, H, self.dv)
                self.w_o_fast = wide.view(self.hidden, H * hd).contiguous()
            self.fast_hd = hd

    def _el(self) -> int:
        return 4 if self.ctx.compute_dtype == torch.float32 else 2

    def _uq_numel(self) -> int:
        return self.w_uq.numel() if self.q_rank else 0

    def _visible(self, pos: int) -> int:
        if not self.window:
            return pos + 1
        return pos % self.window + 1 if self.mask == "chunk" else min(pos + 1, self.window)

    def decode_bytes(self, lens) -> int:
        weights = (self.w_in.numel() + self._uq_numel() + self.w_uk.numel() + self.w_uv.numel() + self.w_o.numel()) * self._el()
        return weights + sum((self.rank + self.rot) * self._el() * self._visible(n - 1) for n in lens)

    def score_flops(self, lens) -> int:
        """Scores and weighted sums over the latent rows, as this part computes them."""
        pairs = 0
        for n in lens:
            w = self.window
            if w and self.mask == "chunk":
                full, rest = divmod(n, w)
                pairs += full * (w * (w + 1) // 2) + rest * (rest + 1) // 2
            else:
                pairs += n * (n + 1) // 2 if not w or n <= w else w * (w + 1) // 2 + (n - w) * w
        if self.fast_hd:        # (a prompt's path: ordinary heads of dim + rot key and value_dim value elements)
            return 2 * pairs * self.heads * (self.dim + self.rot + self.dv)
        return 2 * pairs * self.heads * (2 * self.rank + self.rot)

    def prefill_flops(self, lens) -> int:
        T = sum(lens)
        proj = 2 * T * (self.w_in.numel() + self._uq_numel() + self.w_uk.numel() + self.w_uv.numel() + self.w_o.numel())
        return proj + self.score_flops(lens)

    FAST_PROMPT_ROWS = 64      # from this many rows on a bfloat16 prompt takes the tensor-core path

    def _rows(self, x, batch, view, pitch: int):
        """From the layer's input: the packed query heads (``pitch`` elements each), the step's rows [c | r] (also
        written to the cache), the logits of a gate per head and those of a gate per value (column sections, or None)."""
        H, dim, rot, rank = self.heads, self.dim, self.rot, self.rank
        T, dt, dev = x.shape[0], x.dtype, x.device
        proj = linear(x, self.w_in, out_dtype=torch.float32)
        q = torch.empty(T, H * pitch, dtype=dt, device=dev)
        kvrow = torch.empty(T, rank + rot, dtype=dt, device=dev)
        pos = self.position
        turn = {"inv_freq": pos.inv_freq, "pairing": pos.pairing, "magnitude": pos.magnitude, "table": pos.precise_table(batch)}
        q_part = {"q": q, "q_src": proj[:, : self.off_kv], "pitch": pitch}
        kv_part = {"kvrow": kvrow, "kv_src": proj[:, self.off_kv: self.off_gate], "norm_w": self.norm_w,
                   "kv": view.kv if view.writes else None}
        if self.q_rank:
            cq = torch.empty(T, self.q_rank, dtype=dt, device=dev)
            kernels.latent_prep(batch, H, dim, rot, rank, self.eps, side=cq, side_src=proj[:, : self.q_rank],
                                side_w=self.q_norm_w, **kv_part, **turn)
            up = linear_split(cq, self.w_uq, wide=True)
            q_part["q_src"] = up.parts if isinstance(up, PartialSums) else up
            kernels.latent_prep(batch, H, dim, rot, rank, self.eps, **q_part, **turn)
        else:
            kernels.latent_prep(batch, H, dim, rot, rank, self.eps, **q_part, **kv_part, **turn)
        gate = proj[:, self.off_gate: self.off_gate + H] if self.gate_name else None
        values = proj[:, self.off_gate: self.off_gate + H * self.dv] if self.value_gate_name else None
        return q, kvrow, gate, values

    def _prompt_on_tensor_cores(self, x, batch, view):
        """Keys and values of every head from the step's latent rows by one product, then the attention kernels
        of ordinary heads (a window, a sink, a gate)."""
        H, hd = self.heads, self.fast_hd
        q, kvrow, gate, values = self._rows(x, batch, view, hd)
        if not view.writes:
            kvrow = batch.step_kv[view.cache_id][0]
        elif view.keep_step_kv:
            batch.step_kv[view.cache_id] = (kvrow, kvrow[:, : self.rank])
        kv_up = linear(kvrow, self.w_up)
        ctx = torch.empty(x.shape[0], H * hd, dtype=x.dtype, device=x.device)
        kernels.attn_prefill(ctx, q, kv_up[:, : H * hd], kv_up[:, H * hd:], batch, H, H, hd, self.scale, 0.0,
                             self.window or 0, mask=self.mask, sinks=self.sinks, gate=gate)
        if values is not None:
            kernels.head_gate(ctx, values, H, self.dv, per_value=True, pitch=hd)
        return linear_split(ctx, self.w_o_fast, wide=bool(self.params.get("wide_output", False)))

    def forward(self, x, batch, view):
        H, dim, rot, rank, dv = self.heads, self.dim, self.rot, self.rank, self.dv
        T, dt = x.shape[0], x.dtype
        if batch.is_prefill and self.fast_hd and T >= self.FAST_PROMPT_ROWS:
            return self._prompt_on_tensor_cores(x, batch, view)
        q, kvrow, gate, values = self._rows(x, batch, view, dim + rot)
        # the queries on the latent's side: [W_uk^T q_plain | q_rot] per head
        q_lat = torch.empty(T, H * (rank + rot), dtype=dt, device=x.device)
        kernels.head_project(q_lat, q, self.w_uk, H, dim, rank, extra=rot)
        # a decode step whose key rows have a size the split kernel takes gets whole rows [sum p c | sum p r] back
        # from it (the key pages serve as value pages); the values' part is read from there
        wide = not batch.is_prefill and kernels.attn_decode_fast(dt, rank + rot, batch.n_seqs)
        mix = torch.empty(T, H * (rank + rot if wide else rank), dtype=dt, device=x.device)
        window = self.window or 0
        if batch.is_prefill:
            if not view.writes:
                kvrow = batch.step_kv[view.cache_id][0]
            elif view.keep_step_kv:
                batch.step_kv[view.cache_id] = (kvrow, kvrow[:, :rank])
            kernels.attn_prefill(mix, q_lat, kvrow, kvrow[:, :rank], batch, H, 1, rank + rot, self.scale, 0.0, window,
                                 dv=rank, mask=self.mask, sinks=self.sinks, gate=gate)
        else:
            kernels.attn_decode(mix, q_lat, view.kv, batch, H, 1, rank + rot, self.scale, 0.0, window, dv=rank,
                                mask=self.mask, sinks=self.sinks, gate=gate)
        # back from the latent to the heads' values, then the output projection
        ctx = torch.empty(T, H * dv, dtype=dt, device=x.device)
        kernels.head_project(ctx, mix, self.w_uv, H, rank, dv, x_pitch=rank + rot if wide else rank, gate=values)
        return linear_split(ctx, self.w_o, wide=bool(self.params.get("wide_output", False)))
