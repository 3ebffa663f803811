"""Gated feed-forward: f = W_down (act(W_gate x) * (W_up x)).

Reference: ``src/backend/bindless/sh_layer_v1.wgsl:1024-1070`` (gate and up),
``:1079`` (tanh-GELU), ``:1082`` (SiLU), ``:1104-1140`` (down).  The reference
picks the activation by a proxy (softcap > 0); here it is a parameter.

``routed_experts``: a mixture of small feed-forwards of which a token uses a
few.  The router's scores are sigmoids of its logits (32-bit), the ``top``
largest choose the experts, and a chosen expert's score multiplies the expert's
*input*: f = sum over the chosen e of E_e(s_e h), with E(h) = W_down (act(W_gate h,
W_up h)) and act(g, u) = g' sigmoid(1.702 g') (u' + 1), g' = min(g, limit),
u' = clamp(u, -limit, limit).  A shared expert of the same form (own size and limit)
may run for every token; it is added times sigmoid(w_sg . h).  Nothing is read back
by the host: the pairs are sorted by expert on the device and the products walk
tiles of one expert's pairs, so a decode step can be captured.

Other designs' routers and experts are options of the same part.  The router may add
a learned correction to the scores *for the choice only*, may choose among the
experts of the best groups only (``groups`` equal groups of neighbours, a group's
score the sum of its two largest choice scores, the ``keep`` best kept), and may
divide the chosen scores by their sum and multiply them by a constant.  An expert
may be of one matrix and an activation, E(h) = W_down gelu(W_up h) with the exact
(erf) GELU (``expert`` = "gelu_erf"); its weight then multiplies the expert's
*output* (it is applied behind the activation, in front of the linear down product).

The scores may instead be the softmax of the logits, a group's score its largest choice score alone, and experts may
be ordinary gated ones, E(h) = W_down (silu(W_gate h) * (W_up h)) (``expert`` = "silu_glu"), the weight on their
output.  Behind the experts with matrices the router may have ``identity`` experts without any, whose output is the
input itself (times the weight): they take part in scores, groups and choice, and cost no product.

There may be no router at all: a table of integers then names the ``top`` experts of every token id, each with the
weight 1 / top on its output, which the residual sum applies.  A shared expert of the same form is then, where its size
comes in whole experts (or nearly), so many more experts that every token uses: its features fall apart into
groups, E(h) = sum over groups of W_down,g act(W_gate,g h, W_up,g h), and the one sum over experts holds them all.  Which experts a step's tokens use is then known before its
first layer runs: the pairs of all such layers are sorted by one kernel, at the first of them.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..config.base import ConfigError
from ..weights.loader import WeightDecl
from .base import FeedForward, register_part
from .linear import PartialSums, WeightedSum, gated_linear, linear_split


@register_part("feed_forward", "gated_mlp")
class GatedMlp(FeedForward):
    """Parameters: ``hidden_size``, ``intermediate_size``, ``activation``
    (``gelu_tanh`` or ``silu``), ``gate_weight``/``up_weight``/``down_weight``; optional
    ``wide_output`` (default false): the down projection's result stays float32 on its way
    into the residual sum."""
    graph_safe = True


    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden = int(self.param("hidden_size"))
        self.inter = int(self.param("intermediate_size"))
        self.activation = self.param("activation")
        if self.activation not in kernels.ACTIVATIONS:
            raise ConfigError(f"gated_mlp: unknown activation '{self.activation}' "
                              f"(known: {sorted(kernels.ACTIVATIONS)})")
        self.names = [self.param(k) for k in ("gate_weight", "up_weight", "down_weight")]
        self.w_gu = None
        self.interleaved = False
        self.w_down = None

    def weight_decls(self):
        g, u, d = self.names
        return [WeightDecl(g, (self.inter, self.hidden)), WeightDecl(u, (self.inter, self.hidden)),
                WeightDecl(d, (self.hidden, self.inter))]

    def load(self, weights):
        g, u, d = self.names
        dt = self.ctx.compute_dtype
        wg, wu = weights[g].to(dt), weights[u].to(dt)
        # bfloat16 with a K the tensor-core product takes: gate and up rows interleaved per
        # tile, activation in the product's epilogue; else [gate; up] and a kernel of its own
        self.interleaved = dt == torch.bfloat16 and self.hidden % 8 == 0
        self.w_gu = (kernels.interleave_gate_up(wg, wu) if self.interleaved
                     else torch.cat([wg, wu], dim=0).contiguous())
        self.w_down = weights[d].to(dt).contiguous()

    def decode_bytes(self, lens) -> int:
        return 3 * self.hidden * self.inter * (4 if self.ctx.compute_dtype == torch.float32 else 2)

    def prefill_flops(self, lens) -> int:
        return 2 * sum(lens) * 3 * self.hidden * self.inter

    def forward(self, x, batch):
        h = gated_linear(x, self.w_gu, self.inter, self.activation, self.interleaved)
        return linear_split(h, self.w_down, wide=bool(self.params.get("wide_output", False)))


@register_part("feed_forward", "none")
class NoFeedForward(FeedForward):
    """A layer without a feed-forward: a block that knows of it leaves the
    sublayer and its norm out (``prenorm`` does)."""
    graph_safe = True
    present = False

    def forward(self, x, batch):
        raise ConfigError("a layer without a feed-forward was asked to run one (its block does not leave it out)")


@register_part("feed_forward", "token_side")
class TokenSide(FeedForward):
    """What a token's own id says to a layer: W_proj (act(W_gate x) * e), e the columns [index * dim, (index + 1) * dim) of
    the token's row of a table that all layers share.  Parameters: ``hidden_size``, ``dim``, ``vocab_size``, ``index``,
    ``parts`` (the table holds ``parts`` * ``dim`` columns), ``activation``, ``table_weight`` [vocab, parts dim],
    ``gate_weight`` [dim, hidden], ``proj_weight`` [hidden, dim].  The result is 32-bit rows or partial sums."""
    graph_safe = True

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden, self.dim, self.vocab = (int(self.param(k)) for k in ("hidden_size", "dim", "vocab_size"))
        self.index, self.parts = int(self.param("index")), int(self.param("parts"))
        if not 0 <= self.index < self.parts:
            raise ConfigError(f"token_side: part {self.index} of {self.parts}")
        self.activation = self.param("activation")
        if self.activation not in kernels.ACTIVATIONS:
            raise ConfigError(f"token_side: unknown activation '{self.activation}' (known: {sorted(kernels.ACTIVATIONS)})")
        self.names = [self.param(k) for k in ("table_weight", "gate_weight", "proj_weight")]
        self.table = self.w_gate = self.w_proj = None

    def weight_decls(self):
        t, g, p = self.names
        return [WeightDecl(t, (self.vocab, self.parts * self.dim), "table"), WeightDecl(g, (self.dim, self.hidden)),
                WeightDecl(p, (self.hidden, self.dim))]

    def load(self, weights):
        # (the table in the dtype it was loaded in is that of the compute dtype: the layers hold one tensor)
        self.table, self.w_gate, self.w_proj = (weights[n].to(self.ctx.compute_dtype).contiguous() for n in self.names)

    def _el(self) -> int:
        return 4 if self.ctx.compute_dtype == torch.float32 else 2

    def decode_bytes(self, lens) -> int:
        return (2 * self.hidden + len(lens)) * self.dim * self._el()

    def prefill_flops(self, lens) -> int:
        return 4 * sum(lens) * self.hidden * self.dim

    def forward(self, x, batch):
        z = linear_split(x, self.w_gate, wide=True)
        g = torch.empty(x.shape[0], self.dim, dtype=x.dtype, device=x.device)
        kernels.token_gate(g, z.parts if isinstance(z, PartialSums) else z, self.table, self.index * self.dim, batch.tokens,
                           self.activation)
        return linear_split(g, self.w_proj, wide=True)


@register_part("feed_forward", "routed_experts")
class RoutedExperts(FeedForward):
    """Parameters: ``hidden_size``, ``intermediate_size``, ``num_experts``, ``top``, ``limit``,
    ``router_weight`` ([experts, hidden]) and ``expert_weights``: a pattern with ``{e}`` for the expert's number
    and ``{role}`` for gate / up / down; optional ``shared``: {``intermediate_size``, ``limit``,
    ``gate_weight``, ``up_weight``, ``down_weight``, optional ``mix_weight`` ([1, hidden]; without it the shared expert is
    added as it is)}.  Instead of ``router_weight``: ``table_weight`` (tensor name, int32 [``vocab_size``, top]) and
    ``vocab_size``.  Optional ``expert``:
    "clamped_glu" (the default, with ``limit``), "gelu_erf" (up and down only; the weight on the output; no
    ``limit``) or "silu_glu" (the weight on the output; no ``limit``).  Optional ``router``: {``correction_weight`` (tensor
    name, [experts]), ``groups``: {``count``, ``keep``}, ``normalise`` (bool), ``scale``, ``score`` ("sigmoid" or
    "softmax"), ``group_score`` ("top2": the sum of a group's two largest, or "max"), ``identity`` (experts without
    matrices behind ``num_experts``; router and correction have rows for them)}.  The result is a sum of 32-bit terms that the residual kernel takes."""
    graph_safe = True
    JOIN_MOST = 1.25      # a shared expert is padded with zeros to whole experts if that makes it no larger than this

    def __init__(self, params, ctx):
        super().__init__(params, ctx)
        self.hidden = int(self.param("hidden_size"))
        self.inter = int(self.param("intermediate_size"))
        self.n_experts = int(self.param("num_experts"))
        self.top = int(self.param("top"))
        self.expert = self.params.get("expert", "clamped_glu")
        if self.expert not in ("clamped_glu", "gelu_erf", "silu_glu"):
            raise ConfigError(f"routed_experts: unknown expert '{self.expert}' (known: clamped_glu, gelu_erf, silu_glu)")
        self.gated = self.expert != "gelu_erf"           # gate, up and down matrices
        self.limit = float(self.param("limit")) if self.expert == "clamped_glu" else 0.0
        self.act = None if self.expert == "clamped_glu" else self.expert
        ro = self.params.get("router") or {}
        self.correction_name = ro.get("correction_weight")
        groups = ro.get("groups") or {}
        self.groups, self.keep = int(groups.get("count", 1)), int(groups.get("keep", 1))
        self.normalise = bool(ro.get("normalise", False))
        self.route_scale = float(ro.get("scale", 1.0))
        self.score, self.group_score = ro.get("score", "sigmoid"), ro.get("group_score", "top2")
        if self.score not in kernels.ROUTER_SCORES or self.group_score not in kernels.GROUP_SCORES:
            raise ConfigError(f"routed_experts: unknown score '{self.score}' or group_score '{self.group_score}'")
        self.identity = int(ro.get("identity") or 0)
        self.n_choices = self.n_experts + self.identity
        if self.groups < 1 or self.n_choices % self.groups or not 1 <= self.keep <= self.groups:
            raise ConfigError(f"routed_experts: {self.n_choices} experts in {self.groups} groups of which {self.keep} are kept")
        if self.keep * (self.n_choices // self.groups) < self.top:
            raise ConfigError(f"routed_experts: the kept groups hold fewer than the {self.top} experts a token uses")
        if not 1 <= self.top <= self.n_choices or self.identity < 0:
            raise ConfigError(f"routed_experts: {self.top} of {self.n_choices} experts")
        self.table_name = self.params.get("table_weight")
        self.router_name = None if self.table_name else self.param("router_weight")
        self.vocab = int(self.param("vocab_size")) if self.table_name else 0
        if self.table_name and (ro or self.expert != "clamped_glu"):
            raise ConfigError("routed_experts: experts chosen by a table have no router and are of the kind clamped_glu")
        self.table = self.tables = None      # this layer's table; those of all layers that share a plan
        self.table_index = 0
        self.pattern = self.param("expert_weights")
        self.shared = self.params.get("shared")
        if self.shared is not None:
            missing = [k for k in ("intermediate_size", "limit", "gate_weight", "up_weight", "down_weight")
                       if k not in self.shared]
            if missing:
                raise ConfigError(f"routed_experts: 'shared' needs {missing}")
        self.mixed = self.shared is not None and bool(self.shared.get("mix_weight"))
        if self.mixed and self.table_name:
            raise ConfigError("routed_experts: a shared expert's 'mix_weight' rides with the router, which a table replaces")
        self.joined = 0                      # experts that the shared one adds to the routed ones (0: it runs by itself)
        if self.table_name and self.shared is not None:
            pieces = -(-int(self.shared["intermediate_size"]) // self.inter)
            if pieces * self.inter <= self.JOIN_MOST * int(self.shared["intermediate_size"]):
                self.joined = pieces

    def _name(self, e: int, role: str) -> str:
        return self.pattern.format(e=e, role=role)

    def weight_decls(self):
        h, f = self.hidden, self.inter
        if self.table_name:
            decls = [WeightDecl(self.table_name, (self.vocab, self.top), "choice_table", below=self.n_experts)]
        else:
            decls = [WeightDecl(self.router_name, (self.n_choices, h))]
        if self.correction_name:
            decls.append(WeightDecl(self.correction_name, (self.n_choices,), "norm"))
        for e in range(self.n_experts):
            if self.gated:
                decls.append(WeightDecl(self._name(e, "gate"), (f, h)))
            decls += [WeightDecl(self._name(e, "up"), (f, h)), WeightDecl(self._name(e, "down"), (h, f))]
        if self.shared is not None:
            sf, sh = int(self.shared["intermediate_size"]), self.shared
            decls += [WeightDecl(sh["gate_weight"], (sf, h)), WeightDecl(sh["up_weight"], (sf, h)),
                      WeightDecl(sh["down_weight"], (h, sf))]
            if self.mixed:
                decls.append(WeightDecl(sh["mix_weight"], (1, h)))
        return decls

    def load(self, weights):
        dt = self.ctx.compute_dtype
        E = range(self.n_experts)
        self.w_gate = (torch.stack([weights[self._name(e, "gate")] for e in E]).to(dt).contiguous()
                       if self.gated else None)
        self.correction = (weights[self.correction_name].to(torch.float32).contiguous()
                           if self.correction_name else None)
        self.w_up = torch.stack([weights[self._name(e, "up")] for e in E]).to(dt).contiguous()
        self.w_down = torch.stack([weights[self._name(e, "down")] for e in E]).to(dt).contiguous()
        rows = [] if self.table_name else [weights[self.router_name]]
        if self.mixed:
            rows.append(weights[self.shared["mix_weight"]].reshape(1, self.hidden))       # the shared expert's gate rides with the router
        if self.joined:
            self._join_shared(weights)
        elif self.shared is not None:
            sh = self.shared
            self.s_gate = weights[sh["gate_weight"]].to(dt).unsqueeze(0).contiguous()
            self.s_up = weights[sh["up_weight"]].to(dt).unsqueeze(0).contiguous()
            self.s_down = weights[sh["down_weight"]].to(dt).unsqueeze(0).contiguous()
        self.router = torch.cat(rows, dim=0).to(torch.float32).contiguous() if rows else None     # (router logits are 32-bit)
        if self.table_name:
            self.table = weights[self.table_name].to(torch.int32).contiguous()
            if not 0 <= int(self.table.min()) <= int(self.table.max()) < self.n_experts:
                raise ConfigError(f"routed_experts: {self.table_name} names an expert outside 0 .. {self.n_experts - 1}")
            if self.joined:
                more = torch.arange(self.n_experts, self.n_experts + self.joined, dtype=torch.int32, device=self.table.device)
                self.table = torch.cat([self.table, more.expand(self.vocab, -1)], dim=1).contiguous()
            self.tables = self.table.unsqueeze(0)

    def _join_shared(self, weights) -> None:
        """The shared expert's matrices behind the routed ones', in pieces of an expert's size (zeros behind the last)."""
        sh, n, f = self.shared, self.joined, self.inter
        pad = n * f - int(sh["intermediate_size"])

        def rows(name):
            w = torch.nn.functional.pad(weights[name].to(self.w_up.dtype), (0, 0, 0, pad))
            return w.view(n, f, self.hidden)

        down = torch.nn.functional.pad(weights[sh["down_weight"]].to(self.w_up.dtype), (0, pad))
        self.w_gate = torch.cat([self.w_gate, rows(sh["gate_weight"])]).contiguous()
        self.w_up = torch.cat([self.w_up, rows(sh["up_weight"])]).contiguous()
        self.w_down = torch.cat([self.w_down, down.view(self.hidden, n, f).permute(1, 0, 2)]).contiguous()

    @classmethod
    def link(cls, parts) -> None:
        groups: dict = {}
        for p in parts:
            if p.table is not None:
                groups.setdefault((p.n_experts, p.top, p.joined, p.vocab), []).append(p)
        for same in groups.values():
            tables = torch.stack([p.table for p in same]).contiguous()
            for i, p in enumerate(same):
                p.tables, p.table_index, p.table = tables, i, tables[i]

    def _el(self) -> int:
        return 4 if self.ctx.compute_dtype == torch.float32 else 2

    def _router_numel(self) -> int:
        return self.router.numel() if self.router is not None else 0

    def decode_bytes(self, lens) -> int:
        # the experts whose matrices are read: the expected number under a router that chooses evenly
        used = self.n_experts * (1.0 - (1.0 - self.top / self.n_choices) ** len(lens))
        mats = 3 if self.gated else 2
        total = int(mats * used * self.hidden * self.inter * self._el()) + 4 * self._router_numel()
        if self.shared is not None:
            total += 3 * self.hidden * int(self.shared["intermediate_size"]) * self._el()
        return total

    def prefill_flops(self, lens) -> int:
        top = self.top * self.n_experts / self.n_choices      # (expected: an identity expert has no products)
        per_token = int((3 if self.gated else 2) * self.hidden * self.inter * top) + self._router_numel()
        if self.shared is not None:
            per_token += 3 * self.hidden * int(self.shared["intermediate_size"])
        return 2 * sum(lens) * per_token

    def _plan(self, x, batch, tile: int):
        """(perm, plan, weights of the pairs or None, the shared expert's factor or None, the pairs' experts if some may be
        identity experts): the step's (token, choice) pairs sorted by expert."""
        T, top, dev, i32 = x.shape[0], self.top + self.joined, x.device, torch.int32
        n_experts = self.n_experts + self.joined
        cells = 1 + 3 * kernels.expert_max_tiles(T * top, n_experts, tile)
        if self.table is not None:       # known from the tokens: the plans of all layers that choose alike, made once a step
            key = ("expert_plans", self.tables.data_ptr(), tile)
            if key not in batch.aux:
                n = self.tables.shape[0]
                perms = torch.empty(n, T * top, dtype=i32, device=dev)
                plans = torch.empty(n, cells, dtype=i32, device=dev)
                kernels.expert_table_plan(perms, plans, batch.tokens, self.tables, n_experts, tile)
                batch.aux[key] = (perms, plans)
            perms, plans = batch.aux[key]
            return perms[self.table_index], plans[self.table_index], None, None, None
        ids = torch.empty(T, top, dtype=i32, device=dev)
        wts = torch.empty(T, top, dtype=torch.float32, device=dev)
        mix = torch.empty(T, dtype=torch.float32, device=dev) if self.mixed else None
        perm = torch.empty(T * top, dtype=i32, device=dev)
        plan = torch.empty(cells, dtype=i32, device=dev)
        few = kernels.route_plans_fit(T, self.n_choices, self.groups)
        kernels.expert_route(ids, wts, mix, x, self.router, self.n_choices, correction=self.correction,
                             groups=self.groups, keep=self.keep, normalise=self.normalise, out_scale=self.route_scale,
                             score=self.score, group_score=self.group_score,
                             plan_out=(perm, plan, self.n_experts, tile) if few else None)
        if not few:
            kernels.expert_plan(perm, plan, ids, self.n_experts, tile, identity=self.identity)
        return perm, plan, wts, mix, ids if self.identity else None

    def forward(self, x, batch):
        T, top, dev = x.shape[0], self.top + self.joined, x.device
        # bfloat16 with sizes the tensor-core products take: the rows in sorted order, then grouped products;
        # else the products on the CUDA cores (32-bit, or odd sizes), which fetch their rows themselves
        fast = (kernels.expert_rows_tc_supported(x, self.w_up) and self.inter % 8 == 0)
        act = self.act
        tile = kernels.expert_tc_tile(T * top, self.n_experts + self.joined) if fast else kernels.EXPERT_TILE
        perm, plan, wts, mix, ids = self._plan(x, batch, tile)
        second = (self.n_experts, float(self.shared["limit"])) if self.joined else None
        mid = torch.empty(T * top, self.inter, dtype=x.dtype, device=dev)
        out = torch.empty(top, T, self.hidden, dtype=torch.float32, device=dev)
        if fast:
            rows = torch.empty(T * top, self.hidden, dtype=x.dtype, device=dev)
            kernels.expert_gather(rows, x, perm, top, ids=ids, n_experts=self.n_experts, wts=wts, result=out)
            if self.gated:
                kernels.expert_rows_tc(mid, rows, self.w_gate, self.w_up, perm=perm, plan=plan, pair_weight=wts,
                                       n_tokens=T, top=top, limit=self.limit, tile=tile, second=second, act=act)
            else:
                kernels.expert_rows_tc(mid, rows, self.w_up, perm=perm, plan=plan, pair_weight=wts, n_tokens=T, top=top,
                                       tile=tile, act=act)
            kernels.expert_rows_tc(out, mid, self.w_down, perm=perm, plan=plan, n_tokens=T, top=top, tile=tile)
        else:
            if ids is not None:
                kernels.expert_gather(None, x, perm, top, ids=ids, n_experts=self.n_experts, wts=wts, result=out)
            if self.gated:
                kernels.expert_rows(mid, x, self.w_gate, self.w_up, perm=perm, plan=plan, pair_weight=wts, n_tokens=T,
                                    top=top, limit=self.limit, second=second, act=act)
            else:
                kernels.expert_rows(mid, x, self.w_up, perm=perm, plan=plan, pair_weight=wts, n_tokens=T, top=top, act=act)
            kernels.expert_rows(out, mid, self.w_down, perm=perm, plan=plan, n_tokens=T, top=top)
        if self.joined:
            return WeightedSum([(PartialSums(out[: self.top]), 1.0 / self.top), (PartialSums(out[self.top:]), 1.0)])
        terms = [(PartialSums(out), 1.0 / top if self.table is not None else 1.0)]
        if self.shared is not None:
            sf = int(self.shared["intermediate_size"])
            smid = torch.empty(T, sf, dtype=x.dtype, device=dev)
            sout = torch.empty(1, T, self.hidden, dtype=torch.float32, device=dev)
            rows_fn = kernels.expert_rows_tc if fast and sf % 8 == 0 else kernels.expert_rows
            rows_fn(smid, x, self.s_gate, self.s_up, scale_out=mix, n_tokens=T, top=1, limit=float(self.shared["limit"]))
            rows_fn(sout, smid, self.s_down, n_tokens=T, top=1)
            terms.append((sout[0], 1.0))
        return WeightedSum(terms)
