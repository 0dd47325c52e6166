"""Gated feed-forward with SiLU: down( silu(gate(x)) * up(x) ).

gate and up are one [2I, hidden] matrix (gate rows first) so that the projection is a
single product, as the reference's loader concatenates them
(python/vosti_kernels/model_families/qwen3/loader.py:55-58); the activation is
gate * sigmoid(gate) * up in float32 (kernels/triton_kernels/silu_mul.py:66-87).

Parameters besides `intermediate_size`: `tensor_names`, the checkpoint's names of the gate, up
and down matrices (default: Qwen3's), `float32_out`, for models whose residual stream is
float32: the down projection is then not rounded to the serving type, and `activation`: "silu"
(the default), "relu" or "relu2" (the square of relu) on the gate, or with `bias` "clamped": g sigmoid(`sigmoid_scale` g)
(u + 1) of g = min(gate x + bg, `limit`) and u = up x + bu clamped to [-limit, limit]. `bias`: all three projections have
biases (the tensor's name with ".b"); the down projection's joins in the kernel that reads the product next
(an arrangement that asks for `out_bias`), the others in the activation.

`ExpertMixture` is the same feed-forward as `experts` small ones, of which each token uses
the `top` with the largest router logits, weighted by the softmax over the chosen logits only.
Its experts may also be plain two-matrix feed-forwards, down(gelu(up(x))) with the exact (erf)
GELU, and its weights the chosen experts' shares of a softmax over all experts, divided by
their sum and multiplied by a constant. A third way of routing ("scored") chooses by corrected
softmax scores inside the best groups of experts, may count experts that return their input
among the routed ones, and may add a shared expert behind a per-token gate (see the class).
"""
from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..config.schema import ConfigError, PartSpec
from ..weights.loader import WeightSpec
from .base import FeedForward, register_part
from .linear import linear, prepare_weight, uses_tensor_cores


def stack_gate_up(gate: torch.Tensor, up: torch.Tensor, dtype: torch.dtype, activation: str = "silu"):
    """One [2I, hidden] matrix for the gate and up projections, and whether SiLU(gate)*up can be
    the tensor-core product's epilogue. If so, rows are laid out as blocks of 16 gate rows
    followed by their 16 up rows, so that both halves of an output land in one warp's slice of
    the accumulator; else the gate rows come first."""
    inter = gate.shape[0]
    common = torch.float32 if torch.float32 in (gate.dtype, up.dtype) else gate.dtype
    stacked = torch.cat([gate.to(common), up.to(common)], dim=0)
    fused = (dtype == torch.bfloat16 and inter % 16 == 0 and uses_tensor_cores(dtype, stacked)
             and activation in ops.FUSED_GLU_ACTIVATIONS)
    if not fused:
        return stacked.contiguous(), False
    return prepare_weight(interleave_gate_up(stacked[:inter], stacked[inter:]), dtype), True


def interleave_gate_up(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """Blocks of 16 gate rows followed by their 16 up rows."""
    inter, h = gate.shape
    return torch.stack([gate.view(-1, 16, h), up.view(-1, 16, h)], dim=1).reshape(2 * inter, h).contiguous()


def gated_activation(ctx, x, w_gate_up, fused: bool, activation: str = "silu", glu=(0.0, 0.0)):
    if fused:
        return ops.gemm_tc(ops.materialize(x), w_gate_up, ctx.status, swiglu=True, activation=activation)
    return ops.glu_mul(ops.materialize(linear(ctx, x, w_gate_up)), activation, *glu)


class SwiGLU(FeedForward):
    def __init__(self, spec: PartSpec, hidden_size: int):
        super().__init__(spec, hidden_size)
        self.inter = int(spec["intermediate_size"])
        if self.inter <= 0:
            raise ConfigError("swiglu: intermediate_size must be positive")
        self.names = tuple(spec.get("tensor_names") or ("gate_proj.weight", "up_proj.weight", "down_proj.weight"))
        self.float32_out = bool(spec.get("float32_out", False))
        self.activation = str(spec.get("activation", "silu") or "silu")
        self.partial_out = bool(spec.get("partial_out", False))   # with float32_out: the next kernel sums the down product's K splits
        self.has_bias, self.limit, self.sigmoid_scale = bool(spec.get("bias", False)), 0.0, 0.0
        self.bias_gate_up = self.out_bias = None
        if self.has_bias != (self.activation == "clamped"):
            raise ConfigError("swiglu: the clamped activation and biases go together")
        if self.has_bias:
            self.limit, self.sigmoid_scale = float(spec["limit"]), float(spec["sigmoid_scale"])
            if not self.limit > 0:
                raise ConfigError("swiglu: the clamped activation's limit must be positive")
        if self.activation not in ops.GLU_ACTIVATIONS:
            raise ConfigError(f"swiglu: activation is one of {sorted(ops.GLU_ACTIVATIONS)}")
        self.w_gate_up = self.w_down = None
        self.fused = self.fused_packed = False

    def weight_specs(self) -> Dict[str, WeightSpec]:
        h, i = self.hidden_size, self.inter
        gate, up, down = self.names
        specs = {gate: WeightSpec((i, h)), up: WeightSpec((i, h)), down: WeightSpec((h, i))}
        if self.has_bias:
            specs.update({gate + ".b": WeightSpec((i,), std=0.1), up + ".b": WeightSpec((i,), std=0.1), down + ".b": WeightSpec((h,), std=0.1)})
        return specs

    def load(self, tensors, dtype):
        gate, up, down = self.names
        self.w_down = prepare_weight(tensors[down], dtype)
        if self.has_bias:
            pair, biases = (tensors[gate], tensors[up]), (tensors[gate + ".b"].float(), tensors[up + ".b"].float())
            # blocks of 16 gate and 16 up rows where the tensor-core product may apply the activation itself
            self.fused = dtype == torch.bfloat16 and self.inter % 16 == 0 and all(uses_tensor_cores(dtype, w) for w in pair)
            if self.fused:
                self.w_gate_up = prepare_weight(interleave_gate_up(*pair), dtype)
                self.bias_gate_up = interleave_gate_up(*(b.view(-1, 1) for b in biases)).view(-1).contiguous()
                self.fused_packed = isinstance(self.w_gate_up, ops.PackedWeight)
            else:
                common = torch.float32 if torch.float32 in (pair[0].dtype, pair[1].dtype) else pair[0].dtype
                self.w_gate_up = prepare_weight(torch.cat([w.to(common) for w in pair], dim=0).contiguous(), dtype)
                self.bias_gate_up = torch.cat(biases).contiguous()
            self.out_bias = tensors[down + ".b"].float().contiguous()
            return
        self.w_gate_up, self.fused = stack_gate_up(tensors[gate], tensors[up], dtype, self.activation)

    def first_weight(self):
        return self.w_gate_up

    def _biased_activation(self, ctx, x):
        x = ops.materialize(x)
        if self.fused and self.fused_packed and x.shape[0] > ops.CLAMPED_EPILOGUE_FROM:
            return ops.gemm_tc_clamped(x, self.w_gate_up, self.bias_gate_up, ctx.status, limit=self.limit, sigmoid_scale=self.sigmoid_scale)
        product = linear(ctx, x, self.w_gate_up, out_dtype=torch.float32, allow_partial=True)
        return ops.glu_bias(product, self.bias_gate_up, x.dtype, block=16 if self.fused else 0, limit=self.limit,
                            sigmoid_scale=self.sigmoid_scale)

    def forward(self, ctx, x):
        if self.has_bias:
            y = linear(ctx, self._biased_activation(ctx, x), self.w_down, out_dtype=torch.float32, allow_partial=self.partial_out)
            # an arrangement that leaves the product unsummed adds `out_bias` itself
            y = y if self.partial_out else ops.affine_rows(y, bias=self.out_bias)
            return y if self.float32_out else ops.stream_sum(None, ops.materialize(y), out_dtype=x.dtype)
        mlp = gated_activation(ctx, x, self.w_gate_up, self.fused, self.activation)
        if self.float32_out:
            return linear(ctx, mlp, self.w_down, out_dtype=torch.float32, allow_partial=self.partial_out)
        return linear(ctx, mlp, self.w_down, allow_partial=True)     # summed by the norm that follows


register_part("feed_forward", "swiglu", SwiGLU, replace=True)


class ExpertMixture(FeedForward):
    """Parameters: experts, top, intermediate_size (of one expert), `float32_out`. Tensors:
    `router` [experts, hidden] and `e<i>.gate`, `e<i>.up`, `e<i>.down`. Further parameters:
    `gated` (default true; false: experts are down(gelu(up(x))), no `gate` tensors), `route`
    ("top_softmax", the default: softmax over the chosen logits; "softmax_renorm": softmax over
    all experts, the chosen scores divided by their sum + 1e-20; "softmax": the same, not divided; in bfloat16
    serving it takes the sorted way described for "table" below, the router's choice in the table's place) and `scale`, a constant on the
    weights (default 1).

    With `route` "scored" (experts without a gate only): the router has experts + `identity` rows;
    scores are s = softmax over all of them; rows are chosen by s + `correction` (a tensor,
    present if `correction` is true), among the rows of the `keep` best of `groups` equal groups of
    neighbouring rows (a group's score is its largest corrected score; the other groups' rows count as
    minus infinity); the weights are the chosen rows' s divided by their sum + 1e-20, times `scale`.
    The last `identity` rows are experts without tensors whose output is the feed-forward's input
    itself. `shared` > 0 adds a shared expert of that width (`shared.up`, `shared.down`, same form as
    the others) that runs for every token and is multiplied by sigmoid(w_sg . x), one number per
    token (`shared.sg` [1, hidden]). `activation` ("gelu" by default for experts without a gate, or
    "relu2", the square of relu) is the experts' and the shared expert's. The shared expert's matrices
    stand beside the experts' in the stacked matrices, its gate row under the router's rows, so the
    whole feed-forward is the router kernel, two products, the scaling pass and, with identity experts,
    one pass that adds their share of the input. Long portions take the sorted way described below
    too: identity rows are runs that are copied, the shared expert runs over all tokens afterwards.

    With `route` "table" there is no router: `table` [vocab, top] (integers, the entries of a row differ)
    names the experts of every token id, each with weight 1 / top; the step's ids come from the
    model's embedding part (`ctx.extras["token_ids"]`; `vocab`). In bfloat16 serving every step takes a sorted way
    of its own: one kernel sorts the (token, pick) pairs by expert and gathers their rows, two grouped
    products (`ops.gemm_tc_grouped`) run every expert over its own rows, on the device's word alone (no host
    decision, so that decode steps may be recorded; experts without a token are not read), and a token's
    picks are added by whatever kernel reads the result next. Sizes the grouped product does not take and
    float32 serving run the ways described above. Experts with a gate may be "clamped"
    (`activation`): g sigmoid(`sigmoid_scale` g) (u + 1) of g = min(gate x, `limit`) and u = up x clamped to
    [-limit, limit].

    The router's logits are float32. The experts' gate and up matrices stand side by side as one
    [2 * experts * I, hidden] matrix and their down matrices as one [hidden, experts * I]: every
    token's activation is computed for all experts by one product, each expert's slice is
    multiplied by the token's weight for it (zero if it was not chosen), and one more product
    sums the chosen experts' outputs. No launch depends on the router's choice, so a step may be
    replayed from a CUDA graph.

    A step that brings portions of prompts (`GROUPED_FROM` tokens or more, not all of them single
    tokens; such a step is never recorded as a graph) takes another way, in which no expert
    computes a token that did not choose it: the (token, pick) pairs are sorted by expert on the
    device, the host reads how many each expert got (one synchronisation), every expert with
    work multiplies its run of gathered rows, and a last kernel adds every token's picks in pick
    order. The experts' gate and up matrices are kept a second time for it, one per expert."""

    GROUPED_FROM = 256
    # The scored router's sorted way pays one host synchronisation and some thirty small launches a
    # layer; measured at 8 experts of which 2 are chosen (2,048 tokens) it lost to the side-by-side
    # product (2.85 against 2.47 ms a prompt of a 4-layer model), so it is taken from this many
    # experts per pick on.
    GROUPED_MIN_RATIO = 8

    def __init__(self, spec: PartSpec, hidden_size: int):
        super().__init__(spec, hidden_size)
        self.experts, self.top = int(spec["experts"]), int(spec["top"])
        self.inter = int(spec["intermediate_size"])
        self.float32_out = bool(spec.get("float32_out", False))
        self.gated = bool(spec.get("gated", True))
        self.route, self.scale = spec.get("route", "top_softmax"), float(spec.get("scale", 1.0))
        self.identity = int(spec.get("identity", 0) or 0)
        self.has_correction = bool(spec.get("correction", False))
        self.groups, self.keep = int(spec.get("groups", 1) or 1), int(spec.get("keep", 1) or 1)
        self.shared = int(spec.get("shared", 0) or 0)
        self.partial_out = bool(spec.get("partial_out", False))
        self.activation = spec.get("activation") or ("gelu" if not self.gated else None)
        self.glu, self.gate_activation = (0.0, 0.0), "silu"
        self.table, self.vocab = None, int(spec.get("vocab", 0) or 0)
        if self.gated and self.activation == "clamped":
            self.gate_activation, self.activation = "clamped", None
            self.glu = (float(spec["limit"]), float(spec["sigmoid_scale"]))
            if not self.glu[0] > 0:
                raise ConfigError("moe: the clamped activation's limit must be positive")
        self.correction = None
        if self.experts <= 0 or not 0 < self.top <= self.experts + self.identity or self.inter <= 0:
            raise ConfigError("moe: experts, top (at most experts) and intermediate_size must be positive")
        if self.route not in ("top_softmax", "softmax_renorm", "softmax", "scored", "table") or self.scale != self.scale:
            raise ConfigError("moe: route is 'top_softmax', 'softmax_renorm', 'softmax', 'scored' or 'table' and scale a number")
        if self.route == "table" and (not self.gated or self.scale != 1.0 or self.vocab <= 0):
            raise ConfigError("moe: route 'table' takes gated experts, no scale, and the size of the vocabulary")
        if self.route != "scored" and (self.identity or self.has_correction or self.groups != 1 or self.shared
                                       or self.activation not in (None, "gelu")):
            raise ConfigError("moe: identity experts, a correction, groups, a shared expert and other activations need route 'scored'")
        if self.route == "scored":
            routed = self.experts + self.identity
            if self.gated or self.activation not in ("gelu", "relu2"):
                raise ConfigError("moe: route 'scored' takes experts without a gate, with activation 'gelu' or 'relu2'")
            if self.identity < 0 or self.shared < 0 or self.groups < 1 or routed % self.groups or not 1 <= self.keep <= self.groups:
                raise ConfigError("moe: groups must divide experts + identity, and keep lie between 1 and groups")
            if self.top > routed // self.groups * self.keep:
                raise ConfigError("moe: top exceeds the experts of the kept groups")
        self.router = self.w_gate_up = self.w_down = self.grouped = None
        self.fused, self.per_expert = False, []

    def weight_specs(self) -> Dict[str, WeightSpec]:
        h, i = self.hidden_size, self.inter
        if self.route == "table":
            specs = {"table": WeightSpec((self.vocab, self.top), integer=True, distinct_below=self.experts)}
        else:
            specs = {"router": WeightSpec((self.experts + self.identity, h), std=0.5)}
        if self.has_correction:
            specs["correction"] = WeightSpec((self.experts + self.identity,), std=0.05)
        if self.shared:
            specs.update({"shared.up": WeightSpec((self.shared, h)), "shared.down": WeightSpec((h, self.shared)),
                          "shared.sg": WeightSpec((1, h), std=0.5)})
        for e in range(self.experts):
            specs.update({f"e{e}.up": WeightSpec((i, h)), f"e{e}.down": WeightSpec((h, i))})
            if self.gated:
                specs[f"e{e}.gate"] = WeightSpec((i, h))
        return specs

    def load(self, tensors, dtype):
        self.grouped, self.per_expert = None, []
        if self.route == "table":
            self.table = tensors["table"].to(torch.int32).contiguous()
            if self.table.numel() and (int(self.table.min()) < 0 or int(self.table.max()) >= self.experts):
                raise ConfigError(f"moe: the table names experts outside 0 .. {self.experts - 1}")
        else:
            self.router = tensors["router"].float().contiguous()        # 32-bit logits from exact 32-bit products
        if self.route == "scored":
            return self._load_scored(tensors, dtype)
        if self.route == "table":
            rows = self.table.sort(dim=1).values
            if self.top > 1 and bool((rows[:, 1:] == rows[:, :-1]).any()):
                raise ConfigError("moe: a row of the table names an expert twice")
            if self.top < self.experts and self._load_grouped(tensors, dtype):
                return
        if self.route == "softmax" and self.gated and self.top < self.experts and self._load_grouped(tensors, dtype):
            return
        up = torch.cat([tensors[f"e{e}.up"] for e in range(self.experts)], dim=0)
        if self.gated:
            gate = torch.cat([tensors[f"e{e}.gate"] for e in range(self.experts)], dim=0)
            self.w_gate_up, self.fused = stack_gate_up(gate, up, dtype, self.gate_activation)
        else:
            self.w_gate_up, self.fused = prepare_weight(up.contiguous(), dtype), False
        self.w_down = prepare_weight(torch.cat([tensors[f"e{e}.down"] for e in range(self.experts)], dim=1).contiguous(), dtype)
        self.per_expert = []
        if self.top < self.experts:
            for e in range(self.experts):
                if self.gated:
                    gate_up, fused = stack_gate_up(tensors[f"e{e}.gate"], tensors[f"e{e}.up"], dtype, self.gate_activation)
                else:
                    gate_up, fused = prepare_weight(tensors[f"e{e}.up"], dtype), False
                self.per_expert.append((gate_up, fused, prepare_weight(tensors[f"e{e}.down"], dtype)))

    def _load_grouped(self, tensors, dtype) -> bool:
        """The experts one after the other for the grouped products, if those take their sizes."""
        downs = [tensors[f"e{e}.down"] for e in range(self.experts)]
        pairs = [(tensors[f"e{e}.gate"], tensors[f"e{e}.up"]) for e in range(self.experts)]
        if (dtype != torch.bfloat16 or self.inter % 16 or self.gate_activation not in ops.GROUPED_GLU_ACTIVATIONS
                or not all(uses_tensor_cores(dtype, w) for w in downs + [w for pair in pairs for w in pair])):
            return False
        self.grouped = (ops.ExpertWeights([interleave_gate_up(g, u) for g, u in pairs]), ops.ExpertWeights(downs))
        return True

    def _load_scored(self, tensors, dtype):
        ups = [tensors[f"e{e}.up"] for e in range(self.experts)]
        downs = [tensors[f"e{e}.down"] for e in range(self.experts)]
        if self.shared:
            # the shared expert beside the others; its gate row under the router's
            ups.append(tensors["shared.up"])
            downs.append(tensors["shared.down"])
            self.router = torch.cat([self.router, tensors["shared.sg"].float().reshape(1, -1)], dim=0).contiguous()
        if self.has_correction:
            self.correction = tensors["correction"].float().contiguous()
        self.w_gate_up, self.fused = prepare_weight(torch.cat(ups, dim=0).contiguous(), dtype), False
        self.w_down = prepare_weight(torch.cat(downs, dim=1).contiguous(), dtype)
        # for long portions every expert (and the shared one, last) multiplies its own rows: the matrices one by one
        self.per_expert = []
        if self.top < self.experts + self.identity:
            self.per_expert = [(prepare_weight(up, dtype), False, prepare_weight(down, dtype)) for up, down in zip(ups, downs)]

    def _grouped_scored(self, ctx, x, chosen, weights, dense):
        """No expert computes a token that did not choose it: the (token, pick) pairs sorted by routed row
        (identity rows included), a product pair per expert with work, the identity rows' runs copied,
        a token's picks added in pick order, then the shared expert over all tokens."""
        routed = self.experts + self.identity
        offsets, rows, where = ops.moe_group(chosen, routed)
        gathered = ops.gather_rows(x, rows, ctx.status)
        bounds = offsets.tolist()                      # the host learns the rows' shares here
        y = torch.empty((rows.shape[0], self.hidden_size), dtype=torch.float32, device=x.device)
        for e in range(routed):
            lo, hi = bounds[e], bounds[e + 1]
            if hi <= lo:
                continue
            if e >= self.experts:
                y[lo:hi].copy_(gathered[lo:hi])        # an expert that returns its input
                continue
            up, _, down = self.per_expert[e]
            act = ops.moe_scale(ops.materialize(linear(ctx, gathered[lo:hi], up)), None, self.inter, activation=self.activation)
            y[lo:hi].copy_(ops.materialize(linear(ctx, act, down, out_dtype=torch.float32)))
        out = ops.moe_combine(y, where, weights)
        if self.shared:
            up, _, down = self.per_expert[self.experts]
            gate = dense[:, self.experts:].contiguous()
            act = ops.moe_scale(ops.materialize(linear(ctx, x, up)), gate, self.shared, activation=self.activation)
            out = ops.stream_sum(out, ops.materialize(linear(ctx, act, down, out_dtype=torch.float32)))
        return out

    def _forward_scored(self, ctx, x):
        chosen, weights, dense, ident = ops.moe_router_scored(
            x, self.router, self.top, identity=self.identity, correction=self.correction, groups=self.groups, keep=self.keep,
            gate_row=bool(self.shared), scale=self.scale)
        if (self.per_expert and x.shape[0] >= self.GROUPED_FROM and self.experts > self.GROUPED_MIN_RATIO * self.top
                and not getattr(ctx, "all_decode", True) and not torch.cuda.is_current_stream_capturing()):
            y = self._grouped_scored(ctx, x, chosen, weights, dense)
            return y if self.float32_out else ops.stream_sum(None, y, out_dtype=x.dtype)
        act = ops.moe_scale(ops.materialize(linear(ctx, x, self.w_gate_up)), dense, self.inter, activation=self.activation,
                            tail=self.shared)
        y = linear(ctx, act, self.w_down, out_dtype=torch.float32, allow_partial=self.partial_out and not self.identity)
        if self.identity:
            y = ops.moe_identity(y, ident, x)
        return y if self.float32_out else ops.stream_sum(None, ops.materialize(y), out_dtype=x.dtype)

    def first_weight(self):
        return self.w_gate_up

    def _activation(self, ctx, x, w_first, fused, dense=None):
        """An expert's (or all experts') hidden activation, times the dense weights if given."""
        if self.gated:
            act = gated_activation(ctx, x, w_first, fused, self.gate_activation, self.glu)
            return act if dense is None else ops.moe_scale(act, dense, self.inter)
        return ops.moe_scale(ops.materialize(linear(ctx, x, w_first)), dense, self.inter, gelu=True)

    def _grouped(self, ctx, x, chosen, weights):
        offsets, rows, where = ops.moe_group(chosen, self.experts)
        gathered = ops.gather_rows(x, rows, ctx.status)
        bounds = offsets.tolist()                      # the host learns the experts' shares here
        y = torch.empty((rows.shape[0], self.hidden_size), dtype=torch.float32, device=x.device)
        for e, (gate_up, fused, down) in enumerate(self.per_expert):
            lo, hi = bounds[e], bounds[e + 1]
            if hi > lo:
                act = self._activation(ctx, gathered[lo:hi], gate_up, fused)
                y[lo:hi].copy_(linear(ctx, act, down, out_dtype=torch.float32))
        return ops.moe_combine(y, where, weights)

    def _sorted_products(self, ctx, x, ids, table, weights=None):
        """The experts over their own rows: `table` by token id, or (ids None) a router's choice with its weights."""
        gathered, offsets, where = ops.moe_dispatch(ids, table, self.experts, x, ctx.status)
        act = ops.gemm_tc_grouped(gathered, self.grouped[0], offsets, x.shape[0], ctx.status, activation=self.gate_activation,
                                  glu=self.glu)
        y = ops.gemm_tc_grouped(act, self.grouped[1], offsets, x.shape[0], ctx.status, out_dtype=torch.float32,
                                allow_partial=self.partial_out)
        y = ops.PickedSum(y, where, 1.0 / self.top, weights)
        return y if self.partial_out else y.materialize()

    def _forward_table(self, ctx, x):
        ids = ctx.extras.get("token_ids")
        if ids is None:
            raise ConfigError("moe: route 'table' needs the step's token ids, which the model's embedding does not publish")
        if self.grouped is not None:
            y = self._sorted_products(ctx, x, ids, self.table)
        elif (self.per_expert and x.shape[0] >= self.GROUPED_FROM and not getattr(ctx, "all_decode", True)
                and not torch.cuda.is_current_stream_capturing()):
            chosen, weights, _ = ops.moe_table(ids, self.table, self.experts)
            y = self._grouped(ctx, x, chosen, weights)
        else:
            act = ops.moe_scale_table(self._activation(ctx, x, self.w_gate_up, self.fused), ids, self.table, self.inter)
            y = linear(ctx, act, self.w_down, out_dtype=torch.float32, allow_partial=self.partial_out)
        return y if self.float32_out else ops.stream_sum(None, ops.materialize(y), out_dtype=x.dtype)

    def forward(self, ctx, x):
        x = ops.materialize(x)
        if self.route == "scored":
            return self._forward_scored(ctx, x)
        if self.route == "table":
            return self._forward_table(ctx, x)
        over_all = {"softmax_renorm": 1, "softmax": 2}.get(self.route, 0)
        chosen, weights, dense = ops.moe_router(x, self.router, self.top, over_all=over_all, scale=self.scale)
        if self.grouped is not None:
            y = self._sorted_products(ctx, x, None, chosen, weights)
            return y if self.float32_out else ops.stream_sum(None, ops.materialize(y), out_dtype=x.dtype)
        if (self.per_expert and x.shape[0] >= self.GROUPED_FROM and not getattr(ctx, "all_decode", True)
                and not torch.cuda.is_current_stream_capturing()):
            out = self._grouped(ctx, x, chosen, weights)
            return out if self.float32_out else out.to(x.dtype)
        act = self._activation(ctx, x, self.w_gate_up, self.fused, dense)
        if self.float32_out:
            return linear(ctx, act, self.w_down, out_dtype=torch.float32)
        return linear(ctx, act, self.w_down, allow_partial=True)


register_part("feed_forward", "moe", ExpertMixture, replace=True)
