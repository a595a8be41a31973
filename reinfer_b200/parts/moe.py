"""A mixture of small feed-forward experts.  Each token uses `top` of `experts + identity` choices:

    s      = softmax(router(x))                  over all choices, 32-bit
    chosen = the `top` largest of s + correction (the correction steers the choice only)
    out    = sum over the chosen e of s[e] * expert_e(x)       (the weights are not renormalised)

An expert is down(act(up(x))) with act = relu(.)^2 and no biases; the last `identity` choices are experts that
hand their input back unchanged and have no tensors.

Two options make the other common form.  `gated=True`: an expert is down(f(gate(x)) * up(x)) with f = `activation`
(silu or the tanh form of gelu), three tensors an expert.  `route="chosen_logits"`: the vector beside the router's matrix
(`correction_name`) is a bias of the logits, the `top` largest logits are chosen and the weights are the softmax over the
chosen logits alone.

A third route, `route="group_sigmoid"`: the scores are the sigmoids of the router's outputs, and the weights are the chosen
scores over their total.  `groups` = (count, keep): expert e sits in group e // (experts / count); groups are ranked by what
their top two values of s + correction add up to, and the choice runs over the `keep` first-ranked groups alone.

`shared` = {"inner", "names": ((gate,) up, down), "gate_name", "limit"}: one more expert of a size of its own that every token
takes, times the sigmoid of one number (its row joins the router's matrix; not with "chosen_logits").  In the stacked form its
columns follow the experts'.  `weight_scale`: a factor on the chosen experts' weights; `out_scale`: one on the whole output (both
go into the weights).  An expert without a gate matrix is down(f(up(x))) with f = `activation`: "relu2" (unless said otherwise)
or a gelu.  The gated activation "clamp_swish" takes `limit`: g' sigmoid(1.702 g') (u' + 1) with g' = min(g, limit) and u' = u cut to
[-limit, limit] (the shared expert has a limit of its own).

Over many tokens (a prompt portion) the stacked products compute every expert for every token where a token uses `top`
of them.  A mixture in bfloat16 (gated, or with a shared expert's route) whose tokens use at most half of the experts then takes the grouped form
(`ops.moe_grouped_experts`): rows sorted by expert on the device, two grouped tensor-core products over the chosen
pairs alone, the weighted sum per token in the order of the experts.  A decode step's few tokens touch most experts
anyway and keep the stacked form.

The experts' up matrices are stacked by rows at load and their down matrices side by side, and the router's choice
is kept dense (gates [T, experts], zero where an expert was not chosen): one product makes every expert's inner
activations, the activation kernel multiplies each by its token's gate, and one product with the stacked down
matrices is then the weighted sum over the chosen experts, an expert that was not chosen adding exact zeros.  A
token's result never depends on what else is in the batch.
"""
from __future__ import annotations

import os
from typing import Optional

import torch

from .. import ops
from ..weights.params import ParamSpec
from .base import FeedForward, register_part
from .ffn import activated
from .linear import matmul, matmul_into_residual


GROUPED = os.environ.get("REINFER_B200_MOE_GROUPED", "1") != "0"    # 0: the stacked products at every token count
GROUPED_FROM = 256                                                  # tokens of a step from which the grouped form is taken


class ExpertMixture(FeedForward):
    def __init__(self, hidden: int, experts: int, top: int, inner: int, identity: int = 0,
                 expert_names=("e{}.up", "e{}.down"), router_name: str = "router", correction_name: str = "correction",
                 gated: bool = False, activation: Optional[str] = None, route: str = "scores", groups=None, shared=None,
                 out_scale: float = 1.0, weight_scale: float = 1.0, limit: float = 0.0):
        """expert_names: (up, down), or with `gated` (gate, up, down) - patterns that take the expert's index."""
        self.hidden, self.E, self.I, self.top, self.ff = int(hidden), int(experts), int(identity), int(top), int(inner)
        if self.E < 1 or self.I < 0 or not 1 <= self.top <= self.E + self.I:
            raise ValueError(f"expert mixture: {self.E} experts, {self.I} identity experts, top {self.top}")
        self.gated, self.route, self.out_scale, self.weight_scale = bool(gated), route, float(out_scale), float(weight_scale)
        self.activation = activation or ("silu" if self.gated else "relu2")
        if route not in ops.MOE_MODES or self.activation not in (ops.GLU_ACTS if self.gated else ops.ACTS):
            raise ValueError(f"expert mixture: route {route!r}, activation {activation!r}")
        self.groups = (int(groups[0]), int(groups[1])) if groups else None
        self.shared = dict(shared) if shared else None
        if (route != "group_sigmoid" and self.groups) or (route == "chosen_logits" and (self.shared or self.out_scale != 1.0 or self.weight_scale != 1.0)):
            raise ValueError("expert mixture: groups go with the route 'group_sigmoid', a shared expert and factors with any but 'chosen_logits'")
        if self.I and (self.shared or self.out_scale != 1.0 or self.weight_scale != 1.0):
            raise ValueError("expert mixture: identity experts beside a shared expert or factors")
        self.limits = (float(limit), float(self.shared.get("limit", 0.0)) if self.shared else 0.0) if self.activation == "clamp_swish" else None
        if self.limits and (self.limits[0] <= 0 or (self.shared and self.limits[1] <= 0)):
            raise ValueError(f"expert mixture: limits {self.limits}")
        if self.I and route == "group_sigmoid":
            raise ValueError("expert mixture: the route 'group_sigmoid' knows no identity experts")
        if self.shared and len(self.shared["names"]) != (3 if self.gated else 2):
            raise ValueError("expert mixture: the shared expert has the experts' form")
        # routes whose weights are complete in one row per token (a shared expert's gate last): the stacked form can be cut into
        # inner and outer, and the grouped form has the shared expert as a pair of its own
        self.whole_rows = route == "group_sigmoid" or (route == "scores" and self.gated and not self.I)
        if self.groups and (self.E % self.groups[0] or not 1 <= self.groups[1] <= self.groups[0] or
                            self.E // self.groups[0] * self.groups[1] < self.top):
            raise ValueError(f"expert mixture: {self.E} experts in groups {self.groups}, top {self.top}")
        self.sff = int(self.shared["inner"]) if self.shared else 0
        if len(expert_names) != (3 if self.gated else 2):
            raise ValueError("expert mixture: tensor names for (gate,) up and down")
        self.gate_name = expert_names[0] if self.gated else None
        self.up_name, self.down_name = expert_names[-2:]
        self.router_name, self.correction_name = router_name, correction_name
        self.w_up = self.w_down = self.w_router = self.correction = None

    def param_specs(self):
        h, n = self.hidden, self.E + self.I
        out = {self.router_name: ParamSpec((n, h), std=0.1), self.correction_name: ParamSpec((n,), std=0.02)}
        for e in range(self.E):
            if self.gated:
                out[self.gate_name.format(e)] = ParamSpec((self.ff, h))
            out[self.up_name.format(e)] = ParamSpec((self.ff, h))
            out[self.down_name.format(e)] = ParamSpec((h, self.ff))
        if self.shared:
            *ups, down = self.shared["names"]
            out.update({u: ParamSpec((self.sff, h)) for u in ups})
            out.update({down: ParamSpec((h, self.sff)), self.shared["gate_name"]: ParamSpec((1, h), std=0.1)})
        return out

    def bind(self, t):
        ups = [t[self.up_name.format(e)] for e in range(self.E)]
        downs = [t[self.down_name.format(e)] for e in range(self.E)]
        if self.shared:
            ups, downs = ups + [t[self.shared["names"][-2]]], downs + [t[self.shared["names"][-1]]]
        if self.gated:
            # [all gates; all ups], the shared expert's last in each half: one gated pair over E * ff (+ shared) columns
            ups = [t[self.gate_name.format(e)] for e in range(self.E)] + ([t[self.shared["names"][0]]] if self.shared else []) + ups
        if len({m.dtype for m in ups + downs}) > 1:
            ups, downs = [m.float() for m in ups], [m.float() for m in downs]
        self.w_up = torch.cat(ups, dim=0).contiguous()                  # [E * ff (+ shared), h]  (gated: twice as many rows)
        self.w_down = torch.cat(downs, dim=1).contiguous()              # [h, E * ff (+ shared)]
        self.w_router = t[self.router_name]
        if self.shared:
            sg = t[self.shared["gate_name"]]
            if sg.dtype != self.w_router.dtype:
                sg, self.w_router = sg.float(), self.w_router.float()
            self.w_router = torch.cat([self.w_router, sg], dim=0).contiguous()
        self.correction = t[self.correction_name].float().contiguous()

    def forward(self, ctx, xn, residual):
        T = xn.shape[0]
        if self.whole_rows:
            return self._whole_rows(ctx, xn, residual)
        gates, ident = ops.moe_router(xn, self.w_router, self.correction, self.E, self.top, mode=self.route)     # 32-bit, product and choice
        if self.gated and ident is None and T >= GROUPED_FROM and 2 * self.top <= self.E and GROUPED:
            # (a step of this many tokens is beyond the products that do the next norm's work: nothing is lost by not asking)
            fresh = bool(getattr(ctx, "fresh_residual", False))
            if ops.moe_grouped_experts(xn, gates, self.top, self.w_up, self.w_down, self.ff, self.activation, residual, store=fresh):
                ctx.fresh_residual = False
                return None
        if self.gated:
            act = torch.empty((T, self.E * self.ff), dtype=xn.dtype, device=xn.device)
            # bfloat16: the activation and the expert's weight in the product's epilogue; else 32-bit sums and a kernel behind them
            fused = T and xn.dtype == torch.bfloat16 and self.w_up.dtype == torch.bfloat16 and \
                ops.gemm_bf16_swiglu(xn, self.w_up, act, act=self.activation, gates=gates, ff=self.ff)
            if T and not fused:
                ops.glu_act(matmul(ctx, xn, self.w_up, out_dtype=torch.float32), act, self.activation, None, gates, self.ff)
        else:
            act = activated(ctx, xn, self.w_up, self.activation, gates=gates, ff=self.ff, blocks=self.E)
        if ident is not None:
            ctx.norm_ahead = None           # the stream is not complete behind the down product: nobody's rows can be made there
        left = matmul_into_residual(ctx, act, self.w_down, residual)
        if ident is not None and T:
            # the identity experts' share: the token's own row times the sum of their chosen scores - left to the
            # block where it adds such a term on its way, else added here
            if getattr(ctx, "takes_row_multiple", False) and getattr(ctx, "row_multiple", None) is None:
                ctx.row_multiple = (ident, xn)
            else:
                ops.rows_axpy(residual if left is None else left[0], ident, xn)
        return left

    def splits(self, T: int) -> bool:
        """Whether `inner` and `outer` are the whole of a step of T tokens (the stacked form)."""
        return self.whole_rows and T < GROUPED_FROM

    def _routed(self, xn, side_by_side: bool):
        return ops.moe_router(xn, self.w_router, self.correction, self.E, self.top, mode=self.route, groups=self.groups,
                              scale=self.weight_scale * self.out_scale, shared=self.shared is not None, side_by_side=side_by_side,
                              shared_scale=self.out_scale)

    def _pair(self, ctx, xn, w, cols: int, gates, ff: int, blocks: int, limits, up_row: int = 0):
        """The gated pair over `cols` columns of w ([gates; ups], or the up rows `up_row` below the gate rows) with its weights."""
        act = torch.empty((xn.shape[0], cols), dtype=xn.dtype, device=xn.device)
        if xn.shape[0] == 0:
            return act
        # bfloat16: activation and weights in the product's epilogue; else 32-bit sums and a kernel behind them
        if xn.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and \
                ops.gemm_bf16_swiglu(xn, w, act, act=self.activation, gates=gates, ff=ff, blocks=blocks, limits=limits, up_row=up_row):
            return act
        if up_row:
            w = torch.cat([w[:cols], w[up_row:up_row + cols]])
        ops.glu_act(matmul(ctx, xn, w, out_dtype=torch.float32), act, self.activation, None, gates, ff, blocks, limits)
        return act

    def _stacked(self, ctx, xn, gates):
        if self.gated:
            return self._pair(ctx, xn, self.w_up, self.w_down.shape[1], gates, self.ff, self.E, self.limits)
        return activated(ctx, xn, self.w_up, self.activation, gates=gates, ff=self.ff, blocks=self.E)

    def inner(self, ctx, xn):
        """Router, up product and activation of all experts; touches neither the stream nor the context."""
        return self._stacked(ctx, xn, self._routed(xn, True)[0])

    def outer(self, ctx, act, residual):
        return matmul_into_residual(ctx, act, self.w_down, residual)

    def _whole_rows(self, ctx, xn, residual):
        T, n, total = xn.shape[0], self.E * self.ff, self.w_down.shape[1]
        if self.splits(T):
            return self.outer(ctx, self.inner(ctx, xn), residual)
        grouped = GROUPED and 2 * self.top <= self.E and xn.dtype == torch.bfloat16 and n % 8 == 0
        gates, sg = self._routed(xn, not grouped)
        if grouped:
            w = self.w_up if self.gated else self.w_up[:n]
            if ops.moe_grouped_experts(xn, gates, self.top, w, self.w_down[:, :n], self.ff, self.activation, residual,
                                       store=bool(getattr(ctx, "fresh_residual", False)), gated=self.gated,
                                       limit=self.limits[0] if self.limits else 0.0, up_row=total if self.gated else 0):
                ctx.fresh_residual = False
                if self.shared is None:
                    return None
                if self.gated:
                    act = self._pair(ctx, xn, self.w_up[n:], self.sff, sg, self.sff, 1, self.limits[1] if self.limits else None, up_row=total)
                else:
                    act = activated(ctx, xn, self.w_up[n:], self.activation, gates=sg, ff=self.sff, blocks=1)
                return matmul_into_residual(ctx, act, self.w_down[:, n:], residual)
            if sg is not None:
                gates = torch.cat([gates, sg], dim=1)
        return self.outer(ctx, self._stacked(ctx, xn, gates), residual)


register_part("ffn", "expert_mixture", ExpertMixture)
