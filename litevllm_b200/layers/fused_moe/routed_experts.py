"""Routed experts without biases, each ``W_down (act(W_gate x) * (W_up x))`` (``act`` may be the clipped form of
``ops.gated_linear``).  The router's logits come from outside (they
may share a product with other small 32-bit projections) and the weighted sum over the chosen experts is left to the
caller's residual add.

    s = score(z);  chosen: the ``top`` largest s + correction among the best groups;  weight = s * scale (optionally
    divided by the sum over the chosen)

``groups`` equal groups of neighbouring experts are ranked by the sum of their ``group_best`` largest s + correction; only
experts of the best ``keep`` can be chosen.  The last ``identity`` router outputs stand for experts that return their input.
"""
from __future__ import annotations

import torch
from torch import nn

from ...ops import moe


class RoutedExperts(nn.Module):
    def __init__(self, hidden: int, inter: int, experts: int, top: int, dtype, act: str = "silu", score: str = "sigmoid",
                 groups: int = 1, keep: int = 1, scale: float = 1.0, renormalize: bool = False, group_best: int = 2,
                 identity: int = 0, act_limit: float = 0.0):
        super().__init__()
        self.E, self.top, self.act, self.score, self.inter = experts, top, act, score, inter
        self.groups, self.keep, self.scale, self.renormalize = groups, keep, float(scale), renormalize
        self.group_best, self.act_limit, self.outputs = group_best, float(act_limit), experts + identity
        self.w_gate_up = nn.Parameter(torch.empty(experts, 2 * inter, hidden, dtype=dtype), requires_grad=False)
        self.w_down = nn.Parameter(torch.empty(experts, hidden, inter, dtype=dtype), requires_grad=False)
        self.correction = nn.Parameter(torch.zeros(self.outputs, dtype=torch.float32), requires_grad=False)

    def destinations(self, prefix: str) -> dict:
        """Checkpoint name -> where its values go."""
        d = {}
        for e in range(self.E):
            d[f"{prefix}e{e}.gate"] = self.w_gate_up[e, :self.inter]
            d[f"{prefix}e{e}.up"] = self.w_gate_up[e, self.inter:]
            d[f"{prefix}e{e}.down"] = self.w_down[e]
        d[prefix + "correction"] = self.correction
        return d

    def forward(self, x, logits) -> moe.RoutedRows:
        """x [T, hidden], logits fp32 [T, experts + identity]."""
        ids, w = moe.route(logits, self.top, mode=self.score, bias=self.correction, renormalize=self.renormalize,
                           routed_scale=self.scale, groups=self.groups, keep_groups=self.keep,
                           group_best=self.group_best)
        return moe.expert_rows(x, self.w_gate_up, self.w_down, ids, w, self.act, self.act_limit, self.outputs > self.E)


class AssignedExperts(nn.Module):
    """The same experts without a router: a table gives every token id its ``top`` experts, each of weight 1 / top."""

    def __init__(self, hidden: int, inter: int, experts: int, top: int, vocab: int, dtype, act: str = "silu"):
        super().__init__()
        self.E, self.top, self.act, self.inter = experts, top, act, inter
        self.w_gate_up = nn.Parameter(torch.empty(experts, 2 * inter, hidden, dtype=dtype), requires_grad=False)
        self.w_down = nn.Parameter(torch.empty(experts, hidden, inter, dtype=dtype), requires_grad=False)
        self.table = nn.Parameter(torch.zeros(vocab, top, dtype=torch.int32), requires_grad=False)

    def _take_table(self, tensor: torch.Tensor) -> None:
        if tuple(tensor.shape) != tuple(self.table.shape):
            raise ValueError(f"expert table has shape {tuple(tensor.shape)}, the configuration asks for {tuple(self.table.shape)}")
        if tensor.is_floating_point() or int(tensor.min()) < 0 or int(tensor.max()) >= self.E:
            raise ValueError(f"expert tables hold integers below {self.E}")
        self.table.data.copy_(tensor.to(torch.int32))

    def destinations(self, prefix: str) -> dict:
        """Checkpoint name -> where its values go."""
        d = {prefix + "table": self._take_table}
        for e in range(self.E):
            d[f"{prefix}e{e}.gate"] = self.w_gate_up[e, :self.inter]
            d[f"{prefix}e{e}.up"] = self.w_gate_up[e, self.inter:]
            d[f"{prefix}e{e}.down"] = self.w_down[e]
        return d

    def forward(self, x, token_ids) -> moe.RoutedRows:
        """x [T, hidden], token_ids int64 [T]."""
        return moe.expert_rows(x, self.w_gate_up, self.w_down, moe.Assigned(self.table.data, token_ids), 1.0 / self.top, self.act)
