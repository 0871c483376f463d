"""Two mixers side by side on the same input (kind ``mixer_pair``):

    out = (rmsnorm(left(h)) * w_left + rmsnorm(right(h)) * w_right) / 2        (over the model width, 32-bit)

Any two registered mixers. Each branch's state is its own: its names carry the branch's (``left.kv``, ``right.S``), and
each branch is handed a context in which its states have the names it gave them. Where both branches say that one
projection of ``h`` is all they read of it (``input_projections`` / ``forward_projected``), the two projections are one
product.
"""

from __future__ import annotations

import dataclasses

import torch

from tokenomos_b200 import ops
from tokenomos_b200.parts.contract import StepContext
from tokenomos_b200.parts.delta import padded_rows
from tokenomos_b200.parts.linear import Linear
from tokenomos_b200.parts.registry import Runtime, builder_of, register

BRANCHES = ("left", "right")


class _BranchStates:
    """A step's states (or their groups) as one branch names them."""

    def __init__(self, states, branch: str):
        self.states, self.prefix = states, branch + "."

    def __getitem__(self, key):
        return self.states[(key[0], self.prefix + key[1])]

    def get(self, key, default=None):
        return self.states.get((key[0], self.prefix + key[1]), default)

    def __contains__(self, key):
        return (key[0], self.prefix + key[1]) in self.states


class MixerPair:
    def __init__(self, left, right, left_norm: torch.Tensor, right_norm: torch.Tensor, eps: float):
        self.branches = (left, right)
        self.norms = tuple(n.float().reshape(-1).contiguous() for n in (left_norm, right_norm))
        self.eps = float(eps)
        self.capture_safe = all(getattr(m, "capture_safe", False) for m in self.branches)
        if any(spec.storage == "shared" for m in self.branches for spec in m.state_specs().values()):
            raise ValueError("mixer pair: a branch that reads another layer's state is not built")
        self.in_proj = None
        firsts = [m.input_projections() if hasattr(m, "input_projections") else None for m in self.branches]
        if all(f is not None and f.bias is None for f in firsts) and firsts[0].weight.dtype == firsts[1].weight.dtype:
            a, b = firsts
            rows = padded_rows(a.weight)
            self.split = rows.shape[0]
            self.widths = (a.out_features, b.out_features)
            self.in_proj = Linear(torch.cat((rows, b.weight)), tuning=a.tuning)

    def state_specs(self) -> dict:
        return {f"{branch}.{name}": spec for branch, m in zip(BRANCHES, self.branches) for name, spec in m.state_specs().items()}

    def _contexts(self, ctx: StepContext) -> tuple[StepContext, StepContext]:
        """The step's context as each branch sees it (one pair per step, shared by the layers)."""
        have = ctx.scratch.get("mixer_pair")
        if have is None:
            have = tuple(dataclasses.replace(ctx, states=_BranchStates(ctx.states, b),
                                             state_groups=_BranchStates(ctx.state_groups, b)) for b in BRANCHES)
            ctx.scratch["mixer_pair"] = have
        return have

    def forward(self, x: torch.Tensor, ctx: StepContext, call: int) -> torch.Tensor:
        (left, right), (cl, cr) = self.branches, self._contexts(ctx)
        if self.in_proj is not None:
            proj = self.in_proj(x)
            a = left.forward_projected(proj[:, :self.widths[0]], cl, call)
            b = right.forward_projected(proj[:, self.split:self.split + self.widths[1]], cr, call)
        else:
            a, b = left.forward(x, cl, call), right.forward(x, cr, call)
        return ops.pair_norm_mean(a, b, self.norms[0], self.norms[1], self.eps, 0.5)


@register("mixer", "mixer_pair")
def build_mixer_pair(params: dict, tensors: dict, rt: Runtime) -> MixerPair:
    """``params``: ``left`` and ``right``, each ``{"kind", "params"}`` of a registered mixer, and ``eps``; tensors
    ``left.<role>`` and ``right.<role>`` are the branches', ``left_norm`` and ``right_norm`` the pair's."""
    parts = []
    for branch in BRANCHES:
        own = {k[len(branch) + 1:]: v for k, v in tensors.items() if k.startswith(branch + ".")}
        parts.append(builder_of("mixer", params[branch]["kind"])(params[branch]["params"], own, rt))
    return MixerPair(*parts, tensors["left_norm"], tensors["right_norm"], params["eps"])
