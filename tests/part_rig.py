"""A model folder written for a test, loaded as the framework loads it, with its cache on NaN-poisoned pools: ``Rig.run`` lays
steps out as the step function does and hands each context to one part, so that a part is tested alone over pages, state
rows and unequal portions."""

from __future__ import annotations

import json
from pathlib import Path

import torch


def write_folder(folder: Path, config: dict, tensors: dict) -> None:
    from safetensors.torch import save_file

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))


def cuts_of(n: int, sizes) -> list[tuple[int, int]]:
    out, a, k = [], 0, 0
    while a < n:
        b = min(n, a + sizes[k % len(sizes)])
        out.append((a, b))
        a, k = b, k + 1
    return out


PLANS = {
    "whole": lambda n: [(0, n)],
    "decoded": lambda n: [(0, max(1, n - 20))] + [(i, i + 1) for i in range(max(1, n - 20), n)],
    "portions": lambda n: cuts_of(n, (5, 2, 17, 3, 2, 29, 1, 1, 4)),
    "tokens": lambda n: [(i, i + 1) for i in range(n)],
}


def rows_for(lengths: dict[str, int], width: int, seed: int, scale: float = 1.0) -> dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    return {rid: (scale * torch.randn(n, width, generator=g)).to(torch.bfloat16).double() for rid, n in lengths.items()}


def close(got, want, tol, what):
    for rid, ref in want.items():
        assert torch.isfinite(got[rid]).all(), (what, rid)
        err = (got[rid] - ref).abs().amax(dim=-1)
        bad = (err > tol * ref.abs().max()).nonzero()
        assert bad.numel() == 0, (f"{what}: request {rid}: first wrong row {int(bad[0])} of {len(err)}: "
                                  f"{err[int(bad[0])].item():.3e} against {tol * ref.abs().max().item():.3e}")


class Rig:
    """``run`` feeds requests in unequal portions side by side; a freed slot and freed pages are used again."""

    def __init__(self, config: dict, tensors: dict, dtype: str, folder: Path, page=4, pages=120, slots=2):
        from tokenomos_b200 import models
        from tokenomos_b200.cache.manager import CacheManager
        from tokenomos_b200.engine.step import StepFunction

        write_folder(folder, config, tensors)
        self.config, self.w = config, {k: v.double() for k, v in tensors.items()}
        conf = models.configure(folder, work=dtype)
        self.dtype = conf.work
        self.model = models.load(folder, "cuda", conf)
        self.cache = CacheManager(self.model.state_specs(), page, pages, slots, conf.work, "cuda",
                                  max_len=(pages - 1) * page, poison=True)
        self.steps = StepFunction(self.model, self.cache)
        # hold and return a few pages so that the requests' pages are neither the first nor in order
        self.cache.admit("junk")
        self.cache.extend("junk", 3 * page)
        self.cache.admit("junk2")
        self.cache.extend("junk2", page)
        self.cache.release("junk")
        self.cache.release("junk2")

    def run(self, inputs: dict[str, torch.Tensor], plans: dict[str, list], fn, live=2) -> dict[str, torch.Tensor]:
        """``inputs``: request -> rows [n, width]; ``plans``: request -> list of (a, b) portions. ``fn(x, ctx)`` is called
        with the step's rows in the work dtype; its output rows are collected."""
        from tokenomos_b200.engine.step import StepEntry

        plans = {rid: list(p) for rid, p in plans.items()}
        waiting = list(inputs)
        active, got = [], {rid: [] for rid in inputs}
        while waiting or active:
            while waiting and len(active) < live:
                rid = waiting.pop(0)
                self.cache.admit(rid)
                active.append(rid)
            spans = [(rid, plans[rid].pop(0)) for rid in active]
            entries = [StepEntry(rid, [0] * (b - a), []) for rid, (a, b) in spans]
            ctx, _, _ = self.steps.layout(entries)
            x = torch.cat([inputs[rid][a:b] for rid, (a, b) in spans]).to(self.dtype).cuda().contiguous()
            out = fn(x, ctx)
            o = 0
            for rid, (a, b) in spans:
                self.cache.commit(rid, b - a)
                got[rid].append(out[o:o + b - a].double().cpu())
                o += b - a
            for rid in list(active):
                if not plans[rid]:
                    self.cache.release(rid)
                    active.remove(rid)
            self.cache.check()
        return {rid: torch.cat(parts) for rid, parts in got.items()}
