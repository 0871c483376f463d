"""Linear memories with a fixed-size state per request: the gated delta rule, lightning attention and retention.

``GatedDelta`` (kind ``delta_rule``): per head a matrix S [dim, v_dim] from zero,

    q, k, v = silu(conv(W_q h)), silu(conv(W_k h)), silu(conv(W_v h))     a short causal convolution per channel
    k <- k / sqrt(sum k^2 + 1e-6),  q likewise, then times dim^(-1/2);  value head j reads q/k head j / (heads / kv_heads)
    beta = sigmoid(W_b h);   g = exp(-exp(A_log) softplus(z + dt_bias))
        decay "head":     z = W_a h, one per head
        decay "channel":  z = W_a2 (W_a1 h), one per head and key channel (a row of S each)
    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
    out = W_o (headnorm(o) * w * gate),   gate = silu(W_g h), or sigmoid(W_g2 (W_g1 h))      (w shared by the heads)

``LightningMemory`` (kind ``lightning``): ``q, k, v = silu(W h)``, ``S <- decay[head] S + k v^T``, ``o = S^T q``, the
concatenated heads RMS-normed together, times ``w * sigmoid(W_g h)``, through ``W_o``. Kind ``retention``: the same
recurrence without the silu on q, k and v, with a rotation of q and k by position, ``k`` times ``dim^(-1/2)``, every head's
``o`` RMS-normed on its own (no weight) and the gate ``silu(W_g h)``.

The states, everything that enters a recurrence after the projections and convolutions (beta and the decays from
products with a 32-bit result, unit lengths), and the norms are 32-bit whatever the storage type. Both parts read the
batch from device tensors only, so their steps can be recorded.
"""

from __future__ import annotations

import torch

from tokenomos_b200 import ops
from tokenomos_b200.parts.contract import SlotState, StepContext
from tokenomos_b200.parts.linear import Linear
from tokenomos_b200.parts.registry import Runtime, register
from tokenomos_b200.parts.rope import Rotary


def padded_rows(w: torch.Tensor, to: int = 8) -> torch.Tensor:
    """``w`` with zero rows up to a multiple of ``to`` (whole 16-byte chunks of a product's row)."""
    pad = -w.shape[0] % to
    return torch.cat((w, w.new_zeros(pad, w.shape[1]))) if pad else w


def padded_columns(w: torch.Tensor, to: int = 8) -> torch.Tensor:
    pad = -w.shape[1] % to
    return torch.cat((w, w.new_zeros(w.shape[0], pad)), dim=1).contiguous() if pad else w


class GatedDelta:
    capture_safe = True

    def __init__(self, in_proj: Linear, gate_proj: Linear, out_proj: Linear, taps: torch.Tensor, a_log: torch.Tensor,
                 dt_bias: torch.Tensor, norm: torch.Tensor, heads: int, kv_heads: int, dim: int, v_dim: int, eps: float,
                 gate: str = "silu", decay: str = "head", decay_up: Linear | None = None, gate_up: Linear | None = None,
                 tile: int = 16):
        """``in_proj``: the rows of q, k, v, then the output gate's ([heads v_dim]), or, with ``gate_up`` / ``decay_up``,
        what those two read (padded to whole chunks): first the decay's, then the gate's. ``gate_proj``: beta's rows
        and, with ``decay`` "head", the decay's (32-bit result)."""
        self.in_proj, self.gate_proj, self.out_proj = in_proj, gate_proj, out_proj
        self.heads, self.kv_heads, self.dim, self.v_dim = int(heads), int(kv_heads), int(dim), int(v_dim)
        self.eps, self.gate, self.decay = float(eps), gate, decay
        self.decay_up, self.gate_up = decay_up, gate_up
        self.channels, self.K = taps.shape
        if self.heads % self.kv_heads:
            raise ValueError(f"delta rule: {heads} heads over {kv_heads} q/k heads")
        if self.dim > ops.LINMEM_MAX_DIM:
            raise ValueError(f"delta rule: a key size of {dim} is above the {ops.LINMEM_MAX_DIM} the scan keeps in registers")
        if self.channels != 2 * self.kv_heads * self.dim + self.heads * self.v_dim:
            raise ValueError("delta rule: the convolution does not cover q, k and v")
        if not 1 <= self.K <= ops.SEQ_CONV_MAX_TAPS:
            raise ValueError(f"delta rule: {self.K} taps; 1..{ops.SEQ_CONV_MAX_TAPS} are built")
        if gate not in ops.GATE_KINDS or decay not in ("head", "channel") or (decay == "channel") != (decay_up is not None):
            raise ValueError(f"delta rule: gate {gate!r} with decay {decay!r}")
        extra = self.heads * self.v_dim if gate_up is None else gate_up.in_features
        extra += decay_up.in_features if decay_up is not None else 0
        if in_proj.out_features != self.channels + extra or out_proj.in_features != self.heads * self.v_dim:
            raise ValueError("delta rule: the projections do not match the head sizes")
        self.taps = taps.float().contiguous()
        self.A = torch.exp(a_log.double().reshape(-1)).float().contiguous()
        self.dt_bias = dt_bias.float().reshape(-1).contiguous()
        if self.dt_bias.numel() != self.heads * (self.dim if decay == "channel" else 1):
            raise ValueError("delta rule: the decay's bias does not match the heads")
        self.norm = norm.float().reshape(-1).repeat(self.heads).contiguous()
        self.tile = max(int(tile), self.K - 1, 1)
        self.sm_count = in_proj.tuning.sm_count

    def state_specs(self) -> dict:
        specs = {"S": SlotState((self.heads, self.v_dim, self.dim), torch.float32)}
        if self.K > 1:
            specs["conv"] = SlotState((self.K - 1, self.channels), torch.float32)
        return specs

    def forward(self, x: torch.Tensor, ctx: StepContext, call: int) -> torch.Tensor:
        T, C, H = x.shape[0], self.channels, self.heads
        nk = self.kv_heads * self.dim
        proj = self.in_proj(x)
        z = self.gate_proj(x, out_dtype=torch.float32)
        u = ops.seq_conv(proj[:, :C], self.taps, None, ctx.states.get((call, "conv")), ctx.cu_seqlens, ctx.seq_ctx,
                         ctx.seq_slot, ctx.tiles(ops.seq_conv_tile(self.tile, T, C)), proj.dtype, act=True)
        if self.decay == "channel":
            n = C + self.decay_up.in_features
            decay = self.decay_up(proj[:, C:n], out_dtype=torch.float32)
        else:
            n, decay = C, z[:, H:]
        gate = proj[:, n:] if self.gate_up is None else self.gate_up(proj[:, n:])
        y = ops.linmem_scan(u, (0, nk, 2 * nk), "delta", self.decay, self.A, ctx.states[(call, "S")], ctx.cu_seqlens, ctx.seq_ctx,
                            ctx.seq_slot, ctx.n_seqs, H, self.kv_heads, self.dim, self.v_dim, self.dim ** -0.5, unit=True,
                            beta=z, gates=decay, bias=self.dt_bias, sm_count=self.sm_count)
        return self.out_proj(ops.norm_gate(y, gate, self.norm, self.eps, H, self.gate))


@register("mixer", "delta_rule")
def build_gated_delta(params: dict, tensors: dict, rt: Runtime) -> GatedDelta:
    """Tensors ``q``, ``k``, ``v``, ``q_conv``, ``k_conv``, ``v_conv``, ``b``, ``a_log``, ``dt_bias``, ``norm``, ``o``; decay
    "head": ``a``, "channel": ``a1``, ``a2``; the gate: ``g``, or ``g1`` and ``g2``."""
    decay = params.get("decay", "head")
    mats = [tensors["q"], tensors["k"], tensors["v"]]
    wide = [tensors["b"]]
    decay_up = gate_up = None
    if decay == "channel":
        mats.append(padded_rows(tensors["a1"]))
        decay_up = Linear(padded_columns(tensors["a2"]), tuning=rt.tuning)
    else:
        wide.append(tensors["a"])
    if "g1" in tensors:
        mats.append(padded_rows(tensors["g1"]))
        gate_up = Linear(padded_columns(tensors["g2"]), tuning=rt.tuning)
    else:
        mats.append(tensors["g"])
    taps = torch.cat([tensors[n + "_conv"].float() for n in ("q", "k", "v")])
    return GatedDelta(Linear.fused(mats, tuning=rt.tuning), Linear(padded_rows(torch.cat(wide)), tuning=rt.tuning),
                      Linear(tensors["o"], tuning=rt.tuning), taps, tensors["a_log"], tensors["dt_bias"], tensors["norm"],
                      params["heads"], params["kv_heads"], params["dim"], params["v_dim"], params["eps"],
                      params.get("gate", "silu"), decay, decay_up, gate_up, tile=rt.tuning.conv_tile)


class LightningMemory:
    capture_safe = True

    def __init__(self, in_proj: Linear, out_proj: Linear, decay: list[float], norm: torch.Tensor | None, heads: int, dim: int,
                 v_dim: int, eps: float, act: bool = True, q_scale: float = 1.0, freq: torch.Tensor | None = None,
                 norm_groups: int = 1, gate: str = "sigmoid"):
        """``in_proj``: the rows of q, k (heads x dim each), v and the output gate (heads x v_dim each). ``act``: q, k and v pass
        silu; ``q_scale``: a factor on q (one on k is the same number in every output); ``freq``: the frequencies of a
        rotate-half rotation of q's and k's first columns; ``norm_groups``: equal parts of the output row that are normed on
        their own; ``norm`` None: no weight; ``gate``: silu or sigmoid."""
        self.in_proj, self.out_proj = in_proj, out_proj
        self.heads, self.dim, self.v_dim, self.eps = int(heads), int(dim), int(v_dim), float(eps)
        if self.dim > ops.LINMEM_MAX_DIM:
            raise ValueError(f"lightning attention: a key size of {dim} is above the {ops.LINMEM_MAX_DIM} the scan keeps in "
                             "registers")
        if len(decay) != self.heads:
            raise ValueError(f"lightning attention: {len(decay)} decays for {heads} heads")
        if (in_proj.out_features != 2 * self.heads * (self.dim + self.v_dim)
                or out_proj.in_features != self.heads * self.v_dim):
            raise ValueError("lightning attention: the projections do not match the head sizes")
        if gate not in ops.GATE_KINDS or (freq is not None and 2 * freq.numel() > self.dim):
            raise ValueError(f"linear memory: gate {gate!r}, rotation of {2 * freq.numel() if freq is not None else 0} of {self.dim} "
                             "columns")
        self.norm = norm.float().reshape(-1).contiguous() if norm is not None else None
        self.act, self.q_scale, self.freq = bool(act), float(q_scale), freq
        self.norm_groups, self.gate = int(norm_groups), gate
        self.decay = torch.tensor([float(d) for d in decay], dtype=torch.float32, device=in_proj.weight.device)
        self.sm_count = in_proj.tuning.sm_count

    def state_specs(self) -> dict:
        return {"S": SlotState((self.heads, self.v_dim, self.dim), torch.float32)}

    def input_projections(self) -> Linear:
        return self.in_proj

    def forward(self, x: torch.Tensor, ctx: StepContext, call: int) -> torch.Tensor:
        return self.forward_projected(self.in_proj(x), ctx, call)

    def forward_projected(self, proj: torch.Tensor, ctx: StepContext, call: int) -> torch.Tensor:
        H, D, V = self.heads, self.dim, self.v_dim
        y = ops.linmem_scan(proj, (0, H * D, 2 * H * D), "add", "fixed", self.decay, ctx.states[(call, "S")], ctx.cu_seqlens,
                            ctx.seq_ctx, ctx.seq_slot, ctx.n_seqs, H, H, D, V, q_scale=self.q_scale, act=self.act,
                            sm_count=self.sm_count, freq=self.freq, positions=ctx.positions)
        gate = proj[:, 2 * H * D + H * V:2 * H * (D + V)]
        return self.out_proj(ops.norm_gate(y, gate, self.norm, self.eps, self.norm_groups, self.gate))


@register("mixer", "lightning")
def build_lightning_memory(params: dict, tensors: dict, rt: Runtime) -> LightningMemory:
    mats = [tensors[n] for n in ("q", "k", "v", "gate")]
    return LightningMemory(Linear.fused(mats, tuning=rt.tuning), Linear(tensors["o"], tuning=rt.tuning), params["decay"],
                           tensors["norm"], params["heads"], params["dim"], params["v_dim"], params["eps"])


@register("mixer", "retention")
def build_retention(params: dict, tensors: dict, rt: Runtime) -> LightningMemory:
    """Tensors ``q``, ``k``, ``v``, ``gate``, ``o``; params ``heads``, ``dim``, ``v_dim``, ``decay`` (one per head), ``eps`` and ``rot``
    (``dims``, ``base``; None: no rotation)."""
    mats = [tensors[n] for n in ("q", "k", "v", "gate")]
    rot, freq = params.get("rot"), None
    if rot is not None and rot["dims"]:
        freqs, _ = Rotary.table(rot["dims"], float(rot["base"]), None)
        freq = torch.tensor(freqs, dtype=torch.float64).to(torch.float32).to(rt.device).contiguous()
    return LightningMemory(Linear.fused(mats, tuning=rt.tuning), Linear(tensors["o"], tuning=rt.tuning), params["decay"], None,
                           params["heads"], params["dim"], params["v_dim"], params["eps"], act=False,
                           q_scale=params["dim"] ** -0.5, freq=freq, norm_groups=params["heads"], gate="silu")
