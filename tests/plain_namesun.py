"""A plain, slow implementation of the Namesun decoder: whole sequences, float64, one function per mechanism, nothing
shared with the package. ``cfg`` is the parsed config.json, ``W`` maps tensor names to float64 tensors.

    layer:   x <- x + m * ls1 * n1(mixer(x));   x <- x + m * ls2 * n2(ff(x));   n(y) = y / sqrt(mean(y^2) + eps) * w
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64
ALPHA = 1.702            # the sigmoid's slope in an expert's activation


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def same_chunk(T: int, size: int) -> torch.Tensor:
    """[T, T]: whether query i (row) sees key j (column)."""
    i = torch.arange(T)
    return (i[None, :] <= i[:, None]) & (i[:, None] // size == i[None, :] // size)


def sink_softmax(s: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)) over the keys a row sees."""
    s = s.masked_fill(~seen, -math.inf)
    top = s.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def mix_values(v: torch.Tensor, first: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    return (1.0 - lam) * v + lam * first


def attention(x: torch.Tensor, W: dict, p: str, m: dict, eps: float, first: torch.Tensor | None = None) -> torch.Tensor:
    """``first``: the values of the first layer that mixes them, for a layer that mixes after it."""
    T = x.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((x @ W[p + "q"].T).reshape(T, H, D), eps)
    k = rms((x @ W[p + "k"].T).reshape(T, G, D), eps)
    v = x @ W[p + "v"].T
    if first is not None:
        v = mix_values(v, first, W[p + "vmix"].reshape(()))
    v = v.reshape(T, G, V)
    seen = same_chunk(T, m["mask"]["size"])
    heads = []
    for h in range(H):
        g = h // (H // G)
        heads.append(sink_softmax(q[:, h] @ k[:, g].T * m["scale"], seen) @ v[:, g])
    return torch.cat(heads, -1) @ W[p + "o"].T


def rotate(x: torch.Tensor, rot: dict | None) -> torch.Tensor:
    """``x`` [T, heads, dim], row t at position t."""
    if rot is None or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    i = torch.arange(half, dtype=F64)
    a = torch.arange(x.shape[0], dtype=F64)[:, None] * float(rot["base"]) ** (-2.0 * i / rot["dims"])
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, w = x[..., :half], x[..., half:2 * half]
    return torch.cat((u * c - w * s, w * c + u * s, x[..., 2 * half:]), -1)


def retention_scan(q, k, v, decay):
    """``q``, ``k`` [T, H, D], ``v`` [T, H, V], ``decay`` [H] -> [T, H, V]."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    S = torch.zeros(H, D, v.shape[-1], dtype=F64)
    g = torch.as_tensor(decay, dtype=F64)[:, None, None]
    for t in range(T):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def retention(x: torch.Tensor, W: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T = x.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = rotate((x @ W[p + "q"].T).reshape(T, H, D), m.get("rot"))
    k = rotate((x @ W[p + "k"].T).reshape(T, H, D), m.get("rot")) * D ** -0.5
    o = retention_scan(q, k, (x @ W[p + "v"].T).reshape(T, H, V), m["decay"])
    return (rms(o, eps).reshape(T, H * V) * silu(x @ W[p + "g"].T)) @ W[p + "o"].T


def dense(x: torch.Tensor, W: dict, p: str) -> torch.Tensor:
    return (silu(x @ W[p + "gate"].T) * (x @ W[p + "up"].T)) @ W[p + "down"].T


def expert(x: torch.Tensor, W: dict, p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(x @ W[p + "gate"].T, max=limit)
    u = torch.clamp(x @ W[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(ALPHA * g) * (u + 1.0)) @ W[p + "down"].T


def route(z: torch.Tensor, correction: torch.Tensor, r: dict) -> tuple[list[int], torch.Tensor]:
    """One token's logits -> the chosen experts and their weights."""
    s = torch.softmax(z, -1)
    c = (s + correction).tolist()
    groups = r.get("groups") or {"count": 1, "keep": 1}
    n = r["experts"] // groups["count"]
    best = sorted(range(groups["count"]), key=lambda g: -max(c[g * n:(g + 1) * n]))[:groups["keep"]]
    allowed = [e for e in range(r["experts"]) if e // n in best]
    chosen = sorted(allowed, key=lambda e: -c[e])[:r["top"]]
    return chosen, s[chosen]


def experts(x: torch.Tensor, W: dict, p: str, f: dict) -> torch.Tensor:
    z = x @ W[p + "router"].T
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        chosen, w = route(z[t], W[p + "correction"], f["router"])
        for e, we in zip(chosen, w):
            out[t] += we * expert(x[t], W, f"{p}e{e}.", f["expert"]["limit"])
    if f.get("shared"):
        out = out + expert(x, W, p + "shared.", f["shared"]["limit"])
    return out


def feed_forward(x: torch.Tensor, W: dict, p: str, f: dict) -> torch.Tensor:
    return dense(x, W, p) if f["kind"] == "dense" else experts(x, W, p, f)


def forward(cfg: dict, W: dict, tokens) -> tuple[torch.Tensor, torch.Tensor]:
    """Logits [T, vocab] and the stream after every layer [layers, T, width]."""
    W = {k: v.to(F64) for k, v in W.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    streams, first = [], None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "retention":
            y = retention(x, W, p + "mix.", m, eps)
        else:
            y = attention(x, W, p + "mix.", m, eps, first if m.get("v_mix") else None)
            if m.get("v_mix") and first is None:
                first = x @ W[p + "mix.v"].T
        x = x + mult * (rms(y, eps) * W[p + "norm1"] * W[p + "ls1"])
        if layer.get("mlp") is not None:
            y = feed_forward(x, W, p + "mlp.", layer["mlp"])
            x = x + mult * (rms(y, eps) * W[p + "norm2"] * W[p + "ls2"])
        streams.append(x)
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T, torch.stack(streams)
