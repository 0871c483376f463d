"""A plain, slow implementation of the Tifisun decoder: whole sequences, float64, one function per
mechanism, nothing shared with the package. ``cfg`` is the parsed config.json, ``W`` maps tensor names
to float64 tensors.

    layer:   x <- x + m * n1b(mixer(n1(x)));   x <- x + m * n2b(ff(n2(x)))
    n(x):    x / sqrt(mean(x^2) + eps) * (1 + w)
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """``u`` [T, C], ``taps`` [C, K]: the last column multiplies the current token."""
    T, K = u.shape[0], taps.shape[1]
    padded = torch.cat((torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u))
    return sum(padded[j:j + T] * taps[:, j] for j in range(K))


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, g, beta):
    """``q``, ``k``, ``g`` [T, H, D], ``v`` [T, H, V], ``beta`` [T, H] -> [T, H, V]: the state decays along its key
    channels, the key's stored value moves towards v by beta, the query reads the updated state."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        S = torch.zeros(D, v.shape[-1], dtype=F64)
        for t in range(T):
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + torch.outer(k[t, h], u)
            out[t, h] = S.T @ q[t, h]
    return out


def delta(h: torch.Tensor, W: dict, p: str, m: dict, eps: float, channel: bool) -> torch.Tensor:
    T = h.shape[0]
    H, K, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    u = {n: silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v")}
    spread = [i // (H // K) for i in range(H)]                       # value head -> q/k head
    q = unit(u["q"].reshape(T, K, D))[:, spread] * D ** -0.5
    k = unit(u["k"].reshape(T, K, D))[:, spread]
    v = u["v"].reshape(T, H, V)
    beta = torch.sigmoid(h @ W[p + "b"].T)
    A = torch.exp(W[p + "A_log"])
    if channel:
        dt = softplus((h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]).reshape(T, H, D)
        g = torch.exp(-A[None, :, None] * dt)
        gate = torch.sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T)
    else:
        dt = softplus(h @ W[p + "a"].T + W[p + "dt_bias"])
        g = torch.exp(-A * dt)[:, :, None].expand(T, H, D)
        gate = silu(h @ W[p + "g"].T)
    o = delta_scan(q, k, v, g, beta)
    o = rms(o, eps) * W[p + "norm"]
    return (o.reshape(T, H * V) * gate) @ W[p + "o"].T


def bucket(n: int, rows: int, far: int) -> int:
    half = rows / 2
    if n < half:
        return n
    return min(rows - 1, int(half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


def windowed_attention(h: torch.Tensor, W: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ W[p + "q"].T, eps) * W[p + "q.norm"]).reshape(T, H, D)
    k = (rms(h @ W[p + "k"].T, eps) * W[p + "k.norm"]).reshape(T, G, D)
    v = (h @ W[p + "v"].T).reshape(T, G, V)
    rel = W[p + "rel"]
    by_distance = torch.tensor([bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)])
    i = torch.arange(T)
    dist = i[:, None] - i[None, :]
    seen = (dist >= 0) & (dist < m["mask"]["size"])
    heads = []
    for hd in range(H):
        g = hd // (H // G)
        s = q[:, hd] @ k[:, g].T * m["scale"]
        s = m["softcap"] * torch.tanh(s / m["softcap"])
        s = s + rel[by_distance[dist.clamp(min=0)], hd]
        heads.append(torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1) @ v[:, g])
    return torch.cat(heads, -1) @ W[p + "o"].T


def lightning(h: torch.Tensor, W: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W[p + "q"].T).reshape(T, H, D)
    k = silu(h @ W[p + "k"].T).reshape(T, H, D)
    v = silu(h @ W[p + "v"].T).reshape(T, H, V)
    out = torch.zeros(T, H, V, dtype=F64)
    for hd in range(H):
        S = torch.zeros(D, V, dtype=F64)
        for t in range(T):
            S = m["decay"][hd] * S + torch.outer(k[t, hd], v[t, hd])
            out[t, hd] = S.T @ q[t, hd]
    o = rms(out.reshape(T, H * V), eps) * W[p + "norm"]
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel(h: torch.Tensor, W: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    left = rms(windowed_attention(h, W, p + "left.", m["left"], eps), eps) * W[p + "left.out"]
    right = rms(lightning(h, W, p + "right.", m["right"], eps), eps) * W[p + "right.out"]
    return 0.5 * (left + right)


def feed_forward(h: torch.Tensor, W: dict, p: str) -> torch.Tensor:
    a = gelu_tanh(h @ W[p + "gate"].T + W[p + "gate.b"]) * (h @ W[p + "up"].T + W[p + "up.b"])
    return a @ W[p + "down"].T + W[p + "down.b"]


def mixer(kind: str, h, W, p, m, eps):
    if kind == "parallel":
        return parallel(h, W, p, m, eps)
    return delta(h, W, p, m, eps, channel=kind == "channel_delta")


def forward(cfg: dict, W: dict, tokens) -> tuple[torch.Tensor, torch.Tensor]:
    """Logits [T, vocab] and the stream after every layer [layers, T, width]."""
    W = {k: v.to(F64) for k, v in W.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        j = i
        while cfg["layers"][j].get("weights_of") is not None:
            j = cfg["layers"][j]["weights_of"]
        p = f"l{j}."
        y = mixer(layer["type"], rms(x, eps) * (1 + W[p + "norm1"]), W, p + "mix.", layer["mixer"], eps)
        x = x + mult * (rms(y, eps) * (1 + W[p + "norm1b"]))
        if layer.get("mlp") is not None:
            y = feed_forward(rms(x, eps) * (1 + W[p + "norm2"]), W, p + "mlp.")
            x = x + mult * (rms(y, eps) * (1 + W[p + "norm2b"]))
        streams.append(x)
    return (rms(x, eps) * (1 + W["final.norm"])) @ W["head"].T, torch.stack(streams)
