"""
Plain, slow implementation of the Fuvipel decoder in float64, one function per mechanism, written
from the design's equations.  It shares no code with the engine: tensors come in as a dict by their
checkpoint names, the configuration as the dict config.json holds.  Recurrences walk token by token.

    x_0 = embed[token]
    layer:  x <- x + N1(mixer(x));  x <- x + N2(ff(x))         N: RMS norm with weight, on the branch only
    mixer "delta":    gated delta rule, one decay a head, silu output gate
    mixer "parallel": (L(attention(x)) + R(time_mixing(x))) / 2, L and R RMS norms with weights of their own
    ff:               down(relu(up x)^2)
    logits = embed . N_final(x)
"""

from __future__ import annotations

import torch

F64 = torch.float64


def rms_div(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim]: channels 2i and 2i + 1 of the first rot dims turn by position * base^(-2i/dims)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    y = x.clone()
    for i in range(dims // 2):
        angle = positions.to(F64) * base ** (-2.0 * i / dims)
        c, s = angle.cos()[:, None], angle.sin()[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def softmax_with_sink(s: torch.Tensor, visible: torch.Tensor) -> torch.Tensor:
    """Weights over the visible keys with exp(0) more in the denominator; rows may sum to less than one."""
    s = s.masked_fill(~visible, -float("inf"))
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def sink_attention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """The left half of the parallel mixer over a whole sequence.  h [T, width]; w: tensors under '<layer>.mix.left.'."""
    T = h.shape[0]
    H, G, D = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    pos = torch.arange(T)
    raw_k = (h @ w["k"].T).view(T, G, D)
    q = rms_div(rotate_neighbours((h @ w["q"].T).view(T, H, D), pos, m["rot"]), eps)
    k = rms_div(rotate_neighbours(raw_k, pos, m["rot"]), eps)
    out = torch.zeros(T, H, D, dtype=F64)
    visible = torch.ones(T, T, dtype=torch.bool).tril()
    for head in range(H):
        g = head // (H // G)
        p = softmax_with_sink((q[:, head] @ k[:, g].T) * float(m["scale"]), visible)
        out[:, head] = p @ raw_k[:, g]
    return (out.reshape(T, H * D) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def time_mixing(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """The right half of the parallel mixer.  w: tensors under '<layer>.mix.right.'."""
    T = h.shape[0]
    H, D = int(m["heads"]), int(m["dim"])
    before = torch.cat([torch.zeros(1, h.shape[1], dtype=F64), h[:-1]])
    mix = {s: h + (before - h) * w["mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[s].T).view(T, H, D) for s in "rkv")
    gate = silu(mix["g"] @ w["g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w["w1"].T) @ w["w2"].T + w["w0"])).view(T, H, D)
    out = torch.zeros(T, H, D, dtype=F64)
    for head in range(H):
        S = torch.zeros(D, D, dtype=F64)
        for t in range(T):
            write = torch.outer(k[t, head], v[t, head])
            out[t, head] = (S + w["u"][head][:, None] * write).T @ r[t, head]
            S = decay[t, head][:, None] * S + write
    return (rms_div(out, eps).reshape(T, H * D) * w["norm"] * gate) @ w["o"].T


def parallel_mixer(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    left = rms_div(sink_attention(h, _under(w, "left."), m["left"], eps), eps) * w["left.out"]
    right = rms_div(time_mixing(h, _under(w, "right."), m["right"], eps), eps) * w["right.out"]
    return 0.5 * (left + right)


def short_conv_silu(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, K]: y_t = sum_j taps[:, j] x_(t - (K - 1 - j)), zeros before the start; then silu."""
    T, C = x.shape
    K = taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, C, dtype=x.dtype), x], dim=0)
    y = torch.zeros_like(x)
    for j in range(K):
        y = y + padded[j:j + T] * taps[:, j]
    return silu(y)


def gated_delta_rule(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """w: tensors under '<layer>.mix.'."""
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = short_conv_silu(h @ w["q"].T, w["q.conv"]).view(T, G, D)
    k = short_conv_silu(h @ w["k"].T, w["k.conv"]).view(T, G, D)
    v = short_conv_silu(h @ w["v"].T, w["v.conv"]).view(T, H, V)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = torch.sigmoid(h @ w["b"].T)
    decay = torch.exp(-torch.exp(w["A_log"]) * torch.nn.functional.softplus(h @ w["a"].T + w["dt_bias"], threshold=100.0))   # [T, H]
    out = torch.zeros(T, H, V, dtype=F64)
    for head in range(H):
        g = head // (H // G)
        S = torch.zeros(D, V, dtype=F64)
        for t in range(T):
            S = decay[t, head] * S
            u = beta[t, head] * (v[t, head] - S.T @ k[t, g])
            S = S + torch.outer(k[t, g], u)
            out[t, head] = S.T @ q[t, g]
    out = rms_div(out, eps) * w["norm"] * silu(h @ w["g"].T).view(T, H, V)
    return out.reshape(T, H * V) @ w["o"].T


def dense(h: torch.Tensor, w: dict) -> torch.Tensor:
    return torch.relu(h @ w["up"].T) ** 2 @ w["down"].T


def _under(w: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config: dict, tensors: dict, tokens: list[int], return_layers: bool = False):
    """float64 logits [T, vocab] of one sequence from its start (and the stream after every layer, if asked)."""
    w = {k: v.to(F64) for k, v in tensors.items()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    after = []
    for i, layer in enumerate(config["layers"]):
        lw = _under(w, f"l{i}.")
        mixer = {"delta": gated_delta_rule, "parallel": parallel_mixer}[layer["type"]]
        x = x + rms_div(mixer(x, _under(lw, "mix."), layer["mixer"], eps), eps) * lw["norm1"]
        if layer.get("mlp") is not None:
            x = x + rms_div(dense(x, _under(lw, "mlp.")), eps) * lw["norm2"]
        after.append(x)
    logits = rms_div(x, eps) * w["final.norm"] @ w["embed"].T
    return (logits, torch.stack(after)) if return_layers else logits
