"""
Plain, slow implementation of the Gimotar decoder in float64, one function per mechanism, written from
the design's equations.  It shares no code with the engine: tensors come in as a dict by their
checkpoint names, the configuration as the dict config.json holds.  Every attention builds the whole
score matrix of a sequence, the recurrence walks token by token, experts run token by token.

    x_0[t] = scale * embed[token_t] + bigram[pair row of (token_(t-1), token_t)]
    layer:  h = N1(x);  x <- x + m (mixer(h) + ff(h))         N(x) = x / sqrt(mean(x^2) + eps) * (1 + w)
    mixer "rglru":            Griffin's recurrent block, a real-gated linear recurrent unit
    mixer "latent_attention": keys and values worked out of one normed latent a token, one rotated key part
                              shared by the heads, a sink a head, a sigmoid gate on the heads
    mixer "attention":        heads of q and k normed, rotation by halves, chunks, values mixed with those
                              of the first layer that mixes
    ff "moe":                 softmax over the chosen router logits, a shared expert beside
    logits = embed . N_final(x)
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64
RG_C = 8.0


def rms_div(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


# ---------------------------------------------------------------------- embedding
def pair_rows(tokens: list[int], bigram: dict) -> list[int]:
    """The row of the pair table for every token: of (token before, token), or the last row for the first token."""
    n, a, b = int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"])
    return [n if t == 0 else (tokens[t - 1] * a + tokens[t] * b) % n for t in range(len(tokens))]


def embedded(w: dict, config: dict, tokens: list[int]) -> torch.Tensor:
    e = config["embedding"]
    rows = torch.tensor(pair_rows(tokens, e["bigram"]), dtype=torch.long)
    return w["embed"][torch.tensor(tokens, dtype=torch.long)] * float(e["scale"]) + w["bigram"][rows]


# ---------------------------------------------------------------------- rotation
def frequencies(rot: dict) -> tuple[list[float], float]:
    """(frequency of every pair, what cos and sin are multiplied by)."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return f, 1.0
    where = lambda turns: dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))  # noqa: E731
    lo, hi = max(math.floor(where(float(sc["fast"]))), 0), min(math.ceil(where(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / float(sc["factor"]) * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(float(sc["factor"])) + 1.0


def rotate(x: torch.Tensor, rot: dict, neighbours: bool) -> torch.Tensor:
    """x [T, heads, dim], row t at position t: the first rot dims turn, channel i with i + dims/2 or (neighbours) 2i with 2i + 1."""
    f, gain = frequencies(rot)
    half = len(f)
    y = x.clone()
    for i, fi in enumerate(f):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + half)
        angle = torch.arange(x.shape[0], dtype=F64) * fi
        c, s = gain * angle.cos()[:, None], gain * angle.sin()[:, None]
        y[..., a] = x[..., a] * c - x[..., b] * s
        y[..., b] = x[..., b] * c + x[..., a] * s
    return y


# ---------------------------------------------------------------------- mixers
def causal_conv(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, K]: out_t = bias + sum_j taps[:, j] x_(t - (K - 1 - j)), zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x])
    return bias + sum(padded[j:j + T] * taps[:, j] for j in range(K))


def block_product(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, C] in equal parts, part i times w[i] [out, in], plus b[i]."""
    n, size = w.shape[0], w.shape[1]
    return torch.cat([u[:, i * size:(i + 1) * size] @ w[i].T + b[i] for i in range(n)], dim=-1)


def recurrent_unit(u: torch.Tensor, w: dict) -> torch.Tensor:
    """u [T, C] -> the states after every token."""
    r = torch.sigmoid(block_product(u, w["ra"], w["ra.b"]))
    i = torch.sigmoid(block_product(u, w["ri"], w["ri.b"]))
    log_a = -RG_C * r * softplus(w["lam"])
    S = torch.zeros(u.shape[1], dtype=F64)
    out = []
    for t in range(u.shape[0]):
        a = torch.exp(log_a[t])
        S = a * S + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def rglru(h: torch.Tensor, w: dict, m: dict) -> torch.Tensor:
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    return (recurrent_unit(u, w) * y) @ w["o"].T


def softmax_with_sink(s: torch.Tensor, visible: torch.Tensor, sink: torch.Tensor | None) -> torch.Tensor:
    """Weights over the visible keys, exp(sink) more in the denominator where there is a sink."""
    s = s.masked_fill(~visible, -float("inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink)
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    return e / (total if sink is None else total + torch.exp(sink - top))


def latent_attention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, R, V, rank = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    q = (h @ w["q"].T).view(T, H, D + R)
    down = h @ w["dkv"].T
    c = rms_div(down[:, :rank], eps) * w["dkv.norm"]
    k_rot = rotate(down[:, rank:].view(T, 1, R), m["rot"], neighbours=True)[:, 0]
    q_rot = rotate(q[..., D:], m["rot"], neighbours=True)
    k, v = (c @ w["uk"].T).view(T, H, D), (c @ w["uv"].T).view(T, H, V)
    visible = torch.ones(T, T, dtype=torch.bool).tril()
    out = torch.zeros(T, H, V, dtype=F64)
    for head in range(H):
        s = (q[:, head, :D] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * float(m["scale"])
        out[:, head] = softmax_with_sink(s, visible, w["sink"][head]) @ v[:, head]
    return (out.reshape(T, H * V) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def chunk_mask(T: int, size: int | None) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) if not size else (j <= i) & (i // size == j // size)


def attention(h: torch.Tensor, w: dict, m: dict, eps: float, v_first: torch.Tensor | None) -> tuple[torch.Tensor, torch.Tensor]:
    """`v_first` [T, kv heads * vdim]: the first mixing layer's values (None: there is none before this layer).  Also returns this layer's own."""
    T = h.shape[0]
    H, G, D, V = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    normed = lambda x, n: rms_div((h @ w[x].T).view(T, n, D), eps) * w[x + ".norm"]  # noqa: E731
    q, k = rotate(normed("q", H), m["rot"], neighbours=False), rotate(normed("k", G), m["rot"], neighbours=False)
    own = h @ w["v"].T
    v = own
    if m.get("v_mix") and v_first is not None:
        v = (1.0 - w["vmix"]) * own + w["vmix"] * v_first
    v = v.view(T, G, V)
    visible = chunk_mask(T, int(m["mask"]["size"]) if m.get("mask") else None)
    out = torch.zeros(T, H, V, dtype=F64)
    for head in range(H):
        g = head // (H // G)
        out[:, head] = softmax_with_sink((q[:, head] @ k[:, g].T) * float(m["scale"]), visible, None) @ v[:, g]
    return out.reshape(T, H * V) @ w["o"].T, own


# ---------------------------------------------------------------------- feed-forward
def expert(h: torch.Tensor, w: dict) -> torch.Tensor:
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def experts(h: torch.Tensor, w: dict, f: dict) -> torch.Tensor:
    z = h @ w["router"].T + w["router.b"]
    out = []
    for t in range(h.shape[0]):
        chosen = torch.argsort(z[t], descending=True)[:int(f["router"]["top"])]
        share = torch.softmax(z[t][chosen], dim=0)
        out.append(sum(p * expert(h[t], _under(w, f"e{int(e)}.")) for p, e in zip(share, chosen)))
    y = torch.stack(out)
    return y if not f.get("shared") else y + expert(h, _under(w, "shared."))


# ---------------------------------------------------------------------- the model
def _under(w: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config: dict, tensors: dict, tokens: list[int], return_layers: bool = False):
    """float64 logits [T, vocab] of one sequence from its start (and the stream after every layer, if asked)."""
    w = {k: v.to(F64) for k, v in tensors.items()}
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    norm = lambda x, name: rms_div(x, eps) * (1.0 + w[name])  # noqa: E731
    x = embedded(w, config, tokens)
    v_first, after = None, []
    for i, layer in enumerate(config["layers"]):
        h, m, mw = norm(x, f"l{i}.norm1"), layer["mixer"], _under(w, f"l{i}.mix.")
        if layer["type"] == "rglru":
            y = rglru(h, mw, m)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, mw, m, eps)
        else:
            y, own = attention(h, mw, m, eps, v_first)
            if m.get("v_mix") and v_first is None:
                v_first = own
        if layer.get("mlp") is not None:
            y = y + experts(h, _under(w, f"l{i}.mlp."), layer["mlp"])
        x = x + mult * y
        after.append(x)
    logits = norm(x, "final.norm") @ w["embed"].T
    return (logits, torch.stack(after)) if return_layers else logits
