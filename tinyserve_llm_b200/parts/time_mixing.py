"""
RWKV-style time mixing: a linear recurrence with decays per channel whose read-out sees the current
token under a bonus, and whose inputs are blends of the token's row and the one before it.

    m_s = h + (h' - h) mu_s                 h' the previous token's h (zeros for the first), s in r, k, v, g, w
    r, k, v = W_r m_r, W_k m_k, W_v m_v     a = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))
    o_t = (S_(t-1) + diag(u) k_t v_t^T)^T r_t,   S_t = diag(a_t) S_(t-1) + k_t v_t^T     per head, S [dim, dim]
    y = W_o ( concat(o / rms(o)) * w * silu(W_g m_g) )

One kernel makes the five blends, one grouped product the four projections of equal shape, a small
one with tanh in its epilogue and a second one (float32 out) the decays' logits; then the scan of
`linear_recurrence.cu` in its bonus form (prompt portions: `recurrence_tiles.cu`).  The state (float32: the matrices, then the last h) lives in
the request's slot of the cache manager, so prompts in portions, decoding and mixed batches are one
code path.  Since every projection reads a blend of its own, none of them can join a projection
of h: inside a `ParallelMixer` this branch exposes no input rows and reads h itself.
"""

from __future__ import annotations

import dataclasses

import torch

from tinyserve_llm_b200.config.spec import TimeMixingSpec
from tinyserve_llm_b200.parts.base import Mixer, Runtime, TensorDecl, register_part
from tinyserve_llm_b200.parts.linear import Linear

MAX_HEAD_DIM = 256      # csrc/linear_recurrence.cu


@register_part("mixer", "time_mixing")
class TimeMixing(Mixer):
    graph_safe = True

    @classmethod
    def validate(cls, spec: TimeMixingSpec) -> None:
        if spec.num_heads <= 0 or not 0 < spec.head_dim <= MAX_HEAD_DIM:
            raise ValueError(f"time mixing with {spec.num_heads} heads of {spec.head_dim}: the recurrence kernel takes heads of up to "
                             f"{MAX_HEAD_DIM}")

    @classmethod
    def declare(cls, spec: TimeMixingSpec) -> dict[str, TensorDecl]:
        cls.validate(spec)
        inner, hidden = spec.num_heads * spec.head_dim, spec.hidden_size
        rank = spec.decay_rank if spec.decay_rank > 0 else -1            # -1: the checkpoint's own size
        out = {f"mu.{s}": TensorDecl((hidden,)) for s in "rkvgw"}
        out.update({s: TensorDecl((inner, hidden)) for s in "rkvg"})
        out.update({"w1": TensorDecl((rank, hidden)), "w2": TensorDecl((inner, rank)), "w0": TensorDecl((inner,)),
                    "u": TensorDecl((spec.num_heads, spec.head_dim)), "norm": TensorDecl((inner,), init="unit"),
                    "o": TensorDecl((hidden, inner))})
        return out

    def __init__(self, spec: TimeMixingSpec, tensors: dict[str, torch.Tensor], rt: Runtime, fused: bool = False) -> None:
        super().__init__(spec, tensors, rt)
        self.validate(spec)
        if tensors["w1"].shape[0] != tensors["w2"].shape[1]:
            raise ValueError(f"the inner sizes of w1 and w2 differ: {tuple(tensors['w1'].shape)} and {tuple(tensors['w2'].shape)}")
        f32 = dict(device=rt.device, dtype=torch.float32)
        self.inner_width = spec.num_heads * spec.head_dim
        self.input_rows = None                                           # every projection reads a blend of its own
        self.out_weight = tensors["o"]
        self.mu = torch.stack([tensors[f"mu.{s}"] for s in "rkvgw"]).to(**f32).contiguous()
        self.rkvg = torch.stack([tensors[s] for s in "rkvg"]).to(device=rt.device, dtype=rt.dtype).contiguous()
        self.decay_down, self.decay_up = Linear(tensors["w1"], rt), Linear(tensors["w2"], rt)
        self.w0, self.u, self.norm_weight = (tensors[n].to(**f32).contiguous() for n in ("w0", "u", "norm"))
        self.matrix_bytes = spec.num_heads * spec.head_dim * spec.head_dim * 4
        self.out = None if fused else Linear(self.out_weight, rt)

    def state_bytes(self) -> int:
        return self.matrix_bytes + self.spec.hidden_size * 4

    def inner(self, y: torch.Tensor | None, x: torch.Tensor, ctx, binding, scale: float = 1.0,
              out: torch.Tensor | None = None) -> torch.Tensor:
        """x: the mixer's input (`y`, columns of a projection of it, is not used).  Returns [T, heads * head_dim] * scale."""
        s, ops = self.spec, self.rt.ops
        H, D = s.num_heads, s.head_dim
        matrices = dataclasses.replace(binding, state=binding.state[:, :self.matrix_bytes])
        previous = dataclasses.replace(binding, state=binding.state[:, self.matrix_bytes:self.matrix_bytes + s.hidden_size * 4])
        mixes = ops.token_shift(x, self.mu, ctx, previous)               # [5, T, hidden]
        r, k, v, g = ops.linear_groups(mixes[:4], self.rkvg)
        low = ops.linear_unary(mixes[4], self.decay_down.weight, "tanh")
        z = self.decay_up(low, out_dtype=torch.float32)                   # decay logits, float32 from here on
        o, tiles = None, ops.portions_by_tiles(ctx)
        if tiles:                                        # prompt portions sixteen tokens at a time
            o = ops.mix_tiles(r, k, v, z, self.w0, self.u, ctx, matrices, heads=H, dim=D)
        singles = not tiles or ctx.min_q_len <= 1        # single tokens (or every request) by the scan
        prepared, bonus = ops.time_mix_prepare(r, k, z, self.w0, self.u, x, ctx, previous, heads=H, dim=D,
                                               rows="all" if not tiles else "singles" if singles else "none")
        if singles:
            o = ops.recurrence_scan(prepared, v, ctx, matrices, heads=H, dim=D, vdim=D, bonus=bonus, singles=tiles, out=o)
        return ops.head_norm_gate(o, g, self.norm_weight, H, D, s.out_norm_eps, x.dtype, gate_kind="silu", weight_per_head=True,
                                  scale=scale, out=out)

    def forward(self, x: torch.Tensor, ctx, binding) -> torch.Tensor:
        return self.out(self.inner(None, x, ctx, binding))
