"""
Griffin's recurrent block: a gated branch beside a short convolution and a real-gated linear recurrent unit.

    y = gelu_tanh(W_y h + b_y)        u = conv(W_x h + b_x)       (causal, one filter and a bias a channel)
    r = sigmoid(R_b u_b + c_b), i = sigmoid(I_b u_b + d_b)        part b of u by part b's square matrices
    log a = -decay_rate * r * softplus(lam)
    S_t = a S_(t-1) + sqrt(1 - a^2) i u                           one number a channel, zero before the first token
    out = W_o (S * y)

Both projections are one product [y | x].  The block-diagonal gates are one batched product over the parts, [R_b; I_b]
stacked, with float32 output; everything from there on is float32.  A step in which every request feeds one token runs
from the projection to the input of W_o in one kernel (bfloat16, sizes it takes); other steps in a convolution kernel, the
batched product and a scan that takes long portions in stretches side by side.  The request's slot of the cache manager
holds the convolution's last inputs as a ring by position, then the state: zeroed at admission, given back at release.

Tensors (local names): y, y.b, x, x.b, conv, conv.b, ra, ra.b, ri, ri.b, lam, o.
"""

from __future__ import annotations

import torch

from tinyserve_llm_b200.config.spec import GatedLRUSpec
from tinyserve_llm_b200.parts.base import Mixer, Runtime, TensorDecl, register_part
from tinyserve_llm_b200.parts.linear import Linear, fuse_rows


@register_part("mixer", "gated_lru")
class GatedLRU(Mixer):
    graph_safe = True

    @classmethod
    def validate(cls, spec: GatedLRUSpec) -> None:
        if spec.blocks <= 0 or spec.width <= 0 or spec.width % spec.blocks or spec.conv_taps <= 0:
            raise ValueError(f"a gated linear recurrent unit of {spec.width} channels in {spec.blocks} parts with {spec.conv_taps} taps")

    @classmethod
    def declare(cls, spec: GatedLRUSpec) -> dict[str, TensorDecl]:
        cls.validate(spec)
        W, hidden, B = spec.width, spec.hidden_size, spec.blocks
        part = W // B
        return {"y": TensorDecl((W, hidden)), "y.b": TensorDecl((W,)), "x": TensorDecl((W, hidden)), "x.b": TensorDecl((W,)),
                "conv": TensorDecl((W, spec.conv_taps)), "conv.b": TensorDecl((W,)),
                "ra": TensorDecl((B, part, part)), "ra.b": TensorDecl((B, part)),
                "ri": TensorDecl((B, part, part)), "ri.b": TensorDecl((B, part)),
                "lam": TensorDecl((W,)), "o": TensorDecl((hidden, W))}

    def __init__(self, spec: GatedLRUSpec, tensors: dict[str, torch.Tensor], rt: Runtime, fused: bool = False) -> None:
        super().__init__(spec, tensors, rt)
        self.validate(spec)
        f32 = lambda t: t.to(device=rt.device, dtype=torch.float32).contiguous()  # noqa: E731
        self.input_rows = fuse_rows([tensors["y"], tensors["x"]])
        self.out_weight = tensors["o"]
        self.inner_width = spec.width
        self.y_bias, self.x_bias = f32(tensors["y.b"]), f32(tensors["x.b"])
        self.taps = f32(tensors["conv"].to(torch.float32).t())                 # [taps, width]
        self.conv_bias = f32(tensors["conv.b"])
        self.gates = torch.cat([tensors["ra"], tensors["ri"]], dim=1).to(device=rt.device, dtype=rt.dtype).contiguous()
        self.gate_bias = f32(torch.stack([tensors["ra.b"].reshape(-1), tensors["ri.b"].reshape(-1)]))
        lam = tensors["lam"].to(torch.float64)
        self.rate = f32(-float(spec.decay_rate) * (lam.clamp_min(0.0) + torch.log1p(torch.exp(-lam.abs()))))   # -c softplus(lam)
        self.proj = self.out = None
        if not fused:
            self.proj, self.out = Linear(self.input_rows, rt), Linear(self.out_weight, rt)

    def state_bytes(self) -> int:
        ring = self.spec.conv_taps if self.spec.conv_taps > 1 else 0
        return (ring + 1) * self.spec.width * 4

    def inner(self, y: torch.Tensor, x: torch.Tensor, ctx, binding, scale: float = 1.0,
              out: torch.Tensor | None = None) -> torch.Tensor:
        """y: this mixer's columns [y | x] of the projection of x.  Returns [T, width] * scale."""
        o = self.rt.ops.gated_lru(y, self, ctx, binding)
        if scale != 1.0:
            o = o * scale
        if out is not None:
            out.copy_(o)
            return out
        return o

    def forward(self, x: torch.Tensor, ctx, binding) -> torch.Tensor:
        return self.out(self.inner(self.proj(x), x, ctx, binding))
