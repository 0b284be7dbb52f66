"""
Gated delta rule: a matrix state per request and value head that is decayed, corrected towards the
current value along the current key, and read with the query.

    q, k, v = silu(short_conv(W h))        causal convolution over time per channel, its last inputs carried
    q, k    <- unit vectors per head (x / sqrt(sum x^2 + unit_eps)),  q <- q * q_scale
    beta = sigmoid(W_b h)                   a = exp(-exp(A_log) softplus(W_a2 (W_a1 h) + dt_bias))
    S <- diag(a) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q       per value head, S [key_dim, value_dim]
    y = W_o ( o / rms(o) * w * sigmoid(W_g2 (W_g1 h)) )

Two variants by the spec: one decay a head, a = exp(-exp(A_log) softplus(W_a h + dt_bias)) (`decay_scope`
"head": the decay's logits come with beta's out of one product), and an output gate silu(W_g h) (`gate`
"silu": its rows join the projection of q, k and v).

Value head h uses q/k head h // (heads / kv_heads).  The state (float32: the matrices, then the
convolution's last taps - 1 inputs) lives in the request's slot of the cache manager, so prompts in
portions, decoding and mixed batches are one code path.  Beta's projection and the decay logits
leave their products in float32; everything from the convolution's output on is float32.

Like `GatedAttention` the mixer stands alone or inside a `ParallelMixer` (`input_rows`, `inner`,
`out_weight`).
"""

from __future__ import annotations

import dataclasses

import torch

from tinyserve_llm_b200.config.spec import GatedDeltaRuleSpec
from tinyserve_llm_b200.parts.base import Mixer, Runtime, TensorDecl, register_part
from tinyserve_llm_b200.parts.linear import Linear, fuse_rows

MAX_KEY_DIM = 256       # csrc/linear_recurrence.cu


@register_part("mixer", "gated_delta_rule")
class GatedDeltaRule(Mixer):
    graph_safe = True

    @classmethod
    def validate(cls, spec: GatedDeltaRuleSpec) -> None:
        if spec.num_kv_heads <= 0 or spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"num_heads={spec.num_heads} is not a multiple of num_kv_heads={spec.num_kv_heads}")
        if not 0 < spec.key_dim <= MAX_KEY_DIM:
            raise ValueError(f"key_dim={spec.key_dim} is not supported: the recurrence kernel takes up to {MAX_KEY_DIM}")
        if spec.decay_scope not in ("channel", "head") or spec.gate not in ("low_rank_sigmoid", "silu"):
            raise NotImplementedError(f"delta rule: decay scope {spec.decay_scope!r}, gate {spec.gate!r}")
        if spec.conv_taps < 1:
            raise ValueError(f"conv_taps={spec.conv_taps}: the convolution has at least the current token's tap")

    @classmethod
    def declare(cls, spec: GatedDeltaRuleSpec) -> dict[str, TensorDecl]:
        cls.validate(spec)
        qk, vv, hidden, taps = spec.num_kv_heads * spec.key_dim, spec.num_heads * spec.value_dim, spec.hidden_size, spec.conv_taps
        ra = spec.decay_rank if spec.decay_rank > 0 else -1          # -1: the checkpoint's own size
        rg = spec.gate_rank if spec.gate_rank > 0 else -1
        out = {
            "q": TensorDecl((qk, hidden)), "q.conv": TensorDecl((qk, taps)),
            "k": TensorDecl((qk, hidden)), "k.conv": TensorDecl((qk, taps)),
            "v": TensorDecl((vv, hidden)), "v.conv": TensorDecl((vv, taps)),
            "b": TensorDecl((spec.num_heads, hidden)), "A_log": TensorDecl((spec.num_heads,)),
            "norm": TensorDecl((spec.value_dim,), init="unit"),
            "o": TensorDecl((hidden, vv)),
        }
        if spec.decay_scope == "head":
            out.update({"a": TensorDecl((spec.num_heads, hidden)), "dt_bias": TensorDecl((spec.num_heads,))})
        else:
            out.update({"a1": TensorDecl((ra, hidden)), "a2": TensorDecl((spec.num_heads * spec.key_dim, ra)),
                        "dt_bias": TensorDecl((spec.num_heads * spec.key_dim,))})
        if spec.gate == "silu":
            out["g"] = TensorDecl((vv, hidden))
        else:
            out.update({"g1": TensorDecl((rg, hidden)), "g2": TensorDecl((vv, rg))})
        return out

    def __init__(self, spec: GatedDeltaRuleSpec, tensors: dict[str, torch.Tensor], rt: Runtime, fused: bool = False) -> None:
        super().__init__(spec, tensors, rt)
        self.validate(spec)
        self.head_decay, self.full_gate = spec.decay_scope == "head", spec.gate == "silu"
        for a, b in ([] if self.head_decay else [("a1", "a2")]) + ([] if self.full_gate else [("g1", "g2")]):
            if tensors[a].shape[0] != tensors[b].shape[1]:
                raise ValueError(f"the inner sizes of {a} and {b} differ: {tuple(tensors[a].shape)} and {tuple(tensors[b].shape)}")
        f32 = dict(device=rt.device, dtype=torch.float32)
        self.decay_rank = 0 if self.head_decay else int(tensors["a1"].shape[0])
        gate_rows = tensors["g" if self.full_gate else "g1"]
        self.gate_rank = int(gate_rows.shape[0])
        self.channels = 2 * spec.num_kv_heads * spec.key_dim + spec.num_heads * spec.value_dim
        # one projection for what reads h and may be rounded: columns [q | k | v | a1 h | g1 h], or [q | k | v | g h]
        self.input_rows = fuse_rows([tensors["q"], tensors["k"], tensors["v"]] + ([] if self.head_decay else [tensors["a1"]]) + [gate_rows])
        self.out_weight = tensors["o"]
        self.inner_width = spec.num_heads * spec.value_dim
        self.taps = torch.cat([tensors["q.conv"], tensors["k.conv"], tensors["v.conv"]], dim=0).to(**f32).contiguous()
        # the step sizes' logits, and with one decay a head the decays', in one float32 product
        self.beta = Linear(fuse_rows([tensors["b"], tensors["a"]]) if self.head_decay else tensors["b"], rt)
        self.decay_up = None if self.head_decay else Linear(tensors["a2"], rt)
        self.gate_up = None if self.full_gate else Linear(tensors["g2"], rt)
        self.dt_bias = tensors["dt_bias"].to(**f32).contiguous()
        self.a_log = tensors["A_log"].to(**f32).contiguous()
        self.norm_weight = tensors["norm"].to(**f32).contiguous()
        self.matrix_bytes = spec.num_heads * spec.key_dim * spec.value_dim * 4
        self.conv_bytes = (spec.conv_taps - 1) * self.channels * 4
        self.proj = self.out = None
        if not fused:
            self.proj, self.out = Linear(self.input_rows, rt), Linear(self.out_weight, rt)

    def state_bytes(self) -> int:
        return self.matrix_bytes + self.conv_bytes

    def inner(self, y: torch.Tensor, x: torch.Tensor, ctx, binding, scale: float = 1.0,
              out: torch.Tensor | None = None) -> torch.Tensor:
        """y: this mixer's columns of the projection of x, [q | k | v | a1 h | g1 h or g h].  Returns [T, heads * value_dim] * scale."""
        s, ops = self.spec, self.rt.ops
        H, G, D, V, C = s.num_heads, s.num_kv_heads, s.key_dim, s.value_dim, self.channels
        matrices = dataclasses.replace(binding, state=binding.state[:, :self.matrix_bytes])
        if s.conv_taps > 1:
            carried = dataclasses.replace(binding, state=binding.state[:, self.matrix_bytes:self.matrix_bytes + self.conv_bytes])
        else:
            carried = matrices                      # nothing is carried; the kernel wants a slot all the same
        conv = ops.short_conv_silu(y[:, :C], self.taps, ctx, carried)                        # float32 [T, C]
        gate = y[:, C + self.decay_rank:C + self.decay_rank + self.gate_rank]
        if not self.full_gate:
            gate = self.gate_up(gate.contiguous())
        b = self.beta(x, out_dtype=torch.float32)
        q, k, v = conv[:, :G * D], conv[:, G * D:2 * G * D], conv[:, 2 * G * D:]
        sizes = dict(heads=H, kv_heads=G, dim=D, unit_eps=s.unit_eps, q_scale=s.q_scale)
        if self.head_decay:
            o, tiles = None, ops.portions_by_tiles(ctx)
            if tiles:                                   # prompt portions sixteen tokens at a time
                o = ops.delta_tiles(q, k, v, b, self.dt_bias, self.a_log, ctx, matrices, vdim=V, **sizes)
            if not tiles or ctx.min_q_len <= 1:         # single tokens (or every request) by the scan
                prepared, beta, decay = ops.delta_prepare_head(q, k, b, self.dt_bias, self.a_log, singles=ctx if tiles else None, **sizes)
                o = ops.recurrence_scan(prepared, v, ctx, matrices, heads=H, dim=D, vdim=V, beta=beta, head_decay=decay,
                                        qk_group=H // G, singles=tiles, out=o)
        else:
            z = self.decay_up(y[:, C:C + self.decay_rank].contiguous(), out_dtype=torch.float32)  # decay logits, float32 from here on
            prepared, beta = ops.delta_prepare(q, k, z, self.dt_bias, self.a_log, b, **sizes)
            o = ops.recurrence_scan(prepared, v, ctx, matrices, heads=H, dim=D, vdim=V, beta=beta)
        return ops.head_norm_gate(o, gate, self.norm_weight, H, V, s.out_norm_eps, x.dtype,
                                  gate_kind="silu" if self.full_gate else "sigmoid", scale=scale, out=out)

    def forward(self, x: torch.Tensor, ctx, binding) -> torch.Tensor:
        return self.out(self.inner(self.proj(x), x, ctx, binding))
