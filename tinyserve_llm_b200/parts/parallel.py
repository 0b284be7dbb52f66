"""
Mixers side by side on one input: y = sum_b scale_b * mixer_b(h).

Each branch is a mixer of its own kind that also exposes what lies between its projections
(`input_rows`: the stacked weights that read h; `inner(y, x, ctx, binding, scale, out)`: from its
columns of the fused projection to the input of its output projection, times `scale`; `out_weight`).
The branches' input projections run as one product and so do their output projections,

    [y_1 | y_2 | ...] = h . [W_1; W_2; ...]^T        y = [s_1 inner_1 | s_2 inner_2 | ...] . [O_1 | O_2 | ...]^T

so the weighted sum costs nothing of its own.  A branch whose projections do not read h as it is has no
input rows (`input_rows` None) and gets `y` None.  With a norm on each branch's output,

    y = sum_b s_b * rms_norm(O_b inner_b) * w_b

the output projections stay apart (one grouped launch where the branches are equally wide), and
`forward_branches` hands the pair to the norm that closes the sublayer, which works out the sum in its
own kernel; `forward` gives the sum itself.  At most one branch keeps keys and values (it gets
the cache entry's pages); the branches' states are laid one behind the other in the entry's slot.
"""

from __future__ import annotations

import dataclasses
import inspect

import torch

from tinyserve_llm_b200.config.spec import ParallelMixerSpec
from tinyserve_llm_b200.parts.base import KVNeed, Mixer, Runtime, TensorDecl, part_class, register_part
from tinyserve_llm_b200.parts.linear import Linear, fuse_rows

STATE_ALIGN = 256


@register_part("mixer", "parallel")
class ParallelMixer(Mixer):
    @classmethod
    def declare(cls, spec: ParallelMixerSpec) -> dict[str, TensorDecl]:
        if not spec.branches:
            raise ValueError("a parallel mixer needs at least one branch")
        out: dict[str, TensorDecl] = {}
        for part, prefix, _ in spec.branches:
            for name, decl in part_class("mixer", part).declare(part).items():
                out[prefix + name] = decl
        if spec.norm_names and (len(spec.norm_names) != 2 or len(spec.branches) != 2):
            raise NotImplementedError("norms on the outputs of a parallel mixer's branches: of two branches, one each")
        for name in spec.norm_names:
            out[name] = TensorDecl((spec.hidden_size,), init="unit")
        return out

    def __init__(self, spec: ParallelMixerSpec, tensors: dict[str, torch.Tensor], rt: Runtime) -> None:
        super().__init__(spec, tensors, rt)
        self.branches, self.scales = [], []
        for part, prefix, scale in spec.branches:
            cls = part_class("mixer", part)
            sub = {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}
            if "fused" not in inspect.signature(cls.__init__).parameters:
                raise NotImplementedError(f"a {part.kind} mixer cannot be a branch of a parallel mixer: it does not expose "
                                          "its input rows, inner part and output weight")
            self.branches.append(cls(part, sub, rt, fused=True))
            self.scales.append(float(scale))
        if sum(b.kv_need() is not None for b in self.branches) > 1:
            raise NotImplementedError("at most one branch of a parallel mixer may keep keys and values")
        self.graph_safe = all(getattr(b, "graph_safe", False) for b in self.branches)
        rows = [b.input_rows for b in self.branches if b.input_rows is not None]
        self.proj = Linear(fuse_rows(rows), rt) if rows else None
        self.out, self.outs, self.grouped_out = None, None, None
        if not spec.norm_names:
            self.out = Linear(torch.cat([b.out_weight for b in self.branches], dim=1).contiguous(), rt)
        elif self.branches[0].inner_width == self.branches[1].inner_width:
            self.grouped_out = torch.stack([b.out_weight for b in self.branches]).to(device=rt.device, dtype=rt.dtype).contiguous()
        else:
            self.outs = [Linear(b.out_weight, rt) for b in self.branches]
        self.norm_weights = [tensors[n].to(device=rt.device, dtype=torch.float32).contiguous() for n in spec.norm_names]
        self.in_offsets, self.inner_offsets, self.state_offsets = [0], [0], [0]
        for b in self.branches:
            self.in_offsets.append(self.in_offsets[-1] + (b.input_rows.shape[0] if b.input_rows is not None else 0))
            self.inner_offsets.append(self.inner_offsets[-1] + b.inner_width)
            self.state_offsets.append(self.state_offsets[-1] + -(-int(b.state_bytes()) // STATE_ALIGN) * STATE_ALIGN)
        for b in self.branches:
            b.input_rows = b.out_weight = None          # the fused weights are the ones that stay

    def kv_need(self) -> KVNeed | None:
        return next((b.kv_need() for b in self.branches if b.kv_need() is not None), None)

    def state_bytes(self) -> int:
        return self.state_offsets[-1]

    def _run_branch(self, i: int, y: torch.Tensor | None, x: torch.Tensor, ctx, binding, scale: float, out: torch.Tensor) -> None:
        branch, own = self.branches[i], binding
        lo, size = self.state_offsets[i], int(branch.state_bytes())
        if binding is not None and binding.state is not None:
            own = dataclasses.replace(binding, state=binding.state[:, lo:lo + size] if size else None)
        has_rows = self.in_offsets[i + 1] > self.in_offsets[i]
        branch.inner(y[:, self.in_offsets[i]:self.in_offsets[i + 1]] if has_rows else None, x, ctx, own, scale, out)

    def forward_branches(self, x: torch.Tensor, ctx, binding) -> tuple[torch.Tensor, tuple]:
        """With norms: the first branch's output and (the second's, both norms' weights, both scales); see `Ops.normed_sum`."""
        y = self.proj(x) if self.proj is not None else None
        T, widths = x.shape[0], [b.inner_width for b in self.branches]
        if self.grouped_out is not None:
            inner = torch.empty((2, T, widths[0]), dtype=x.dtype, device=x.device)
        else:
            inner = [torch.empty((T, w), dtype=x.dtype, device=x.device) for w in widths]
        for i in range(2):
            self._run_branch(i, y, x, ctx, binding, 1.0, inner[i])
        if self.grouped_out is not None:
            a, b = self.rt.ops.linear_groups(inner, self.grouped_out)
        else:
            a, b = (out(h) for out, h in zip(self.outs, inner))
        return a, (b, *self.norm_weights, *self.scales)

    def forward(self, x: torch.Tensor, ctx, binding) -> torch.Tensor:
        if self.norm_weights:
            a, pair = self.forward_branches(x, ctx, binding)
            return self.rt.ops.normed_sum(a, pair, float(self.spec.norm_eps))
        y = self.proj(x) if self.proj is not None else None
        inner = torch.empty((x.shape[0], self.inner_offsets[-1]), dtype=x.dtype, device=x.device)
        for i, scale in enumerate(self.scales):
            self._run_branch(i, y, x, ctx, binding, scale, inner[:, self.inner_offsets[i]:self.inner_offsets[i + 1]])
        return self.out(inner)
