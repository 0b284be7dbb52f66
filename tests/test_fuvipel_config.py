"""Host-side tests of the Fuvipel configuration, its model description and the plain implementation."""

import copy

import pytest
import torch

import fuvipel_configs as C
import plain_fuvipel as plain
from tinyserve_llm_b200.cache.manager import plan_layout
from tinyserve_llm_b200.config import ConfigError
from tinyserve_llm_b200.config.fuvipel import FuvipelConfig, fuvipel_model_spec
from tinyserve_llm_b200.config.registry import resolve_architecture
from tinyserve_llm_b200.config.spec import GatedAttentionSpec, GatedDeltaRuleSpec, ParallelMixerSpec, TimeMixingSpec
from tinyserve_llm_b200.parts.base import KVNeed
from tinyserve_llm_b200.parts.model import declared_tensors
from tinyserve_llm_b200.weights import random_tensors


def test_every_size_and_constant_comes_from_the_configuration():
    spec = fuvipel_model_spec(FuvipelConfig.from_dict(C.MIXED))
    assert resolve_architecture(C.MIXED).name == "Fuvipel"
    assert spec.vocab_size == 300 and spec.hidden_size == 96 and len(spec.blocks) == 5 and spec.lm_head_name is None
    assert all(b.arrangement == "post_norm_stream" and b.mixer_norm is None and b.mixer_post_norm.eps == 1e-5 for b in spec.blocks)
    first = spec.blocks[0].mixer
    assert isinstance(first, ParallelMixerSpec) and [(b[1], b[2]) for b in first.branches] == [("left.", 0.5), ("right.", 0.5)]
    assert first.norm_names == ("left.out", "right.out") and first.norm_eps == 1e-5 and first.hidden_size == 96
    left, right = first.branches[0][0], first.branches[1][0]
    assert isinstance(left, GatedAttentionSpec) and isinstance(right, TimeMixingSpec)
    assert (left.num_heads, left.num_kv_heads, left.head_dim, left.value_dim, left.scale) == (4, 2, 20, 20, 0.3)
    assert (left.position.dims, left.position.base, left.position.interleaved) == (12, 5000.0, True)
    assert left.values == "keys" and left.sink == 0.0 and left.output_gate and left.qk_norm and not left.qk_norm_weight
    assert left.qk_norm_scope == "head" and left.qk_norm_eps == 1e-5 and not left.bias and left.window == 0
    assert (right.num_heads, right.head_dim, right.decay_rank, right.out_norm_eps) == (3, 24, 10, 1e-5)
    rule = spec.blocks[1].mixer
    assert isinstance(rule, GatedDeltaRuleSpec) and (rule.decay_scope, rule.gate) == ("head", "silu")
    assert (rule.num_heads, rule.num_kv_heads, rule.key_dim, rule.value_dim, rule.conv_taps) == (4, 2, 20, 24, 3)
    assert rule.q_scale == 20 ** -0.5 and rule.unit_eps == 1e-6
    assert spec.blocks[1].feed_forward is None and spec.blocks[3].feed_forward is None
    assert (spec.blocks[2].feed_forward.intermediate_size, spec.blocks[2].feed_forward.activation) == (40, "relu2")


def test_declared_tensors_follow_the_sizes():
    d = declared_tensors(fuvipel_model_spec(FuvipelConfig.from_dict(C.MIXED)))
    assert d["embed"].shape == (300, 96) and d["final.norm"].shape == (96,) and d["l0.norm1"].shape == (96,)
    assert d["l0.mix.left.q"].shape == (80, 96) and d["l0.mix.left.k"].shape == (40, 96) and d["l0.mix.left.g"].shape == (80, 96)
    assert d["l0.mix.left.o"].shape == (96, 80) and d["l0.mix.left.out"].shape == (96,) and d["l0.mix.right.out"].shape == (96,)
    assert not any(n.startswith("l0.mix.left.v") or n.startswith("l0.mix.left.q.") for n in d)
    assert d["l0.mix.right.w1"].shape == (10, 96) and d["l0.mix.right.w2"].shape == (72, 10) and d["l0.mix.right.w0"].shape == (72,)
    assert d["l0.mix.right.u"].shape == (3, 24) and d["l0.mix.right.mu.w"].shape == (96,) and d["l0.mix.right.norm"].shape == (72,)
    assert d["l1.mix.a"].shape == (4, 96) and d["l1.mix.dt_bias"].shape == (4,) and d["l1.mix.A_log"].shape == (4,)
    assert d["l1.mix.g"].shape == (96, 96) and d["l1.mix.v.conv"].shape == (96, 3) and d["l2.mix.k.conv"].shape == (108, 5)
    assert not any(".a1" in n or ".g1" in n for n in d)
    assert d["l2.mlp.up"].shape == (40, 96) and d["l2.norm2"].shape == (96,)
    assert not any(n.startswith("l1.mlp.") or n == "l1.norm2" or n == "l3.norm2" for n in d)
    raw = copy.deepcopy(C.MIXED)
    del raw["layers"][0]["mixer"]["right"]["decay_rank"]                      # the size is then the checkpoint's
    assert declared_tensors(fuvipel_model_spec(FuvipelConfig.from_dict(raw)))["l0.mix.right.w1"].shape == (-1, 96)


@pytest.mark.parametrize("edit, message", [
    (lambda r: r["layers"][0].update(type="attention"), "layers[0].type"),
    (lambda r: r["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][0]["mixer"]["left"].update(vdim=24), "vdim"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=22), "rot.dims"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda r: r["layers"][0]["mixer"]["right"].pop("dim"), "dim"),
    (lambda r: r["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda r: r["layers"][2]["mlp"].update(kind="moe"), "mlp"),
    (lambda r: r["norm"].pop("eps"), "norm.eps"),
])
def test_what_cannot_be_served_is_refused_with_the_key(edit, message):
    raw = copy.deepcopy(C.MIXED)
    edit(raw)
    with pytest.raises(ConfigError, match=message.replace("[", r"\[").replace("]", r"\]")):
        FuvipelConfig.from_dict(raw)


def test_other_mixers_refuse_a_rotation_of_neighbouring_channels():
    from tinyserve_llm_b200.config.spec import InlineRotarySpec, LinearRecurrenceSpec
    from tinyserve_llm_b200.parts.base import Runtime, part_class
    spec = LinearRecurrenceSpec(hidden_size=8, num_heads=1, key_dim=4, value_dim=4, head_decays=(0.5,),
                                position=InlineRotarySpec(dims=4, interleaved=True))
    cls = part_class("mixer", spec)
    tensors = {n: torch.zeros(d.shape) for n, d in cls.declare(spec).items()}
    with pytest.raises(NotImplementedError, match="neighbouring"):
        cls(spec, tensors, Runtime(dtype=torch.float32, device=torch.device("cpu"), ops=None))


def test_cache_layout_has_pages_for_the_attention_and_a_slot_for_every_state():
    from tinyserve_llm_b200.parts.base import Runtime, part_class
    spec = fuvipel_model_spec(FuvipelConfig.from_dict(C.MIXED))
    rt = Runtime(dtype=torch.float32, device=torch.device("cpu"), ops=None)
    needs = []
    for block in spec.blocks:
        cls = part_class("mixer", block.mixer)
        tensors = {n: torch.zeros(d.shape) for n, d in cls.declare(block.mixer).items()}
        mixer = cls(block.mixer, tensors, rt)
        needs.append((mixer.kv_need(), int(mixer.state_bytes())))
    assert needs[0][0] == KVNeed(2, 20) and needs[3][0] == KVNeed(1, 16) and needs[1][0] is None
    assert needs[0][1] >= 4 * (3 * 24 * 24 + 96) and needs[1][1] == 4 * (4 * 20 * 24 + 2 * (2 * 2 * 20 + 4 * 24))
    layout = plan_layout(needs, 16)
    assert layout is not None
    recurrent = fuvipel_model_spec(FuvipelConfig.from_dict(C.RECURRENT))
    assert all(part_class("mixer", b.mixer).kv_need is not None for b in recurrent.blocks)


def test_the_plain_model_does_not_depend_on_later_tokens_and_reads_far_ones():
    """Causality of every mechanism of the plain implementation, and a state that carries the first token to the last."""
    raw = C.MIXED
    tensors = dict(random_tensors(declared_tensors(fuvipel_model_spec(FuvipelConfig.from_dict(raw))), 5, **C.WEIGHTS))
    g = torch.Generator().manual_seed(0)
    ids = torch.randint(0, raw["vocab"], (40,), generator=g).tolist()
    full = plain.forward(raw, tensors, ids)
    torch.testing.assert_close(plain.forward(raw, tensors, ids[:17]), full[:17], atol=1e-10, rtol=1e-10)
    other = list(ids)
    other[0] = (ids[0] + 1) % raw["vocab"]
    assert float((plain.forward(raw, tensors, other)[-1] - full[-1]).abs().max()) > 1e-6


def test_plain_softmax_with_a_sink_by_hand():
    s = torch.tensor([[0.0, 7.0], [1.0, -2.0]], dtype=torch.float64)
    p = plain.softmax_with_sink(s, torch.tensor([[True, False], [True, True]]))
    e1, e2 = torch.exp(torch.tensor(1.0, dtype=torch.float64)), torch.exp(torch.tensor(-2.0, dtype=torch.float64))
    torch.testing.assert_close(p, torch.stack([torch.tensor([0.5, 0.0], dtype=torch.float64), torch.stack([e1, e2]) / (1 + e1 + e2)]))
