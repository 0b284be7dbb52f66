"""Host-side tests of the Gimotar configuration, its model description, its step data and the plain implementation."""

import copy
from types import SimpleNamespace

import pytest
import torch

import gimotar_configs as C
import plain_gimotar as plain
from tinyserve_llm_b200.cache.manager import CacheManager, plan_layout
from tinyserve_llm_b200.config import ConfigError
from tinyserve_llm_b200.config.gimotar import GimotarConfig, gimotar_model_spec
from tinyserve_llm_b200.config.registry import resolve_architecture
from tinyserve_llm_b200.config.spec import GatedAttentionSpec, GatedLRUSpec, LatentAttentionSpec
from tinyserve_llm_b200.parts.base import KVNeed
from tinyserve_llm_b200.parts.model import declared_tensors
from tinyserve_llm_b200.weights import random_tensors


def spec_of(raw):
    return gimotar_model_spec(GimotarConfig.from_dict(raw))


def test_every_size_and_constant_comes_from_the_configuration():
    spec = spec_of(C.MIXED)
    assert resolve_architecture(C.MIXED).name == "Gimotar"
    assert spec.vocab_size == 300 and spec.hidden_size == 96 and len(spec.blocks) == 7 and spec.lm_head_name is None
    assert spec.embedding_scale == 3.0
    pairs = spec.embedding_pairs
    assert (pairs.size, pairs.buckets, pairs.mul_prev, pairs.mul_cur, pairs.name) == (96, 101, 13, 5, "bigram")
    for b in spec.blocks:
        assert b.arrangement == "parallel_stream" and b.branch_scale == 0.7 and b.feed_forward_norm is None
        assert (b.mixer_norm.eps, b.mixer_norm.weight_offset) == (1e-5, 1.0)
    lru = spec.blocks[0].mixer
    assert isinstance(lru, GatedLRUSpec) and (lru.width, lru.blocks, lru.conv_taps, lru.decay_rate) == (120, 5, 3, 8.0)
    att = spec.blocks[1].mixer
    assert isinstance(att, GatedAttentionSpec) and (att.num_heads, att.num_kv_heads, att.head_dim, att.value_dim) == (4, 2, 20, 36)
    assert (att.scale, att.chunk, att.position.dims, att.position.base, att.position.interleaved) == (0.3, 11, 12, 500.0, False)
    assert att.qk_norm and att.qk_norm_scope == "head" and att.qk_norm_weight and att.qk_norm_eps == 1e-5 and not att.bias
    lat = spec.blocks[2].mixer
    assert isinstance(lat, LatentAttentionSpec) and (lat.num_heads, lat.head_dim, lat.rot_dim, lat.value_dim, lat.kv_rank) == (5, 24, 12, 20, 40)
    assert lat.sink and lat.output_gate and lat.q_rank == 0 and lat.window == 0 and lat.norm_eps == 1e-5 and lat.scale == 0.2
    assert lat.position.interleaved and (lat.position.yarn.factor, lat.position.yarn.original, lat.position.yarn.fast, lat.position.yarn.slow) == (4.0, 64.0, 16.0, 2.0)
    moe = spec.blocks[0].feed_forward
    assert (moe.num_experts, moe.top, moe.expert.intermediate_size, moe.shared.intermediate_size) == (5, 2, 40, 24)
    assert moe.scoring == "softmax_chosen" and moe.router_bias_name == "router.b" and moe.expert.activation == "silu"
    assert spec.blocks[2].feed_forward is None and spec.blocks[3].feed_forward.shared is None


def test_the_first_mixing_layer_gives_its_values_and_the_others_mix_them_in():
    spec = spec_of(C.MIXED)
    assert [b.mixer.value_mix for b in spec.blocks if isinstance(b.mixer, GatedAttentionSpec)] == ["source", "none", "mixed", "mixed"]
    d = declared_tensors(spec)
    assert "l1.mix.vmix" not in d and "l3.mix.vmix" not in d and d["l4.mix.vmix"].shape == () and d["l6.mix.vmix"].shape == ()
    assert spec.optional_tensors == ("l1.mix.vmix",)               # a checkpoint may carry the source layer's number
    raw = copy.deepcopy(C.MIXED)
    raw["layers"][1]["mixer"]["v_mix"] = False
    assert spec_of(raw).optional_tensors == ("l4.mix.vmix",)
    assert spec_of(C.RECURRENT).optional_tensors == ()


def test_declared_tensors_follow_the_sizes():
    d = declared_tensors(spec_of(C.MIXED))
    assert d["embed"].shape == (300, 96) and d["bigram"].shape == (102, 96) and d["final.norm"].shape == (96,)
    assert d["l0.norm1"].shape == (96,) and "l0.norm2" not in d
    assert d["l0.mix.y"].shape == (120, 96) and d["l0.mix.x.b"].shape == (120,) and d["l0.mix.conv"].shape == (120, 3)
    assert d["l0.mix.ra"].shape == (5, 24, 24) and d["l0.mix.ri.b"].shape == (5, 24) and d["l0.mix.lam"].shape == (120,)
    assert d["l0.mix.o"].shape == (96, 120)
    assert d["l1.mix.q"].shape == (80, 96) and d["l1.mix.k"].shape == (40, 96) and d["l1.mix.v"].shape == (72, 96)
    assert d["l1.mix.q.norm"].shape == (20,) and d["l1.mix.o"].shape == (96, 144) and "l1.mix.q.b" not in d
    assert d["l2.mix.q"].shape == (180, 96) and d["l2.mix.dkv"].shape == (52, 96) and d["l2.mix.dkv.norm"].shape == (40,)
    assert d["l2.mix.uk"].shape == (120, 40) and d["l2.mix.uv"].shape == (100, 40) and d["l2.mix.sink"].shape == (5,)
    assert d["l2.mix.g"].shape == (100, 96) and d["l2.mix.o"].shape == (96, 100)
    assert d["l0.mlp.router"].shape == (5, 96) and d["l0.mlp.router.b"].shape == (5,) and d["l0.mlp.e4.down"].shape == (96, 40)
    assert d["l0.mlp.shared.gate"].shape == (24, 96) and not any(n.startswith("l2.mlp.") for n in d) and "l3.mlp.shared.up" not in d


@pytest.mark.parametrize("edit, message", [
    (lambda r: r["layers"][0].update(type="mamba"), "layers[0].type"),
    (lambda r: r["layers"][0]["mixer"].update(blocks=7), "blocks"),
    (lambda r: r["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda r: r["layers"][1]["mixer"]["rot"].update(dims=22), "rot.dims"),
    (lambda r: r["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda r: r["layers"][2]["mixer"]["rot"].update(dims=10), "rot_dim"),
    (lambda r: r["layers"][2]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda r: r["layers"][4]["mixer"].update(vdim=20), "mixes its values"),
    (lambda r: r["layers"][0]["mlp"].update(kind="dense"), "mlp"),
    (lambda r: r["layers"][0]["mlp"]["router"].update(top=6), "router.top"),
    (lambda r: r["embedding"]["bigram"].pop("mul_prev"), "mul_prev"),
    (lambda r: r.pop("residual_mult"), "residual_mult"),
    (lambda r: r["norm"].pop("eps"), "norm.eps"),
])
def test_what_cannot_be_served_is_refused_with_the_key(edit, message):
    raw = copy.deepcopy(C.MIXED)
    edit(raw)
    with pytest.raises(ConfigError, match=message.replace("[", r"\[").replace("]", r"\]")):
        GimotarConfig.from_dict(raw)


def _parts(raw):
    from tinyserve_llm_b200.parts.base import Runtime, part_class
    rt = Runtime(dtype=torch.float32, device=torch.device("cpu"), ops=None)
    out = []
    for block in spec_of(raw).blocks:
        cls = part_class("mixer", block.mixer)
        out.append(cls(block.mixer, {n: torch.zeros(d.shape) for n, d in cls.declare(block.mixer).items()}, rt))
    return out


def test_cache_layout_keeps_chunks_latents_and_states():
    needs = [(m.kv_need(), int(m.state_bytes())) for m in _parts(C.MIXED)]
    assert needs[0] == (None, 4 * 120 * (3 + 1)) and needs[5] == (None, 4 * 84)          # a ring of `conv` inputs, and none for one tap
    assert needs[1][0] == KVNeed(2, 20, 11, True, 36) and needs[2][0] == KVNeed(1, 52, 0, values=False)
    layout = plan_layout(needs, 16)
    assert not layout.prefix_reuse_possible and layout.state_bytes > 0
    assert plan_layout([(m.kv_need(), int(m.state_bytes())) for m in _parts(C.LATENT)], 16).prefix_reuse_possible


def test_neighbouring_channels_are_reordered_into_halves():
    from tinyserve_llm_b200.parts.latent_attention import evens_then_odds
    assert evens_then_odds(torch.arange(6)[:, None])[:, 0].tolist() == [0, 2, 4, 1, 3, 5]


def test_a_step_carries_the_token_before_each_requests_first_one():
    """Of a new request none, of one that goes on its last committed token; padding requests of a replayed step none."""
    from tinyserve_llm_b200.engine.step import StepEntry, StepRunner, StepShape
    manager = CacheManager(plan_layout([(KVNeed(1, 16), 0)], 16), 8, caching=False)
    runner = StepRunner.__new__(StepRunner)
    runner.manager, runner._pairs = manager, True
    manager.admit("a", [5, 6, 7])
    manager.commit("a", 3)
    manager.extend("a", [8])
    manager.admit("b", [3, 4])
    entries = [StepEntry("a", [8], [0]), StepEntry("b", [3, 4], [])]
    words, offsets, sizes = runner._index_data(entries, None)
    assert words[offsets[-1]:offsets[-1] + 2] == [7, -1] and sizes["seqs"] == 2
    words, offsets, _ = runner._index_data(entries, StepShape(64, 4, 1, 64, True, (1,)))
    assert words[offsets[-1]:offsets[-1] + 4] == [7, -1, -1, -1]
    runner._pairs = False                                        # other models' steps carry no such section
    words, offsets, _ = runner._index_data(entries, None)
    assert len(words) == offsets[-1] + 4 and words[offsets[-1]:] == [0, 0, 0, 0]


def test_a_forked_stream_is_used_in_replayed_steps_only():
    from tinyserve_llm_b200.parts import overlap
    rt = SimpleNamespace(ops=SimpleNamespace(overlap=True), shared={}, device=None)
    assert overlap.fork(rt, SimpleNamespace(replayed=False), "x") is None and overlap.fork(rt, SimpleNamespace(), "x") is None
    rt.ops.overlap = False
    assert overlap.fork(rt, SimpleNamespace(replayed=True), "x") is None
    with overlap.on(None):
        overlap.join(None)


# ---------------------------------------------------------------------------------------------- the plain implementation
def test_the_plain_model_does_not_depend_on_later_tokens_and_reads_far_ones():
    """Causality of every mechanism, and a state that carries the first token to the last."""
    raw = C.MIXED
    tensors = dict(random_tensors(declared_tensors(spec_of(raw)), 5, **C.WEIGHTS))
    C.telling(tensors)
    g = torch.Generator().manual_seed(0)
    ids = torch.randint(0, raw["vocab"], (40,), generator=g).tolist()
    full = plain.forward(raw, tensors, ids)
    torch.testing.assert_close(plain.forward(raw, tensors, ids[:17]), full[:17], atol=1e-10, rtol=1e-10)
    other = list(ids)
    other[0] = (ids[0] + 1) % raw["vocab"]
    assert float((plain.forward(raw, tensors, other)[-1] - full[-1]).abs().max()) > 1e-6


def test_plain_pair_rows_chunks_and_sinks_by_hand():
    assert plain.pair_rows([3, 4, 4], {"buckets": 10, "mul_prev": 7, "mul_cur": 2}) == [10, 29 % 10, 36 % 10]
    assert plain.chunk_mask(5, 2).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    s = torch.tensor([[0.0, 7.0], [1.0, -2.0]], dtype=torch.float64)
    e = torch.exp(torch.tensor([1.0, -2.0, 0.5], dtype=torch.float64))
    p = plain.softmax_with_sink(s, torch.tensor([[True, False], [True, True]]), torch.tensor(0.5, dtype=torch.float64))
    torch.testing.assert_close(p, torch.stack([torch.stack([1 / (1 + e[2]), e[2] * 0]), e[:2] / e.sum()]))


def test_plain_recurrent_unit_by_hand():
    """One channel: r = i = 1/2, softplus(0) = ln 2, so a = 2^-4 and the input enters times sqrt(1 - 2^-8) / 2."""
    w = {n: torch.zeros(1, 1, 1, dtype=torch.float64) for n in ("ra", "ri")}
    w.update({"ra.b": torch.zeros(1, 1, dtype=torch.float64), "ri.b": torch.zeros(1, 1, dtype=torch.float64), "lam": torch.zeros(1, dtype=torch.float64)})
    S = plain.recurrent_unit(torch.tensor([[2.0], [0.0], [4.0]], dtype=torch.float64), w)[:, 0]
    gain = 0.5 * (1 - 2.0 ** -8) ** 0.5
    torch.testing.assert_close(S, torch.tensor([2 * gain, 2 * gain / 16, 2 * gain / 256 + 4 * gain], dtype=torch.float64))
