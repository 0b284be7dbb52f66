"""
The Fuvipel decoder in the engine against the plain implementation of tests/plain_fuvipel.py: each
mechanism alone (with weights or inputs made so that a fault shows), whole prompts, prompts against
token-by-token decoding, portions down to two tokens, unequal requests in one batch against each
alone, pages and state slots that are freed and taken again, far keys, page borders, the first
tokens, long decoding, several sizes (the tensor-core kernels' among them), steps replayed from CUDA
graphs, the replay program and greedy generation through the engine's entry point.
"""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import fuvipel_configs as C
import plain_fuvipel as plain
from test_nipizen import TOL, Engine, _ctx, _i32, _in_steps, _mixer, _runtime, _Slots, ids_of, read_tensors, rows_close

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CONFIGS = {"mixed": C.MIXED, "recurrent": C.RECURRENT, "wide": C.WIDE, "grouped": C.GROUPED}
SEEDS = {"mixed": 711, "recurrent": 722, "wide": 733, "grouped": 744}
PAGE = {"mixed": 16, "recurrent": 16, "wide": 64, "grouped": 64}
F64 = torch.float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from tinyserve_llm_b200.weights.safetensors_io import write_safetensors
    from tinyserve_llm_b200.weights import write_random_model
    out = {}
    for name, raw in CONFIGS.items():
        folder = str(tmp_path_factory.mktemp(f"fuvipel_{name}"))
        write_random_model(folder, raw, SEEDS[name], **C.WEIGHTS)
        tensors = read_tensors(folder)
        C.steady_reads(tensors)
        write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
        out[name] = folder
    return out


_PLAIN = {}


def plain_logits(folder, ids):
    key = (folder, tuple(ids))
    if key not in _PLAIN:
        with open(os.path.join(folder, "config.json")) as f:
            raw = json.load(f)
        _PLAIN[key] = plain.forward(raw, read_tensors(folder), ids)
    return _PLAIN[key]


def close(got, want, dtype):
    """
    float32: every position to rounding.  bfloat16: the error's root mean square against the logits' own spread, in the
    median and in the bulk; one position in a hundred (at least one) may be far off (a read-out that nearly cancels).
    """
    if dtype == "float32":
        torch.testing.assert_close(got, want, atol=3e-4, rtol=1e-4)
    else:
        err = (got - want).pow(2).mean(-1).sqrt() / want.std()
        far_off = float((err > 0.12).double().mean())
        assert int((err > 0.4).sum()) <= max(1, err.numel() // 100) and far_off <= 0.04 and float(err.median()) < 0.05, \
            f"relative error: {far_off:.3f} of the positions over 0.12, worst {float(err.max()):.3f} at {int(err.argmax())}, " \
            f"median {float(err.median()):.3f}"


# ---------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_equals_the_plain_model(folders, name, dtype):
    ids = ids_of(CONFIGS[name]["vocab"], 83, 1)
    got = Engine(folders[name], dtype, page=PAGE[name]).run("a", ids, [len(ids)])
    close(got, plain_logits(folders[name], ids), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_then_token_by_token_and_portions_of_many_sizes(folders, name, dtype):
    """The same logits whether the tokens come at once, one by one after a head, or in portions down to two tokens."""
    ids = ids_of(CONFIGS[name]["vocab"], 120, 2)
    want = plain_logits(folders[name], ids)
    page = PAGE[name]
    decoded = Engine(folders[name], dtype, page=page).run("a", ids, [30] + [1] * 90)
    close(decoded, want, dtype)
    portions = Engine(folders[name], dtype, page=page).run("a", ids, [2, 3, 17, 2, 16, 5, 31, 1, 1, 2])   # shorter than the convolution too
    close(portions, want, dtype)
    one_by_one = Engine(folders[name], dtype, page=page).run("a", ids[:40], [1])      # the first tokens, alone
    close(one_by_one, want[:40], dtype)
    if dtype == "float32":                                                           # the cut changes nothing beyond rounding
        torch.testing.assert_close(decoded, portions, atol=5e-5, rtol=1e-5)


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_batch_and_reused_pages_and_slots(folders, dtype, graphs):
    """
    Five requests through three state slots and a pool that holds less than their sum: portions of
    some beside single tokens of others, requests that sit a step out, ended requests whose pages
    and slots the next ones take (a matrix, a previous row or a convolution's inputs that are not zeroed, or
    a page read through a stale table, show).  With `graphs`, every step is replayed from a CUDA
    graph from its first sighting on.
    """
    name = "mixed"
    vocab = CONFIGS[name]["vocab"]
    reqs = {k: ids_of(vocab, n, 10 + i) for i, (k, n) in enumerate((("a", 70), ("b", 33), ("c", 9), ("d", 58), ("e", 41)))}
    eng = Engine(folders[name], dtype, page=16, pages=12, slots=3, cuda_graphs=graphs)
    eng.step([("a", reqs["a"][:40]), ("b", reqs["b"][:2])])
    eng.step([("a", reqs["a"][40:41]), ("b", reqs["b"][2:19]), ("c", reqs["c"][:9])], end=["c"])
    eng.step([("b", reqs["b"][19:20])])                                             # a sits this one out
    eng.step([("d", reqs["d"][:3]), ("a", reqs["a"][41:70]), ("b", reqs["b"][20:33])], end=["a", "b"])   # d takes c's slot
    eng.step([("d", reqs["d"][3:35]), ("e", reqs["e"][:1])])
    eng.step([("e", reqs["e"][1:2]), ("d", reqs["d"][35:36])])
    for i in range(36, 58):
        both = [("d", reqs["d"][i:i + 1])]
        j = 2 + (i - 36)
        if j < 41:
            both.append(("e", reqs["e"][j:j + 1]))
        eng.step(both, end=["d"] if i == 57 else [])
    eng.step([("e", reqs["e"][24:41])], end=["e"])
    assert eng.manager.stats().pages_in_use == 0 and eng.manager.free_state_slots() == 3
    if graphs:
        assert eng.runner.graph_replays > 20
    for k, ids in reqs.items():
        close(eng.logits(k), plain_logits(folders[name], ids), dtype)
        alone = Engine(folders[name], dtype, page=16, pages=12, slots=3).run(k, ids, [len(ids)])
        if dtype == "float32":
            torch.testing.assert_close(eng.logits(k), alone, atol=5e-5, rtol=1e-5)


def test_tensor_core_attention_also_from_a_graph(folders):
    """
    Pages of 64 tokens and heads of 64 channels: the attention with its sink runs on the tensor-core kernels, prompt
    portions and decoded tokens.  Same logits.
    """
    name, dtype = "wide", "bfloat16"
    ids = ids_of(CONFIGS[name]["vocab"], 200, 7)
    eng = Engine(folders[name], dtype, page=64, pages=8, cuda_graphs=True)
    ops = eng.model.rt.ops
    before = dict(ops.calls)
    got = eng.run("a", ids, [70, 64, 2, 44, 1, 1, 18], last_only=True)
    for kernel in ("ts_paged_attention_bf16_masked", "ts_prefill_attention_tcgen05_masked"):
        assert ops.calls.get(kernel, 0) > before.get(kernel, 0)
    assert eng.runner.graph_replays >= 3
    close(got, plain_logits(folders[name], ids)[[69, 133, 135, 179, 180, 181, 199]], dtype)


def test_long_decoding_keeps_its_state(folders):
    """260 tokens one by one after a short head, over several pages."""
    name, dtype = "mixed", "float32"
    ids = ids_of(CONFIGS[name]["vocab"], 260, 3)
    got = Engine(folders[name], dtype, page=16, pages=18).run("a", ids, [7] + [1] * 253)
    close(got, plain_logits(folders[name], ids), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_sizes_of_a_real_model(tmp_path, dtype):
    """
    Heads of 128 channels, a width of 1,024: a prompt of 600 tokens in one step, a portion over it, single tokens from
    graphs.
    """
    from tinyserve_llm_b200.weights import write_random_model
    from tinyserve_llm_b200.weights.safetensors_io import write_safetensors
    raw = C.model(1000, 1024, 1e-6, [
        (C.delta(8, 2, 128, 128, 4), None),
        (C.parallel(C.attention(8, 2, 128, 0.08, 128, base=500000.0), C.mixing(8, 128, 64)), C.dense(2048)),
    ])
    folder = str(tmp_path / "model")
    write_random_model(folder, raw, 77, std=0.03, unit_std=0.2)
    tensors = read_tensors(folder)
    C.steady_reads(tensors)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    ids = ids_of(raw["vocab"], 660, 5)
    eng = Engine(folder, dtype, page=64, pages=12, cuda_graphs=True)
    got = eng.run("a", ids, [600, 50, 1, 1, 1, 1, 1, 5])
    assert eng.runner.graph_replays > 0
    close(got, plain_logits(folder, ids), dtype)


# ---------------------------------------------------------------------------------------------- attention alone
def _attention_spec(width, heads, kv_heads, dim, scale, rot, base=300.0, gate=True):
    from tinyserve_llm_b200.config.spec import GatedAttentionSpec, InlineRotarySpec
    return GatedAttentionSpec(hidden_size=width, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, value_dim=dim, scale=scale,
                              qk_norm=True, qk_norm_scope="head", qk_norm_weight=False, qk_norm_eps=1e-5, values="keys", sink=0.0,
                              output_gate=gate, position=InlineRotarySpec(dims=rot, base=base, interleaved=True))


def _plain_attention(heads, kv_heads, dim, scale, rot, base=300.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "scale": scale, "rot": {"dims": rot, "base": base}}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, kv_heads, dim, rot, page", [(4, 2, 24, 16, 16), (3, 1, 64, 64, 64), (5, 5, 12, 4, 16), (6, 2, 128, 96, 64),
                                                              (2, 2, 64, 32, 128)])
def test_sink_attention_alone(dtype, heads, kv_heads, dim, rot, page):
    """
    The attention mixer against the plain one: neighbouring channels rotated over part of a head and over all of it,
    heads normed without a weight, the keys as values, the sink, the output gate; two requests of unequal length fed in
    portions that end inside pages, then token by token.
    """
    width, scale = 64, 4.0 / dim
    mixer, w = _mixer(_attention_spec(width, heads, kv_heads, dim, scale, rot), dtype, 3)
    g = torch.Generator().manual_seed(1)
    lens = [300, 21]
    x_of = [torch.randn(n, width, generator=g).to(dtype) for n in lens]
    want = [plain.sink_attention(x.double(), w, _plain_attention(heads, kv_heads, dim, scale, rot), 1e-5) for x in x_of]
    cuts = [[(0, 17), (0, 2)], [(17, 33), (2, 19)], [(33, 34), (19, 20)], [(34, 290), (20, 21)], *[[(i, i + 1), (21, 21)] for i in range(290, 300)]]
    got = _in_steps(_Slots(mixer, dtype, lens, page=page), x_of, cuts)
    for a, b in zip(got, want):
        rows_close(a, b, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sign", [-1.0, 1.0])
@pytest.mark.parametrize("dim, page", [(20, 16), (64, 64), (128, 64)])
def test_the_sink_takes_the_weight_that_low_scores_leave(dtype, dim, page, sign):
    """
    All inputs point the same way: every score is +-dim * scale = +-5 (positions aside: nothing rotates).  With -5 the sink
    holds most of the weight until hundreds of keys are seen, with +5 next to none; the output is known in closed form,
    n e^s / (1 + n e^s) times the one key, gate 1/2.
    """
    width, n = 32, 280
    spec = _attention_spec(width, 1, 1, dim, 5.0 / dim, 2, base=1.0)

    def edit(t):
        g = torch.Generator().manual_seed(2)
        t["k"] = (torch.randn(dim, width, generator=g) * 0.3).to(t["k"].dtype)
        t["k"][:2] = 0                                # the two channels that rotate hold nothing
        t["q"] = sign * t["k"]
        t["g"] = torch.zeros_like(t["g"])

    mixer, w = _mixer(spec, dtype, 5, edit)
    g = torch.Generator().manual_seed(3)
    x = torch.randn(1, width, generator=g).repeat(n, 1).to(dtype)
    got = _in_steps(_Slots(mixer, dtype, [n], page=page), [x], [[(0, 1)], [(1, 3)], [(3, 200)], [(200, 270)], *[[(i, i + 1)] for i in range(270, n)]])[0]
    seen = torch.arange(1, n + 1, dtype=F64)
    e = torch.exp(torch.tensor(5.0 * sign, dtype=F64))
    weight = seen * e / (1 + seen * e)
    full = (0.5 * (x.double() @ w["k"].T)) @ w["o"].T
    assert (float(weight[0]) < 0.01) == (sign < 0)
    err = (got - weight[:, None] * full).norm(dim=-1) / (weight * full.norm(dim=-1))
    assert float(err.max()) < (2e-4 if dtype == torch.float32 else 0.03), f"worst relative error {float(err.max()):.4f} at {int(err.argmax())}"


@pytest.mark.parametrize("prompt_kernel", ["tcgen05", "mma"])
@pytest.mark.parametrize("dim, page, far", [(24, 16, 63), (64, 64, 63), (64, 64, 64), (128, 64, 127)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_finds_a_far_key_at_a_page_border(monkeypatch, dtype, dim, page, far, prompt_kernel):
    """
    One key, hundreds of positions back at a page's last or first slot, points where every query points (in channels that
    do not rotate) and all others point the other way: the queries return its value, the key as projected, as a prompt
    portion and as single tokens; a query before it finds the sink alone.
    """
    from tinyserve_llm_b200.ops import get_ops
    monkeypatch.setattr(get_ops(), "tcgen05_attention", prompt_kernel == "tcgen05")
    width, n = 32, 400
    spec = _attention_spec(width, 1, 1, dim, 12.0 / dim, 4)

    def edit(t):
        t["q"] = torch.zeros_like(t["q"])
        t["q"][4, 0] = 1.0                                # every query points along channel 4
        t["k"] = torch.zeros_like(t["k"])
        t["k"][4, 1] = 1.0                                # keys along it by their input's channel 1
        t["k"][5, 2] = 1.0                                # and along channel 5 by channel 2: the far key alone has it, as a mark
        t["g"] = torch.zeros_like(t["g"])

    mixer, w = _mixer(spec, dtype, 5, edit)
    x = torch.zeros(n, width)
    x[:, 0], x[:, 1] = 3.0, -1.0
    x[far, 1], x[far, 2] = 8.0, 1.0
    x = x.to(dtype)
    got = _in_steps(_Slots(mixer, dtype, [n], page=page), [x], [[(0, far + 1)], [(far + 1, 390)], *[[(i, i + 1)] for i in range(390, n)]])[0]
    want = plain.sink_attention(x.double(), w, _plain_attention(1, 1, dim, 12.0 / dim, 4), 1e-5)
    rows_close(got[far:], want[far:], dtype)
    mark = 0.5 * torch.stack([w["o"][:, 4] * 8.0 + w["o"][:, 5]]).double()           # the far key's value through gate and output
    assert float((want[far + 1:] - mark).norm(dim=-1).max() / mark.norm()) < 0.01     # the premise
    assert float(got[:far].norm(dim=-1).max()) < 0.01 * float(mark.norm())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dims", [6, 20])
def test_keys_are_stored_rotated_by_neighbours_and_normed_and_values_as_they_are(dtype, dims):
    from tinyserve_llm_b200.config.spec import InlineRotarySpec
    from tinyserve_llm_b200.cache.storage import EntryBinding
    from tinyserve_llm_b200.ops import get_ops
    from tinyserve_llm_b200.parts.base import part_class
    ops, H, G, D, page, start, n = get_ops(), 4, 2, 20, 16, 1000, 9
    spec = InlineRotarySpec(dims=dims, base=50.0, interleaved=True)
    position = part_class("position", spec)(spec, {}, _runtime(dtype))
    g = torch.Generator().manual_seed(1)
    y = (torch.randn(n, (H + G) * D + 5, generator=g) * 3).to(dtype)
    pages = (start + n) // page + 1
    k, v = (torch.zeros(pages, 1, G, page, D, dtype=dtype, device="cuda") for _ in range(2))
    binding = EntryBinding(k, v, G * page * D, 0, page, pages, _i32([list(range(pages))]), pages, True, 0, None, None, G * page * D, 0)
    q = ops.qk_norm_rope_store(y.cuda(), (0, H * D, H * D), None, None, 1e-5, position, _ctx([(start, start + n)]), binding, H, G, D, D,
                               unweighted_norm=True)
    pos = torch.arange(start, start + n)
    rot = {"dims": dims, "base": 50.0}
    yq, yk = y.double()[:, :H * D].view(n, H, D), y.double()[:, H * D:(H + G) * D].view(n, G, D)
    tol = dict(atol=3e-4, rtol=1e-4) if dtype == torch.float32 else dict(atol=0.02, rtol=0.01)
    torch.testing.assert_close(q.cpu().double().view(n, H, D), plain.rms_div(plain.rotate_neighbours(yq, pos, rot), 1e-5), **tol)
    stored = lambda pool: torch.stack([pool[p // page, 0, :, p % page] for p in pos.tolist()]).cpu().double()  # noqa: E731
    torch.testing.assert_close(stored(k), plain.rms_div(plain.rotate_neighbours(yk, pos, rot), 1e-5), **tol)
    assert torch.equal(stored(v), yk)


# ---------------------------------------------------------------------------------------------- delta rule alone
def _delta_spec(width, heads, kv_heads, dim, vdim, taps):
    from tinyserve_llm_b200.config.spec import GatedDeltaRuleSpec
    return GatedDeltaRuleSpec(hidden_size=width, num_heads=heads, num_kv_heads=kv_heads, key_dim=dim, value_dim=vdim, conv_taps=taps,
                              q_scale=dim ** -0.5, out_norm_eps=1e-5, decay_scope="head", gate="silu")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, taps", [(4, 2, 20, 24, 3), (2, 2, 72, 37, 4), (3, 1, 16, 16, 1), (2, 1, 130, 8, 2),
                                                               (6, 2, 64, 64, 4), (2, 1, 128, 128, 4), (1, 1, 256, 40, 3)])
def test_gated_delta_rule_with_one_decay_a_head_alone(dtype, heads, kv_heads, dim, vdim, taps):
    """
    The delta rule against the plain one: two requests in one launch, cut at places that are no multiples of the scan's
    tile and shorter than the convolution, sizes that are no multiples of the kernel's own, decays from nearly one to
    nearly zero, step sizes all over (0, 1), slots that are not in order.
    """
    width = 64

    def edit(t):
        t["A_log"] = torch.linspace(-5.0, 3.0, heads).to(t["A_log"].dtype) if heads > 1 else t["A_log"]
        t["a"] = t["a"] * 6
        t["b"] = t["b"] * 4

    mixer, w = _mixer(_delta_spec(width, heads, kv_heads, dim, vdim, taps), dtype, 7, edit)
    g = torch.Generator().manual_seed(3)
    lens = [131, 26]
    x_of = [torch.randn(n, width, generator=g).to(dtype) for n in lens]
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps}
    want = [plain.gated_delta_rule(x.double(), w, m, 1e-5) for x in x_of]
    cuts = [[(0, 1), (0, 2)], [(1, 2), (2, 3)], [(2, 4), (3, 3)], [(4, 41), (3, 5)], [(41, 42), (5, 26)], [(42, 125), (26, 26)],
            *[[(i, i + 1), (26, 26)] for i in range(125, 131)]]
    got = _in_steps(_Slots(mixer, dtype, lens), x_of, cuts)
    for a, b in zip(got, want):
        rows_close(a, b, dtype)


def test_delta_rule_reads_the_first_token_far_later():
    """With decays close to one the first token's write is still read 200 tokens on: a state lost on the way shows."""
    width, H, D, V = 32, 2, 16, 16

    def edit(t):
        t["A_log"] = torch.full_like(t["A_log"], -9.0)
        t["dt_bias"] = torch.zeros_like(t["dt_bias"])
        t["b"] = torch.zeros_like(t["b"])

    mixer, w = _mixer(_delta_spec(width, H, H, D, V, 2), torch.float32, 9, edit)
    g = torch.Generator().manual_seed(4)
    x = torch.randn(210, width, generator=g)
    x[0] *= 4
    m = {"heads": H, "kv_heads": H, "dim": D, "vdim": V, "conv": 2}
    want = plain.gated_delta_rule(x.double(), w, m, 1e-5)
    other = x.clone()
    other[0] = -other[0]
    assert float((plain.gated_delta_rule(other.double(), w, m, 1e-5)[-1] - want[-1]).abs().max()) > 1e-3      # the premise
    got = _in_steps(_Slots(mixer, torch.float32, [210]), [x], [[(0, 50)], [(50, 203)], *[[(i, i + 1)] for i in range(203, 210)]])[0]
    torch.testing.assert_close(got, want, **TOL[torch.float32])


# ---------------------------------------------------------------------------------------------- time mixing alone
def _mixing_spec(width, heads, dim, rank):
    from tinyserve_llm_b200.config.spec import TimeMixingSpec
    return TimeMixingSpec(hidden_size=width, num_heads=heads, head_dim=dim, decay_rank=rank, out_norm_eps=1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width, heads, dim, rank", [(64, 3, 24, 6), (96, 2, 64, 32), (64, 4, 20, 16), (32, 1, 128, 3), (64, 2, 130, 5),
                                                      (40, 1, 256, 8)])
def test_time_mixing_alone(dtype, width, heads, dim, rank):
    """
    Time mixing against the plain one: two requests in one launch, cut at every kind of place (the previous token's row
    crosses each cut), blends of their own for the five projections, decays from nearly one to nearly zero, a bonus that
    matters, a step of many tokens (the library's products) beside steps of few.
    """
    def edit(t):
        g = torch.Generator().manual_seed(1)
        for s in "rkvgw":
            t[f"mu.{s}"] = torch.rand(width, generator=g).to(t["r"].dtype)
        t["w0"] = torch.linspace(-6.0, 2.0, heads * dim).to(t["w0"].dtype)
        t["w2"] = t["w2"] * 4
        t["u"] = (torch.randn(heads, dim, generator=g) * 2).to(t["u"].dtype)

    mixer, w = _mixer(_mixing_spec(width, heads, dim, rank), dtype, 11, edit)
    g = torch.Generator().manual_seed(5)
    lens = [131, 19]
    x_of = [torch.randn(n, width, generator=g).to(dtype) for n in lens]
    want = [plain.time_mixing(x.double(), w, {"heads": heads, "dim": dim}, 1e-5) for x in x_of]
    cuts = [[(0, 1), (0, 2)], [(1, 3), (2, 2)], [(3, 37), (2, 19)], [(37, 38), (19, 19)], [(38, 125), (19, 19)],
            *[[(i, i + 1), (19, 19)] for i in range(125, 131)]]
    got = _in_steps(_Slots(mixer, dtype, lens), x_of, cuts)
    for a, b in zip(got, want):
        rows_close(a, b, dtype)


def test_time_mixing_weighs_the_current_token_by_its_bonus_and_the_first_token_has_no_predecessor():
    """
    With u = 0 the first token reads an empty state (output zero); with u != 0 it reads its own write alone; the second
    reads the first one's write undecayed, whatever the decay of the second says.
    """
    width, H, D = 32, 2, 16
    g = torch.Generator().manual_seed(6)
    x = torch.randn(2, width, generator=g)
    for bonus in (0.0, 1.5):
        def edit(t):
            t["u"] = torch.full_like(t["u"], bonus)
            t["w0"] = torch.full_like(t["w0"], 3.0)                       # decays of e^-20
        mixer, w = _mixer(_mixing_spec(width, H, D, 4), torch.float32, 13, edit)
        got = _in_steps(_Slots(mixer, torch.float32, [2]), [x], [[(0, 1)], [(1, 2)]])[0]
        torch.testing.assert_close(got, plain.time_mixing(x.double(), w, {"heads": H, "dim": D}, 1e-5), **TOL[torch.float32])
        assert (float(got[0].abs().max()) < 1e-6) == (bonus == 0.0) and float(got[1].abs().max()) > 1e-3


def test_time_mixing_reads_the_first_token_far_later():
    width, H, D = 32, 2, 16

    def edit(t):
        t["w0"] = torch.full_like(t["w0"], -9.0)
        t["w2"] = torch.zeros_like(t["w2"])

    mixer, w = _mixer(_mixing_spec(width, H, D, 4), torch.float32, 15, edit)
    g = torch.Generator().manual_seed(7)
    x = torch.randn(210, width, generator=g)
    x[0] *= 8
    m = {"heads": H, "dim": D}
    want = plain.time_mixing(x.double(), w, m, 1e-5)
    other = x.clone()
    other[0] = 0
    assert float((plain.time_mixing(other.double(), w, m, 1e-5)[-1] - want[-1]).abs().max()) > 1e-3      # the premise
    got = _in_steps(_Slots(mixer, torch.float32, [210]), [x], [[(0, 50)], [(50, 203)], *[[(i, i + 1)] for i in range(203, 210)]])[0]
    torch.testing.assert_close(got, want, **TOL[torch.float32])


# ---------------------------------------------------------------------------------------------- tiles of tokens
@pytest.mark.parametrize("kind", ["delta", "mixing"])
@pytest.mark.parametrize("tiles", [True, False])
def test_portions_by_tiles_and_token_by_token_agree_with_the_plain_recurrence(monkeypatch, kind, tiles):
    """
    Three requests in one launch: a long portion (several tiles, the last one cut short), one of exactly a tile, and a
    single token beside them, then portions of two tokens and up that start inside what would be a tile; decays near one, so
    that sums over hundreds of tokens show, and a head whose decays are zero in float32.
    """
    from tinyserve_llm_b200.ops import get_ops
    monkeypatch.setattr(get_ops(), "recurrence_tiles", tiles)
    width, H, D = 48, 3, 72
    if kind == "delta":
        spec, m = _delta_spec(width, H, 1, D, 40, 3), {"heads": H, "kv_heads": 1, "dim": D, "vdim": 40, "conv": 3}
        want_of = lambda x, w: plain.gated_delta_rule(x, w, m, 1e-5)  # noqa: E731

        def edit(t):
            t["A_log"] = torch.tensor([-8.0, -2.0, 6.0]).to(t["A_log"].dtype)
            t["q"] = t["k"] + t["q"] / 4
            t["q.conv"] = t["k.conv"]
    else:
        spec, m = _mixing_spec(width, H, D, 4), {"heads": H, "dim": D}
        want_of = lambda x, w: plain.time_mixing(x, w, m, 1e-5)  # noqa: E731

        def edit(t):
            t["w0"] = torch.tensor([-8.0, -2.0, 6.0]).repeat_interleave(D).to(t["w0"].dtype)
            t["r"] = t["k"] + t["r"] / 4
            t["u"] = t["u"] + 1

    mixer, w = _mixer(spec, torch.float32, 31, edit)
    g = torch.Generator().manual_seed(8)
    lens = [420, 60, 45]
    x_of = [torch.randn(n, width, generator=g) for n in lens]
    cuts = [[(0, 333), (0, 16), (0, 1)], [(333, 335), (16, 17), (1, 18)], [(335, 418), (17, 49), (18, 45)], [(418, 420), (49, 60), (45, 45)]]
    before = dict(get_ops().calls)
    got = _in_steps(_Slots(mixer, torch.float32, lens), x_of, cuts)
    name = "ts_delta_tiles" if kind == "delta" else "ts_mix_tiles"
    assert (get_ops().calls.get(name, 0) > before.get(name, 0)) == tiles
    for a, x in zip(got, x_of):
        want = want_of(x.double(), w)
        err = (a - want).norm(dim=-1) / want.norm(dim=-1)
        assert float(err.max()) < 2e-4 and float(err.median()) < 5e-6, f"worst {float(err.max()):.2e}, median {float(err.median()):.2e}"


# ---------------------------------------------------------------------------------------------- both halves, norms, products
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layer", [0, 3])
def test_parallel_mixer_averages_its_normed_halves(dtype, layer):
    """Halves of unequal inner width (0) and of equal width (3), whose output projections run as one grouped product."""
    from tinyserve_llm_b200.config.fuvipel import FuvipelConfig
    raw = C.MIXED
    mixer, w = _mixer(FuvipelConfig.from_dict(raw).mixer_spec(layer), dtype, 13)
    assert (mixer.grouped_out is not None) == (layer == 3)
    g = torch.Generator().manual_seed(6)
    lens = [80, 7]
    x_of = [torch.randn(n, raw["width"], generator=g).to(dtype) for n in lens]
    want = [plain.parallel_mixer(x.double(), w, raw["layers"][layer]["mixer"], 1e-5) for x in x_of]
    got = _in_steps(_Slots(mixer, dtype, lens), x_of, [[(0, 15), (0, 7)], [(15, 16), (7, 7)], [(16, 80), (7, 7)]])
    for a, b in zip(got, want):
        rows_close(a, b, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [100, 1056])
def test_stream_kernel_closes_one_branch_or_a_pair_and_copies_the_stream(dtype, width):
    from tinyserve_llm_b200.ops import get_ops
    ops = get_ops()
    g = torch.Generator().manual_seed(3)
    T, eps = 7, 1e-3
    stream = torch.randn(T, width, generator=g) * 3
    a, b = ((torch.randn(T, width, generator=g) * s).to(dtype) for s in (0.05, 9.0))
    w1, w2, wc, wo = (1 + torch.randn(width, generator=g) * 0.3 for _ in range(4))
    d = lambda t: t.double()  # noqa: E731
    tol = dict(atol=2e-5, rtol=2e-5) if dtype == torch.float32 else dict(atol=0.03, rtol=0.01)
    single = d(stream) + plain.rms_div(d(a), eps) * d(wc)
    pair_sum = 0.5 * plain.rms_div(d(a), eps) * d(w1) + 0.25 * plain.rms_div(d(b), eps) * d(w2)
    both = d(stream) + plain.rms_div(pair_sum, eps) * d(wc)
    pair = (b.cuda(), w1.cuda(), w2.cuda(), 0.5, 0.25)
    for p, want in ((None, single), (pair, both)):
        s = stream.cuda()
        out = ops.stream_norm(a.cuda(), wc.cuda(), s, None, eps, dtype, copy_out=True, pair=p)
        torch.testing.assert_close(s.cpu().double(), want, atol=2e-5, rtol=2e-5)         # the stream stays float32 in both dtypes
        assert torch.equal(out.cpu(), s.cpu().to(dtype))
        s = stream.cuda()
        normed = ops.stream_norm(a.cuda(), wc.cuda(), s, wo.cuda(), eps, dtype, pair=p)
        torch.testing.assert_close(normed.cpu().double(), plain.rms_div(want, eps) * d(wo), **tol)
        before = s.clone()
        s2 = stream.cuda()
        picked = ops.stream_norm(a.cuda(), wc.cuda(), s2, wo.cuda(), eps, dtype, rows=_i32([5, 0]), pair=p)
        assert torch.equal(s2.cpu(), stream) and torch.equal(before, s)                   # with rows, the stream is read only
        torch.testing.assert_close(picked.cpu().double(), (plain.rms_div(want, eps) * d(wo))[[5, 0]], **tol)
    s = stream.cuda()
    ops.stream_norm(a.cuda(), None, s, wo.cuda(), eps, dtype, plain_add=True, pair=pair)
    torch.testing.assert_close(s.cpu().double(), d(stream) + pair_sum, atol=2e-5, rtol=2e-5)
    torch.testing.assert_close(ops.normed_sum(a.cuda(), pair, eps).cpu().double(), pair_sum, **tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_embedding_rows_start_the_stream_and_are_read_as_they_are(dtype):
    from tinyserve_llm_b200.ops import get_ops
    table = torch.randn(11, 36).to(dtype)
    ids = _i32([3, 10, 0, 3])
    stream = torch.empty(4, 36, device="cuda")
    out = get_ops().stream_norm(None, None, stream, None, 1e-6, dtype, table=table.cuda(), ids=ids, copy_out=True)
    assert torch.equal(out.cpu(), table[[3, 10, 0, 3]]) and torch.equal(stream.cpu(), table[[3, 10, 0, 3]].float())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("groups, rows, n, k", [(4, 1, 64, 96), (4, 7, 48, 64), (2, 32, 1040, 128), (5, 33, 32, 64), (3, 5, 20, 64), (4, 6, 32, 20)])
def test_grouped_products_each_read_an_input_of_their_own(dtype, groups, rows, n, k):
    from tinyserve_llm_b200.ops import get_ops
    g = torch.Generator().manual_seed(9)
    x, w = (torch.randn(groups, rows, k, generator=g).to(dtype), torch.randn(groups, n, k, generator=g).to(dtype))
    want = x.double() @ w.double().transpose(1, 2)
    got = get_ops().linear_groups(x.cuda(), w.cuda())
    assert got.dtype == dtype
    tol = dict(atol=1e-4, rtol=1e-4) if dtype == torch.float32 else dict(atol=0.1, rtol=0.01)
    torch.testing.assert_close(got.cpu().double(), want, **tol)
    got = get_ops().linear_groups(x.cuda(), w.cuda(), out_dtype=torch.float32)
    torch.testing.assert_close(got.cpu().double(), want, atol=1e-3, rtol=1e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows", [3, 40])
def test_product_with_tanh(dtype, rows):
    from tinyserve_llm_b200.ops import get_ops
    g = torch.Generator().manual_seed(10)
    x, w = torch.randn(rows, 64, generator=g).to(dtype), (torch.randn(24, 64, generator=g) * 0.2).to(dtype)
    got = get_ops().linear_unary(x.cuda(), w.cuda(), "tanh").cpu().double()
    tol = dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=0.02, rtol=0.01)
    torch.testing.assert_close(got, torch.tanh(x.double() @ w.double().T), **tol)


def test_dense_feed_forward_with_squared_relu():
    from tinyserve_llm_b200.config.spec import PlainMLPSpec
    from tinyserve_llm_b200.parts.base import part_class
    from tinyserve_llm_b200.weights import random_tensors
    spec = PlainMLPSpec(hidden_size=64, intermediate_size=104, activation="relu2")
    cls = part_class("feed_forward", spec)
    tensors = dict(random_tensors(cls.declare(spec), 3, std=0.2))
    for dtype in (torch.float32, torch.bfloat16):
        part = cls(spec, {k: v.cuda() for k, v in tensors.items()}, _runtime(dtype))
        for rows in (5, 90):
            x = torch.randn(rows, 64, generator=torch.Generator().manual_seed(rows)).to(dtype)
            want = plain.dense(x.double(), {k: v.double() for k, v in tensors.items()})
            rows_close(part.forward(x.cuda(), None).cpu().double(), want, dtype)


# ---------------------------------------------------------------------------------------------- entry points
def test_replay_program_on_a_model_folder(folders, tmp_path):
    """bin/trace_run on a Fuvipel folder: portions, a decoded tail, two requests side by side, a reused slot."""
    name = "wide"
    vocab = CONFIGS[name]["vocab"]
    a, b = ids_of(vocab, 90, 21), ids_of(vocab, 70, 22)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:64], "want": [0, 63]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[64:66], "want": [1]}, {"id": "b", "tokens": b[:69], "want": [68]}], "end": []},
        {"step": 2, "entries": [{"id": "b", "tokens": b[69:], "want": [0]}], "end": ["b"]},
        {"step": 3, "entries": [{"id": "a", "tokens": a[66:], "want": [23]}], "end": ["a"]},
        {"step": 4, "entries": [{"id": "c", "tokens": b, "want": [69]}], "end": ["c"]},
    ]
    rows = {0: [("a", 0), ("a", 63)], 1: [("a", 65), ("b", 68)], 2: [("b", 69)], 3: [("a", 89)], 4: [("b", 69)]}
    want = {"a": plain_logits(folders[name], a), "b": plain_logits(folders[name], b)}
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folders[name], "--dtype", dtype,
                               "--out", str(out), "--max-tokens", "256", "--max-requests", "2"],
                              input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [line for line in proc.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(5)]
        got, expected = [], []
        for step, places in rows.items():
            got.append(torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(places), vocab)).double())
            expected += [want[r][p] for r, p in places]
        close(torch.cat(got), torch.stack(expected), dtype)


@pytest.mark.parametrize("name", ["mixed", "recurrent"])
def test_greedy_generation_through_the_entry_point(folders, name):
    """LLM.generate with the scheduler, prompt portions, CUDA graphs and running ahead: the plain model's greedy tokens."""
    from tinyserve_llm_b200 import LLM, CacheConfig, SamplingParams, SchedulerConfig
    raw = CONFIGS[name]
    tensors = read_tensors(folders[name])
    prompts = [ids_of(raw["vocab"], n, 30 + n) for n in (3, 41, 18, 77, 1)]
    new = 12
    want = []
    for p in prompts:
        ids = list(p)
        for _ in range(new):
            ids.append(int(plain.forward(raw, tensors, ids)[-1].argmax()))
        want.append(ids[len(p):])
    llm = LLM(folders[name], SchedulerConfig(max_model_len=128, max_num_seqs=3, max_num_batched_tokens=48, prefill_chunk=20),
              CacheConfig(block_size=16), dtype="float32", num_blocks=24, seed=0)
    done = llm.generate(prompts, SamplingParams(max_tokens=new, temperature=0.0, ignore_eos=True))
    assert [c.token_ids[0] for c in done] == want
