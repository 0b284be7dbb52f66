"""
The Gimotar decoder in the engine against the plain implementation of tests/plain_gimotar.py: each
mechanism alone (with weights or inputs made so that a fault shows), whole prompts, prompts against
token-by-token decoding, portions down to two tokens, unequal requests in one batch against each
alone, pages and state slots that are freed and taken again, keys far away, at page borders and just
inside and just outside a chunk, the first tokens, long decoding, several sizes (the tensor-core kernels'
among them), steps replayed from CUDA graphs, cached prefixes, the replay program and greedy generation
through the engine's entry point.
"""

import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import gimotar_configs as C
import plain_gimotar as plain
from test_nipizen import TOL, Engine, _ctx, _i32, _in_steps, _mixer, _runtime, _Slots, ids_of, read_tensors, rows_close

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CONFIGS = {"mixed": C.MIXED, "latent": C.LATENT, "recurrent": C.RECURRENT, "wide": C.WIDE, "grouped": C.GROUPED}
SEEDS = {"mixed": 811, "latent": 822, "recurrent": 833, "wide": 844, "grouped": 855}
PAGE = {"mixed": 16, "latent": 16, "recurrent": 16, "wide": 64, "grouped": 64}
F64 = torch.float64


def _write(folder, raw, seed, weights):
    from tinyserve_llm_b200.weights import write_random_model
    from tinyserve_llm_b200.weights.safetensors_io import write_safetensors
    write_random_model(folder, raw, seed, **weights)
    tensors = read_tensors(folder)
    C.telling(tensors)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """
    A folder for the float32 comparisons (routing included) and one for the bfloat16 comparisons, in which every token
    uses all experts of a layer: with fewer, a token whose router scores at the edge of the chosen set lie closer than
    bfloat16's rounding of its activations takes another expert than the float64 model.  Routing in bfloat16 is
    compared by the test of the routed feed-forward alone.
    """
    out = {}
    for name, raw in CONFIGS.items():
        every = copy.deepcopy(raw)
        for layer in every["layers"]:
            if layer["mlp"] is not None:
                layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
        for dtype, cfg in (("float32", raw), ("bfloat16", every)):
            folder = str(tmp_path_factory.mktemp(f"gimotar_{name}_{dtype}"))
            _write(folder, cfg, SEEDS[name], C.WEIGHTS)
            out[name, dtype] = folder
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
    """float32: every position to rounding.  bfloat16: the error's root mean square against the logits' own spread."""
    if dtype == "float32":
        torch.testing.assert_close(got, want, atol=5e-4, rtol=2e-4)
    else:
        err = (got - want).pow(2).mean(-1).sqrt() / want.std()
        assert float(err.max()) < 0.2 and float(err.median()) < 0.05, \
            f"relative error: worst {float(err.max()):.3f} at {int(err.argmax())}, median {float(err.median()):.3f}"


# ---------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_equals_the_plain_model(folders, name, dtype):
    ids = ids_of(CONFIGS[name]["vocab"], 300 if PAGE[name] == 64 else 150, 1)
    got = Engine(folders[name, dtype], dtype, page=PAGE[name]).run("a", ids, [len(ids)])
    close(got, plain_logits(folders[name, dtype], ids), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_then_token_by_token_and_portions_of_many_sizes(folders, name, dtype):
    """The same logits whether the tokens come at once, one by one after a head, or in portions down to two tokens."""
    n = 230 if PAGE[name] == 64 else 150
    ids = ids_of(CONFIGS[name]["vocab"], n, 2)
    folder = folders[name, dtype]
    want = plain_logits(folder, ids)
    page = PAGE[name]
    decoded = Engine(folder, dtype, page=page).run("a", ids, [30] + [1] * (n - 30))             # chunks pass over decoded tokens
    close(decoded, want, dtype)
    portions = Engine(folder, dtype, page=page).run("a", ids, [2, 3, 17, 2, 16, 5, 31, 1, 1, 2, 64, 3])   # shorter than a convolution too
    close(portions, want, dtype)
    one_by_one = Engine(folder, dtype, page=page).run("a", ids[:40], [1])                       # the first tokens, alone
    close(one_by_one, want[:40], dtype)
    if dtype == "float32":                                                                      # the cut changes nothing beyond rounding
        torch.testing.assert_close(decoded, portions, atol=1e-4, rtol=2e-5)


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_requests_in_one_batch_and_reused_pages_and_slots(folders, name, dtype, graphs):
    """
    Five requests through three state slots and a pool that holds less than their sum: portions of some beside
    single tokens of others, requests that sit a step out, ended requests whose pages and slots the next ones take
    (a state or a convolution's inputs that are not zeroed, a page read through a stale table, the token before
    taken from another request, show).  With `graphs`, every step is replayed from a CUDA graph from its first
    sighting on.
    """
    vocab, page = CONFIGS[name]["vocab"], PAGE[name]
    k = page // 16
    folder = folders[name, dtype]
    reqs = {key: ids_of(vocab, n, 10 + i) for i, (key, n) in enumerate((("a", 70 * k), ("b", 33 * k), ("c", 9), ("d", 58 * k), ("e", 41 * k)))}
    a, b, c, d, e = (reqs[x] for x in "abcde")
    eng = Engine(folder, dtype, page=page, pages=12, slots=3, cuda_graphs=graphs)
    eng.step([("a", a[:40 * k]), ("b", b[:2])])
    eng.step([("a", a[40 * k:40 * k + 1]), ("b", b[2:19 * k]), ("c", c[:9])], end=["c"])
    eng.step([("b", b[19 * k:19 * k + 1])])                                          # a sits this one out
    eng.step([("d", d[:3]), ("a", a[40 * k + 1:]), ("b", b[19 * k + 1:])], end=["a", "b"])   # d takes c's slot
    eng.step([("d", d[3:35 * k]), ("e", e[:1])])
    eng.step([("e", e[1:2]), ("d", d[35 * k:35 * k + 1])])
    for i in range(20):
        eng.step([("d", d[35 * k + 1 + i:35 * k + 2 + i]), ("e", e[2 + i:3 + i])])
    eng.step([("e", e[22:]), ("d", d[35 * k + 21:])], end=["d", "e"])
    assert eng.manager.stats().pages_in_use == 0 and eng.manager.free_state_slots() == 3
    if graphs:
        assert eng.runner.graph_replays > 20
    for key, ids in reqs.items():
        close(eng.logits(key), plain_logits(folder, ids), dtype)
        if dtype == "float32":
            alone = Engine(folder, dtype, page=page, pages=12, slots=3).run(key, ids, [len(ids)])
            torch.testing.assert_close(eng.logits(key), alone, atol=1e-4, rtol=2e-5)


def test_the_kernels_for_large_sizes_run_also_from_a_graph(folders):
    """
    Pages of 64 tokens, heads of 64 channels, bfloat16: the chunked attention runs on the tensor-core kernels, the latent
    one on its own, the recurrence's decode steps in one kernel and its portions in stretches, many (token, expert)
    pairs on the library's grouped product.  Same logits.
    """
    name, dtype = "wide", "bfloat16"
    ids = ids_of(CONFIGS[name]["vocab"], 290, 7)
    eng = Engine(folders[name, dtype], dtype, page=64, pages=8, cuda_graphs=True)
    ops = eng.model.rt.ops
    old, ops.grouped_mm_min_pairs = ops.grouped_mm_min_pairs, 64
    try:
        before = dict(ops.calls)
        got = eng.run("a", ids, [70, 154, 2, 44, 1, 1, 18], last_only=True)
    finally:
        ops.grouped_mm_min_pairs = old
    for kernel in ("ts_paged_attention_bf16_masked", "ts_prefill_attention_tcgen05_masked", "ts_latent_attention", "ts_lru_decode",
                   "ts_lru_scan", "library_grouped_mm"):
        assert ops.calls.get(kernel, 0) > before.get(kernel, 0), kernel
    assert eng.runner.graph_replays >= 3
    close(got, plain_logits(folders[name, dtype], ids)[[69, 223, 225, 269, 270, 271, 289]], dtype)


@pytest.mark.parametrize("name", ["mixed", "recurrent"])
def test_long_decoding_keeps_its_state(folders, name):
    """260 tokens one by one after a short head, over several pages and chunks."""
    dtype = "float32"
    ids = ids_of(CONFIGS[name]["vocab"], 260, 3)
    got = Engine(folders[name, dtype], dtype, page=16, pages=18).run("a", ids, [7] + [1] * 253)
    close(got, plain_logits(folders[name, dtype], ids), dtype)


def test_many_requests_decode_in_one_step(folders):
    """Nine and then seventy requests of unequal lengths in one decode step: more rows than the kernels' tiles of tokens."""
    name, dtype = "recurrent", "bfloat16"
    folder = folders[name, dtype]
    for count in (9, 70):
        reqs = {f"r{i}": ids_of(CONFIGS[name]["vocab"], 3 + i % 5, 50 + i) for i in range(count)}
        eng = Engine(folder, dtype, page=16, pages=4, slots=count)
        eng.step([(k, ids[:-1]) for k, ids in reqs.items()])
        eng.step([(k, ids[-1:]) for k, ids in reqs.items()])
        close(torch.cat([eng.logits(k) for k in reqs]), torch.cat([plain_logits(folder, ids) for ids in reqs.values()]), dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_sizes_of_a_real_model(tmp_path, dtype):
    """Heads of 128 channels, a width of 1,024, parts of 256 channels: a long prompt in one step, a portion over it, single tokens from graphs."""
    raw = C.model(1000, 1024, 1e-6, 0.5, 4.0, (997, 31, 7), [
        (C.attention(8, 2, 128, 128, 0.08, 256, 64, base=500000.0), C.moe(4, 4, 512, 1024)),
        (C.rglru(2048, 8, 4), None),
        (C.latent(8, 128, 64, 128, 512, 0.07, base=10000.0, yarn=(4.0, 256, 32.0, 1.0)), None),
        (C.attention(8, 2, 128, 128, 0.08, 256, 64, base=500000.0), None),
    ])
    folder = str(tmp_path / "model")
    _write(folder, raw, 77, dict(std=0.03, unit_std=0.2))
    ids = ids_of(raw["vocab"], 660, 5)
    eng = Engine(folder, dtype, page=64, pages=12, cuda_graphs=True)
    got = eng.run("a", ids, [600, 50, 1, 1, 1, 1, 1, 5])
    assert eng.runner.graph_replays > 0
    close(got, plain_logits(folder, ids), dtype)


# ---------------------------------------------------------------------------------------------- recurrence alone
def _lru(width, channels, blocks, taps, dtype, seed, edit=None):
    from tinyserve_llm_b200.config.spec import GatedLRUSpec
    spec = GatedLRUSpec(hidden_size=width, width=channels, blocks=blocks, conv_taps=taps, decay_rate=8.0)

    def prepare(t):
        C.telling(t)
        if edit:
            edit(t)
    return _mixer(spec, dtype, seed, prepare)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("channels, blocks, taps", [(96, 4, 4), (60, 5, 3), (35, 7, 2), (64, 64, 1), (264, 1, 4), (51, 3, 11),
                                                    (1040, 2, 4), (640, 2, 8), (320, 8, 2)])
def test_gated_linear_recurrent_unit_alone(dtype, channels, blocks, taps):
    """
    Two requests in one launch, cut at places shorter than the convolution and longer than the scan's stretches, sizes
    that are no multiples of the kernels' own, one part and as many as channels, slots that are not in order; then
    single tokens, of both requests and of one.
    """
    width = 64
    mixer, w = _lru(width, channels, blocks, taps, dtype, 7)
    g = torch.Generator().manual_seed(3)
    lens = [240, 47]
    x_of = [torch.randn(n, width, generator=g).to(dtype) for n in lens]
    want = [plain.rglru(x.double(), w, {}) for x in x_of]
    cuts = [[(0, 1), (0, 2)], [(1, 2), (2, 3)], [(2, 4), (3, 3)], [(4, 41), (3, 5)], [(41, 42), (5, 42)], [(42, 171), (42, 43)],
            *[[(i, i + 1), (i - 128, i - 127)] for i in range(171, 175)], [(175, 239), (47, 47)], [(239, 240), (47, 47)]]
    got = _in_steps(_Slots(mixer, dtype, lens), x_of, cuts)
    for a, b in zip(got, want):
        rows_close(a, b, dtype)


@pytest.mark.parametrize("fused", [True, False])
@pytest.mark.parametrize("channels, blocks, taps", [(96, 4, 4), (512, 2, 3), (64, 8, 1), (1024, 2, 5)])
def test_decode_kernel_and_the_kernels_of_portions_carry_the_same_state(monkeypatch, fused, channels, blocks, taps):
    """bfloat16 single tokens by the one-kernel form and by the others, in turn with portions, over the ring's every phase."""
    from tinyserve_llm_b200.ops import get_ops
    ops = get_ops()
    monkeypatch.setattr(ops, "lru_fused_decode", fused)
    width, dtype = 32, torch.bfloat16
    mixer, w = _lru(width, channels, blocks, taps, dtype, 17)
    g = torch.Generator().manual_seed(4)
    lens = [60, 41]
    x_of = [torch.randn(n, width, generator=g).to(dtype) for n in lens]
    cuts = [[(0, 1), (0, 0)], [(1, 2), (0, 3)], *[[(i, i + 1), (i + 1, i + 2)] for i in range(2, 20)], [(20, 23), (21, 22)],
            *[[(i, i + 1), (i - 1, i)] for i in range(23, 42)], [(42, 60), (41, 41)]]
    before = ops.calls.get("ts_lru_decode", 0)
    got = _in_steps(_Slots(mixer, dtype, lens), x_of, cuts)
    assert (ops.calls.get("ts_lru_decode", 0) > before) == fused
    for a, x in zip(got, x_of):
        rows_close(a, plain.rglru(x.double(), w, {}), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_recurrence_reads_the_first_token_far_later(dtype):
    """With decays close to one the first token is still read 300 tokens on: a state lost on the way, or a stretch left out, shows."""
    width, channels = 32, 64

    def edit(t):
        t["lam"] = torch.full_like(t["lam"], -11.0)

    mixer, w = _lru(width, channels, 4, 3, dtype, 9, edit)
    g = torch.Generator().manual_seed(4)
    x = torch.randn(310, width, generator=g) * 0.3
    x[0] *= 60
    x = x.to(dtype)
    want = plain.rglru(x.double(), w, {})
    other = x.clone()
    other[0] = 0
    far = (plain.rglru(other.double(), w, {})[-1] - want[-1]).norm() / want[-1].norm()
    assert float(far) > 0.3                                                                     # the premise
    got = _in_steps(_Slots(mixer, dtype, [310]), [x], [[(0, 50)], [(50, 303)], *[[(i, i + 1)] for i in range(303, 310)]])[0]
    rows_close(got, want, dtype)


def test_the_first_token_enters_the_state_as_any_other():
    """S_0 = sqrt(1 - a^2) i u with the token's own decay, and zeros stand before the start in the convolution."""
    width, channels, taps = 16, 24, 4
    mixer, w = _lru(width, channels, 3, taps, torch.float32, 19)
    x = torch.randn(1, width, generator=torch.Generator().manual_seed(5))
    h = x.double()
    u = w["conv.b"] + w["conv"][:, -1] * (h @ w["x"].T + w["x.b"])
    r = torch.sigmoid(plain.block_product(u, w["ra"], w["ra.b"]))
    i = torch.sigmoid(plain.block_product(u, w["ri"], w["ri.b"]))
    a = torch.exp(-8.0 * r * torch.nn.functional.softplus(w["lam"]))
    want = (torch.sqrt(1 - a * a) * i * u * plain.gelu_tanh(h @ w["y"].T + w["y.b"])) @ w["o"].T
    got = _in_steps(_Slots(mixer, torch.float32, [1]), [x], [[(0, 1)]])[0]
    torch.testing.assert_close(got, want, **TOL[torch.float32])


# ---------------------------------------------------------------------------------------------- latent attention alone
def _latent(width, heads, dim, rot, vdim, rank, scale, yarn, dtype, seed, edit=None):
    from tinyserve_llm_b200.config.spec import InlineRotarySpec, LatentAttentionSpec, YarnScaling
    spec = LatentAttentionSpec(hidden_size=width, num_heads=heads, head_dim=dim, rot_dim=rot, value_dim=vdim, q_rank=0, kv_rank=rank,
                               scale=scale, norm_eps=1e-5, output_gate=True, sink=True,
                               position=InlineRotarySpec(dims=rot, base=200.0, interleaved=True, yarn=YarnScaling(*yarn) if yarn else None))
    m = C.latent(heads, dim, rot, vdim, rank, scale, base=200.0, yarn=yarn)["mixer"]
    mixer, w = _mixer(spec, dtype, seed, edit)
    return mixer, w, m


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, dim, rot, vdim, rank, yarn, page", [
    (5, 24, 12, 20, 40, (4.0, 64, 16.0, 2.0), 16), (3, 16, 16, 40, 64, None, 64), (1, 8, 2, 12, 20, (2.0, 32, 8.0, 1.0), 16),
    (18, 32, 16, 16, 96, (8.0, 16, 4.0, 0.5), 64), (4, 128, 64, 128, 512, (4.0, 128, 32.0, 1.0), 64), (16, 16, 48, 16, 32, None, 128)])
def test_latent_attention_with_sinks_alone(dtype, heads, dim, rot, vdim, rank, yarn, page):
    """
    Neighbouring channels rotated with and without YaRN (the magnitude on the rotated part only), value heads of another
    size than key heads, one head and more than a tile of them, sinks, the output gate; two requests in portions that
    end inside pages and token by token over split keys.
    """
    def edit(t):
        t["sink"] = torch.linspace(-2.0, 3.0, heads).to(t["sink"].dtype)
    mixer, w, m = _latent(48, heads, dim, rot, vdim, rank, 3.0 / (dim + rot), yarn, dtype, 3, edit)
    g = torch.Generator().manual_seed(1)
    lens = [330, 21]
    x_of = [torch.randn(n, 48, generator=g).to(dtype) for n in lens]
    want = [plain.latent_attention(x.double(), w, m, 1e-5) for x in x_of]
    cuts = [[(0, 17), (0, 2)], [(17, 33), (2, 19)], [(33, 34), (19, 20)], [(34, 320), (20, 21)], *[[(i, i + 1), (21, 21)] for i in range(320, 330)]]
    got = _in_steps(_Slots(mixer, dtype, lens, page=page), x_of, cuts)
    for a, b in zip(got, want):
        rows_close(a, b, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank, page", [(20, 16), (64, 64)])
def test_each_heads_sink_takes_the_weight_that_its_scores_leave(dtype, rank, page):
    """
    Every score is zero, so head h's output is n / (n + exp(sink_h)) times the common value whatever the number n of keys:
    one head whose sink holds nearly everything (above every score), one in between, one without any weight on it.
    """
    width, heads, n = 32, 3, 300
    sinks = [7.0, 2.0, -30.0]

    def edit(t):
        t["q"], t["g"] = torch.zeros_like(t["q"]), torch.zeros_like(t["g"])
        t["sink"] = torch.tensor(sinks).to(t["sink"].dtype)

    mixer, w, m = _latent(width, heads, 8, 16, 24, rank, 0.5, None, dtype, 5, edit)
    x = torch.randn(1, width, generator=torch.Generator().manual_seed(3)).repeat(n, 1).to(dtype)
    got = _in_steps(_Slots(mixer, dtype, [n], page=page), [x], [[(0, 1)], [(1, 3)], [(3, 200)], *[[(i, i + 1)] for i in range(200, n)]])[0]
    seen = torch.arange(1, n + 1, dtype=F64)[:, None]
    share = seen / (seen + torch.exp(torch.tensor(sinks, dtype=F64)))                     # [n, heads]
    c = plain.rms_div(x.double()[:1] @ w["dkv"][:rank].T, 1e-5) * w["dkv.norm"]
    v = (c @ w["uv"].T).view(1, heads, 24)
    want = (0.5 * share[..., None] * v).reshape(n, -1) @ w["o"].T
    assert float(share[0, 0]) < 0.01 and float(share[-1, 0]) < 0.25 and float(share[0, 2]) > 0.99
    assert float((got - want).norm(dim=-1).div(want.norm(dim=-1)).max()) < (2e-4 if dtype == torch.float32 else 0.03)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank, page, by", [(24, 16, "latent"), (64, 64, "latent"), (24, 16, "rotated"), (64, 64, "rotated")])
def test_latent_attention_finds_a_far_key_at_a_page_border(dtype, rank, page, by):
    """
    One token, hundreds of positions back at a page's last slot, is the only one that queries match, by its latent or by the
    rotated part (a pair of channels that turns too slowly to matter): they return its value, as a prompt portion and as
    single tokens; queries before it leave their weight to the sink.
    """
    width, dim, rot, vdim, far = 32, 16, 16, 24, 4 * page - 1

    def edit(t):
        for name in ("q", "uk", "g"):
            t[name] = torch.zeros_like(t[name])
        t["sink"] = torch.zeros_like(t["sink"]) + 4.0
        t["dkv"][0] = 0.0
        t["dkv"][0, 1] = 1.0                             # the latent's first channel, and the last rotated pair, read input channel 1
        t["dkv.norm"][0] = 1.0
        t["dkv"][rank:] = 0.0
        if by == "latent":
            t["q"][0, 0] = t["uk"][0, 0] = 1.0
        else:
            t["q"][dim + rot - 2, 0] = 1.0
            t["dkv"][rank + rot - 2, 1] = 1.0

    # YaRN with a factor of 10^5 leaves the last pair all but still
    mixer, w, m = _latent(width, 1, dim, rot, vdim, rank, 1.0, (1e5, 64, 32.0, 20.0), dtype, 8, edit)
    n = far + 150
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(4)) * 0.3
    x[:, 0], x[:, 1] = 8.0, 0.0
    x[far, 1] = 30.0 if by == "latent" else 6.0
    x = x.to(dtype)
    want = plain.latent_attention(x.double(), w, m, 1e-5)
    got = _in_steps(_Slots(mixer, dtype, [n], page=page), [x], [[(0, far - 2)], [(far - 2, far + 100)], *[[(i, i + 1)] for i in range(far + 100, n)]])[0]
    rows_close(got, want, dtype)
    c = plain.rms_div(x.double()[far:far + 1] @ w["dkv"][:rank].T, 1e-5) * w["dkv.norm"]
    alone = 0.5 * (c @ w["uv"].T) @ w["o"].T
    assert float((want[far:] - alone).norm(dim=-1).max() / alone.norm()) < 0.05               # the premise
    assert float((want[far - 1] - alone).norm() / alone.norm()) > 0.5


def test_rotated_parts_keep_their_pairs_and_the_magnitude_is_on_them_alone():
    """
    Only the rotated part scores: with one pair of channels set, the score of query i and key j is
    magnitude^2 cos((i - j) f) times their product, for every pair; the unrotated part scores without the magnitude.
    """
    width, dim, rot, n = 16, 4, 8, 40
    yarn = (6.0, 48, 12.0, 1.5)
    f, gain = plain.frequencies({"dims": rot, "base": 200.0, "scaling": dict(zip(("factor", "original", "fast", "slow"), yarn))})
    assert gain > 1.1
    x = torch.zeros(n, width)
    x[:, 0], x[:, 1] = 1.0, 1.0
    x[:, 2] = torch.linspace(-2.0, 2.0, n)              # what the values read
    for pair in list(range(rot // 2)) + [None]:
        def edit(t):
            for name in ("q", "dkv", "uk", "g"):
                t[name] = torch.zeros_like(t[name])
            t["sink"] = torch.zeros_like(t["sink"]) - 60.0
            t["dkv"][0, 2] = t["dkv"][1, 1] = 1.0
            t["dkv.norm"] = torch.ones_like(t["dkv.norm"])
            if pair is None:
                t["q"][0, 0] = 3.0
                t["uk"][0, 1] = 1.0
            else:
                t["q"][dim + 2 * pair, 0] = 3.0
                t["dkv"][20 + 2 * pair, 1] = 1.0
        mixer, w, m = _latent(width, 1, dim, rot, 12, 20, 1.0, yarn, torch.float32, 21, edit)
        c = plain.rms_div(x.double() @ w["dkv"][:20].T, 1e-5)
        d = torch.arange(n, dtype=F64)[:, None] - torch.arange(n, dtype=F64)[None, :]
        s = 3.0 * c[None, :, 1].expand(n, n) if pair is None else 3.0 * gain ** 2 * torch.cos(d * f[pair])
        p = torch.softmax(s.masked_fill(~torch.ones(n, n, dtype=torch.bool).tril(), -float("inf")), -1)
        want = 0.5 * ((p @ c) @ w["uv"].T) @ w["o"].T
        got = _in_steps(_Slots(mixer, torch.float32, [n]), [x], [[(0, 30)], *[[(i, i + 1)] for i in range(30, n)]])[0]
        torch.testing.assert_close(got, want, **TOL[torch.float32])


@pytest.mark.parametrize("heads, dim, rot, rank, page", [(3, 64, 64, 64, 64), (5, 64, 16, 40, 16), (2, 128, 64, 512, 64), (4, 128, 8, 128, 16),
                                                         (1, 64, 40, 24, 128)])
def test_latent_attention_of_long_portions_unfolded(heads, dim, rot, rank, page):
    """
    bfloat16, key and value heads of one size the tcgen05 prompt kernel takes: portions of 128 tokens and more attend over
    keys and values worked out for the step, the rotated parts shared by the heads, with the sinks, beside a request that
    feeds one token (which stays on the folded form); shorter steps before and after run the folded form alone.
    """
    dtype = torch.bfloat16

    def edit(t):
        t["sink"] = torch.linspace(-1.0, 4.0, heads).to(t["sink"].dtype)
    mixer, w, m = _latent(48, heads, dim, rot, dim, rank, 2.0 / (dim + rot) ** 0.5, (4.0, 128, 32.0, 1.0), dtype, 11, edit)
    lens = [420, 150, 40]
    g = torch.Generator().manual_seed(1)
    x_of = [torch.randn(n, 48, generator=g).to(dtype) for n in lens]
    cuts = [[(0, 200), (0, 3), (0, 1)], [(200, 201), (3, 140), (1, 2)], [(201, 406), (140, 150), (2, 40)], *[[(i, i + 1), (150, 150), (40, 40)] for i in range(406, 420)]]
    calls = mixer.rt.ops.calls
    before = calls.get("ts_prefill_attention_tcgen05_dense", 0)
    got = _in_steps(_Slots(mixer, dtype, lens, page=page), x_of, cuts)
    assert calls.get("ts_prefill_attention_tcgen05_dense", 0) == before + 3
    for a, x in zip(got, x_of):
        rows_close(a, plain.latent_attention(x.double(), w, m, 1e-5), dtype)


@pytest.mark.parametrize("by", ["latent", "rotated"])
@pytest.mark.parametrize("dim, rot", [(64, 16), (128, 64)])
def test_unfolded_portions_find_a_far_key_and_leave_the_rest_to_the_sink(dim, rot, by):
    """As above for the folded form: one far token that queries match by its latent or by its rotated part, in portions of hundreds of tokens."""
    dtype, width, rank, page, far = torch.bfloat16, 32, 64, 64, 191

    def edit(t):
        for name in ("q", "uk", "g"):
            t[name] = torch.zeros_like(t[name])
        t["sink"] = torch.zeros_like(t["sink"]) + 4.0
        t["dkv"][0] = 0.0
        t["dkv"][0, 1] = t["dkv.norm"][0] = 1.0
        t["dkv"][rank:] = 0.0
        if by == "latent":
            t["q"][0, 0] = t["uk"][0, 0] = 1.0
        else:
            t["q"][dim + rot - 2, 0] = t["dkv"][rank + rot - 2, 1] = 1.0

    mixer, w, m = _latent(width, 1, dim, rot, dim, rank, 1.0, (1e5, 64, 32.0, 20.0), dtype, 8, edit)
    n = 700
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(4)) * 0.3
    x[:, 0], x[:, 1] = 8.0, 0.0
    x[far, 1] = 30.0 if by == "latent" else 6.0
    x = x.to(dtype)
    want = plain.latent_attention(x.double(), w, m, 1e-5)
    calls = mixer.rt.ops.calls
    before = calls.get("ts_prefill_attention_tcgen05_dense", 0)
    got = _in_steps(_Slots(mixer, dtype, [n], page=page), [x], [[(0, far - 2)], [(far - 2, 500)], [(500, n)]])[0]
    assert calls.get("ts_prefill_attention_tcgen05_dense", 0) == before + 3
    rows_close(got, want, dtype)
    c = plain.rms_div(x.double()[far:far + 1] @ w["dkv"][:rank].T, 1e-5) * w["dkv.norm"]
    alone = 0.5 * (c @ w["uv"].T) @ w["o"].T
    assert float((want[far:] - alone).norm(dim=-1).max() / alone.norm()) < 0.05               # the premise
    assert float((got[far:] - alone).norm(dim=-1).max() / alone.norm()) < 0.08


# ---------------------------------------------------------------------------------------------- chunked attention, value mixing
class _WithSourceValues:
    """An attention mixer behind a layer whose values are a product of the same input: what a mixing layer finds in the step's scratch."""

    def __init__(self, mixer, weight, dtype):
        self.mixer, self.weight = mixer, weight.cuda().to(dtype)

    def __getattr__(self, name):
        return getattr(self.mixer, name)

    def forward(self, x, ctx, binding):
        from tinyserve_llm_b200.parts.gated_attention import SOURCE_VALUES
        wide = torch.cat([torch.zeros(x.shape[0], 8, dtype=x.dtype, device=x.device), x @ self.weight.T], dim=1)
        ctx.scratch[SOURCE_VALUES] = wide[:, 8:]                                    # a stretch of wider rows, as a projection's columns are
        return self.mixer.forward(x, ctx, binding)


def _attention(width, heads, kv_heads, dim, vdim, scale, chunk, rot, mix, dtype, seed, edit=None):
    from tinyserve_llm_b200.config.spec import GatedAttentionSpec, InlineRotarySpec
    spec = GatedAttentionSpec(hidden_size=width, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, value_dim=vdim, scale=scale,
                              qk_norm=True, qk_norm_scope="head", qk_norm_eps=1e-5, chunk=chunk, value_mix=mix,
                              position=InlineRotarySpec(dims=rot, base=300.0))
    m = C.attention(heads, kv_heads, dim, vdim, scale, chunk, rot, base=300.0, v_mix=mix != "none")["mixer"]
    mixer, w = _mixer(spec, dtype, seed, edit)
    return mixer, w, m


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, kv_heads, dim, vdim, chunk, rot, mix, page", [
    (4, 2, 24, 40, 11, 16, 0.35, 16), (3, 1, 64, 64, 64, 64, 0.8, 64), (5, 5, 12, 20, 1000, 4, None, 16), (6, 2, 128, 128, 100, 96, 0.5, 64),
    (2, 2, 64, 64, 37, 32, 1.0, 128), (4, 4, 64, 64, 16, 8, 0.0, 64)])
def test_chunked_attention_with_mixed_values_alone(dtype, heads, kv_heads, dim, vdim, chunk, rot, mix, page):
    """
    Heads normed with weights, rotation by halves over part of a head and over all of it, chunks shorter than a page, of one,
    and longer than the requests, values mixed with an earlier layer's in several shares (and not); portions that end
    inside pages and chunks, then token by token.
    """
    width = 64
    edit = None if mix is None else lambda t: t.update(vmix=torch.tensor(mix))
    mixer, w, m = _attention(width, heads, kv_heads, dim, vdim, 4.0 / dim, chunk, rot, "none" if mix is None else "mixed", dtype, 3, edit)
    g = torch.Generator().manual_seed(1)
    source = (torch.randn(kv_heads * vdim, width, generator=g) * 0.15).to(dtype)
    if mix is not None:
        mixer = _WithSourceValues(mixer, source, dtype)
    lens = [300, 21]
    x_of = [torch.randn(n, width, generator=g).to(dtype) for n in lens]
    want = [plain.attention(x.double(), w, m, 1e-5, x.double() @ source.double().T)[0] for x in x_of]
    cuts = [[(0, 17), (0, 2)], [(17, 33), (2, 19)], [(33, 34), (19, 20)], [(34, 285), (20, 21)], *[[(i, i + 1), (21, 21)] for i in range(285, 300)]]
    got = _in_steps(_Slots(mixer, dtype, lens, page=page), x_of, cuts)
    for a, b in zip(got, want):
        rows_close(a, b, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, page, chunk, far", [(24, 16, 40, 43), (64, 64, 96, 101), (64, 64, 64, 64), (128, 64, 130, 259)])
def test_a_key_is_seen_to_the_end_of_its_chunk_and_no_further(dtype, dim, page, chunk, far):
    """
    One key outshines all others of its chunk (queries meet it in channels that do not rotate): every query of the chunk
    returns its value, the first query of the next chunk does not see it, nor does the first of the chunk that comes before
    it; in a portion across the border and in single tokens across it.
    """
    width, n = 16, (far // chunk + 1) * chunk + 20

    def edit(t):
        for name in ("q", "k"):
            t[name] = torch.zeros_like(t[name])
        t["q"][dim - 1, 0] = 1.0
        t["k"][dim - 1, 1] = t["k"][dim - 2, 2] = 1.0
        t["q.norm"], t["k.norm"] = torch.ones_like(t["q.norm"]), torch.ones_like(t["k.norm"])

    mixer, w, m = _attention(width, 1, 1, dim, dim, 12.0 / dim, chunk, 4, "none", dtype, 5, edit)
    x = torch.randn(n, width, generator=torch.Generator().manual_seed(6)) * 0.3
    x[:, 0], x[:, 1], x[:, 2] = 2.0, 0.0, 2.0
    x[far, 1], x[far, 2] = 2.0, 0.0
    x = x.to(dtype)
    want, own = plain.attention(x.double(), w, m, 1e-5, None)
    end = (far // chunk + 1) * chunk
    marked = own[far] @ w["o"].T
    assert float((want[far:end] - marked).norm(dim=-1).max() / marked.norm()) < 0.05          # the premise
    assert float((want[end] - marked).norm() / marked.norm()) > 0.3
    for cuts in ([[(0, far)], [(far, max(far, end - 3))], [(max(far, end - 3), n)]],
                 [[(0, far + 1)], [(far + 1, end - 2)], *[[(i, i + 1)] for i in range(max(far + 1, end - 2), n)]]):
        cuts = [c for c in cuts if c[0][1] > c[0][0]]
        got = _in_steps(_Slots(mixer, dtype, [n], page=page), [x], cuts)[0]
        rows_close(got, want, dtype)
        assert float((got[end - 1] - marked).norm() / marked.norm()) < 0.06 and float((got[end] - marked).norm() / marked.norm()) > 0.3


# ---------------------------------------------------------------------------------------------- stream, embedding, experts
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [100, 1056])
def test_stream_kernel_adds_scaled_branches_as_they_are(dtype, width):
    from tinyserve_llm_b200.ops import get_ops
    ops = get_ops()
    g = torch.Generator().manual_seed(3)
    T, eps = 7, 1e-3
    stream = torch.randn(T, width, generator=g) * 3
    a, b = ((torch.randn(T, width, generator=g) * s).to(dtype) for s in (0.5, 9.0))
    wo = 1 + torch.randn(width, generator=g) * 0.3
    tol = dict(atol=2e-5, rtol=2e-5) if dtype == torch.float32 else dict(atol=0.03, rtol=0.01)
    for other, scale in ((b, 0.3), (None, 0.3), (b, 1.0)):
        want = stream.double() + scale * (a.double() + (other.double() if other is not None else 0))
        pair = (other.cuda() if other is not None else None, None, None, scale, scale)
        s = stream.cuda()
        out = ops.stream_norm(a.cuda(), None, s, wo.cuda(), eps, dtype, plain_add=True, pair=pair)
        torch.testing.assert_close(s.cpu().double(), want, atol=2e-5, rtol=2e-5)         # the stream stays float32 in both dtypes
        torch.testing.assert_close(out.cpu().double(), plain.rms_div(want, eps) * wo.double(), **tol)
        s = stream.cuda()
        picked = ops.stream_norm(a.cuda(), None, s, wo.cuda(), eps, dtype, rows=_i32([5, 0]), plain_add=True, pair=pair)
        assert torch.equal(s.cpu(), stream)                                               # with rows, the stream is read only
        torch.testing.assert_close(picked.cpu().double(), (plain.rms_div(want, eps) * wo.double())[[5, 0]], **tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("buckets, mul_prev, mul_cur", [(17, 5, 3), (1, 1, 1), (1000, 2_000_000_011, 1_999_999_973)])
def test_pair_rows_follow_the_previous_token_across_steps_and_requests(dtype, buckets, mul_prev, mul_cur):
    """Four requests in a batch, at their start and in their middle, one token and several; the last row is a first token's alone; a padding row."""
    from tinyserve_llm_b200.config.spec import PairEmbeddingSpec
    from tinyserve_llm_b200.ops import get_ops
    width, vocab = 24, 90
    g = torch.Generator().manual_seed(5)
    table = torch.randn(vocab, width, generator=g).to(dtype)
    second = torch.randn(buckets + 1, width, generator=g).to(dtype)
    spec = PairEmbeddingSpec(size=width, buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)
    whole = [ids_of(vocab, n, 60 + n) for n in (5, 9, 1, 6)]
    ranges = [(0, 5), (4, 9), (0, 1), (5, 6)]
    ctx = _ctx(ranges)
    ctx.prev_tokens = _i32([w[a - 1] if a else -1 for w, (a, _) in zip(whole, ranges)])
    ids = [t for w, (a, b) in zip(whole, ranges) for t in w[a:b]] + [3]
    ctx.seq_of_token = torch.cat([ctx.seq_of_token, _i32([-1])])
    stream = torch.empty(len(ids), width, device="cuda")
    out = get_ops().stream_norm(None, None, stream, torch.ones(width, device="cuda"), 1e-6, dtype, table=table.cuda(), ids=_i32(ids), scale=2.5,
                                pairs=(second.cuda(), spec, ctx))
    want = []
    for w, (a, b) in zip(whole, ranges):
        rows = plain.pair_rows(w, {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur})
        want.append(torch.stack([2.5 * table[w[t]].double() + second[rows[t]].double() for t in range(a, b)]))
    want = torch.cat(want)
    torch.testing.assert_close(stream[:-1].cpu().double(), want, atol=1e-5, rtol=1e-5)
    tol = dict(atol=1e-5, rtol=1e-5) if dtype == torch.float32 else dict(atol=0.02, rtol=0.01)
    torch.testing.assert_close(out[:-1].cpu().double(), plain.rms_div(want, 1e-6), **tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width, experts, top, shared, rows", [(64, 7, 2, 24, 5), (64, 5, 5, 0, 90), (64, 33, 3, 40, 130), (72, 2, 1, 16, 1),
                                                               (320, 9, 3, 40, 40), (72, 40, 4, 8, 33)])
def test_routed_experts_with_a_shared_one_alone(dtype, width, experts, top, shared, rows):
    from tinyserve_llm_b200.config.gimotar import GimotarConfig
    from tinyserve_llm_b200.parts.base import part_class
    from tinyserve_llm_b200.weights import random_tensors
    raw = C.model(50, width, 1e-6, 1.0, 1.0, (5, 1, 1), [(C.rglru(16, 1, 2), C.moe(experts, top, 40, shared))])
    spec = GimotarConfig.from_dict(raw).feed_forward_spec(0)
    cls = part_class("feed_forward", spec)
    tensors = dict(random_tensors(cls.declare(spec), 3, std=0.2))
    tensors["router.b"] = tensors["router.b"] * 8                          # a bias that changes who is chosen
    part = cls(spec, {k: v.cuda() for k, v in tensors.items()}, _runtime(dtype))
    x = torch.randn(rows, width, generator=torch.Generator().manual_seed(rows)).to(dtype)
    want = plain.experts(x.double(), {k: v.double() for k, v in tensors.items()}, raw["layers"][0]["mlp"])
    rows_close(part.forward(x.cuda(), _ctx([(0, rows)])).cpu().double(), want, dtype)


# ---------------------------------------------------------------------------------------------- entry points
def test_cached_prefixes_are_reused_with_the_token_before_them(folders):
    """
    Latent layers alone keep every key and no state: a second request takes the first one's pages, and its first own token
    forms its pair with the last reused one.
    """
    from tinyserve_llm_b200.engine.loading import build_cache, load_model
    from tinyserve_llm_b200.engine.step import StepEntry, StepRunner
    folder = folders["latent", "float32"]
    model = load_model(folder, "float32", "cuda")
    _, manager, storage = build_cache(model, 16, 12, caching=True)
    runner = StepRunner(model, manager, storage)
    first = ids_of(CONFIGS["latent"]["vocab"], 60, 40)
    second = first[:41] + ids_of(CONFIGS["latent"]["vocab"], 9, 41)
    assert manager.admit("a", first)
    runner.step([StepEntry("a", first, [59])])
    manager.commit("a", 60)
    manager.release("a")
    assert manager.admit("b", second, reuse_limit=len(second) - 1)
    taken = manager.committed_tokens("b")
    assert taken == 41
    got = runner.step([StepEntry("b", second[taken:], list(range(9)))]).cpu().double()
    manager.commit("b", 9)
    close(got, plain_logits(folder, second)[41:], "float32")


def test_a_forked_request_goes_on_with_its_own_state_and_previous_token(folders):
    folder = folders["mixed", "float32"]
    vocab = CONFIGS["mixed"]["vocab"]
    head, tails = ids_of(vocab, 37, 70), (ids_of(vocab, 6, 71), ids_of(vocab, 6, 72))
    eng = Engine(folder, "float32", page=16, pages=12, slots=3)
    eng.step([("a", head)])
    eng.manager.fork("a", "b")
    for i in range(6):
        eng.step([("a", tails[0][i:i + 1]), ("b", tails[1][i:i + 1])])
    close(eng.logits("a"), plain_logits(folder, head + tails[0]), "float32")
    close(eng.logits("b"), plain_logits(folder, head + tails[1])[37:], "float32")


def test_replay_program_on_a_model_folder(folders, tmp_path):
    """bin/trace_run on a Gimotar folder: portions, a decoded tail, two requests side by side, a reused slot."""
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
    for dtype in ("float32", "bfloat16"):
        folder = folders[name, dtype]
        want = {"a": plain_logits(folder, a), "b": plain_logits(folder, b)}
        out = tmp_path / dtype
        proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
                               "--out", str(out), "--max-tokens", "256", "--max-requests", "2"],
                              input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [line for line in proc.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(5)]
        got, expected = [], []
        for step, places in rows.items():
            got.append(torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(places), vocab)).double())
            expected += [want[r][p] for r, p in places]
        close(torch.cat(got), torch.stack(expected), dtype)


@pytest.mark.parametrize("name", ["mixed", "latent", "recurrent"])
def test_greedy_generation_through_the_entry_point(name, tmp_path):
    """
    LLM.generate with the scheduler, prompt portions, CUDA graphs and running ahead: the plain model's greedy tokens.  The
    token embedding is scaled down and the pair embedding up, so that a tied head does not answer every token with itself.
    """
    from tinyserve_llm_b200 import LLM, CacheConfig, SamplingParams, SchedulerConfig
    from tinyserve_llm_b200.weights.safetensors_io import write_safetensors
    raw = copy.deepcopy(CONFIGS[name])
    raw["embedding"]["scale"] = 0.05
    folder = str(tmp_path / "model")
    _write(folder, raw, SEEDS[name], C.WEIGHTS)
    tensors = read_tensors(folder)
    tensors["bigram"] = tensors["bigram"] * 3
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    prompts = [ids_of(raw["vocab"], n, 130 + n) for n in (3, 41, 18, 77, 1)]
    new = 12
    want = []
    for p in prompts:
        ids = list(p)
        for _ in range(new):
            ids.append(int(plain.forward(raw, tensors, ids)[-1].argmax()))
        want.append(ids[len(p):])
    assert min(len(set(w)) for w in want) > 3                             # the premise: the answers vary
    llm = LLM(folder, SchedulerConfig(max_model_len=128, max_num_seqs=3, max_num_batched_tokens=48, prefill_chunk=20),
              CacheConfig(block_size=16), dtype="float32", num_blocks=24, seed=0)
    for _ in range(2):                                                    # the second time over cached prefixes, where the model allows it
        done = llm.generate(prompts, SamplingParams(max_tokens=new, temperature=0.0, ignore_eos=True))
        assert [c.token_ids[0] for c in done] == want
