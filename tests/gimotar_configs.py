"""
Small Gimotar configurations for the tests, as config.json dictionaries.  They differ from one another in
every size and in the order of layers: widths, head counts and parts that are not powers of two, value heads of
other sizes than key heads, chunks shorter than a page and longer than every prompt, convolutions of 1 to 9 taps,
one part and many, YaRN and plain rotation, attention layers that mix values beside ones that do not, layers without
a feed-forward and feed-forwards without a shared expert.
"""

import torch


def attention(heads, kv_heads, dim, vdim, scale, chunk, rot_dims, base=500.0, v_mix=True):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": chunk}, "rot": {"base": base, "dims": rot_dims}, "v_mix": v_mix}}


def rglru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=300.0, yarn=None):
    rot = {"base": base, "dims": rot_dim}
    if yarn:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale, "rot": rot}}


def moe(experts, top, ff, shared):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    return dict(out, shared={"ff": shared}) if shared else out


def model(vocab, width, eps, mult, scale, bigram, layers):
    return {"architecture": "Gimotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))},
            "layers": [dict(mixer, mlp=mlp) for mixer, mlp in layers]}


# every mechanism, the recurrence first; value mixing over layers of unequal head sizes and equal value widths
MIXED = model(300, 96, 1e-5, 0.7, 3.0, (101, 13, 5), [
    (rglru(120, 5, 3), moe(5, 2, 40, 24)),
    (attention(4, 2, 20, 36, 0.3, 11, 12), moe(6, 3, 24, 40)),
    (latent(5, 24, 12, 20, 40, 0.2, yarn=(4.0, 64, 16.0, 2.0)), None),
    (attention(3, 3, 16, 12, 0.3, 1000, 16, v_mix=False), moe(4, 1, 32, 0)),
    (attention(6, 3, 28, 24, 0.25, 37, 8, base=90.0), moe(3, 3, 48, 16)),
    (rglru(84, 3, 1), None),
    (attention(2, 1, 40, 72, 0.2, 16, 40), moe(7, 2, 16, 8)),
])

# latent attention only: pages that keep every key, no state slot, so that cached prefixes are reused
LATENT = model(211, 64, 1e-6, 1.0, 1.0, (17, 100003, 999983), [
    (latent(3, 16, 8, 24, 32, 0.25), moe(4, 2, 24, 32)),
    (latent(18, 8, 20, 16, 24, 0.3, base=40.0, yarn=(8.0, 16, 4.0, 0.5)), None),
])

# recurrences only: state slots, no page
RECURRENT = model(150, 80, 1e-5, 0.4, 5.0, (64, 3, 1), [
    (rglru(96, 1, 4), moe(4, 2, 24, 16)),
    (rglru(60, 12, 9), None),
    (rglru(64, 4, 2), moe(2, 1, 40, 0)),
])

# sizes the bfloat16 kernels for a few tokens and the tensor-core attention kernels take
WIDE = model(512, 128, 1e-6, 0.6, 8.0, (251, 127, 31), [
    (attention(4, 2, 64, 64, 0.125, 96, 32), moe(8, 3, 64, 96)),
    (latent(4, 32, 16, 48, 96, 0.14, yarn=(3.0, 128, 24.0, 1.5)), moe(6, 2, 32, 64)),
    (rglru(192, 3, 4), moe(4, 2, 64, 32)),
    (attention(2, 2, 64, 64, 0.15, 200, 64), None),
    (rglru(256, 2, 2), None),
    (latent(17, 16, 32, 16, 128, 0.15), moe(4, 4, 32, 32)),
])

# heads of 128 channels, three query heads a key/value head
GROUPED = model(257, 128, 1e-5, 0.9, 2.0, (90, 7, 11), [
    (latent(3, 128, 64, 128, 160, 0.07, base=10000.0), moe(4, 2, 64, 64)),
    (attention(6, 2, 128, 128, 0.09, 130, 128), moe(3, 1, 32, 48)),
    (rglru(160, 5, 4), moe(4, 3, 32, 0)),
    (attention(4, 2, 128, 128, 0.08, 64, 64), None),
])

WEIGHTS = {"std": 0.1, "unit_std": 0.25}


def telling(tensors):
    """
    Random tensors, in place, of sizes at which every mechanism matters: decays from nearly one to nearly zero,
    convolution taps of ordinary size, sinks on both sides of the scores, values mixed by about a third, router
    scores that stand apart.
    """
    for i, name in enumerate(sorted(tensors)):
        last = name.rpartition(".")[2]
        t = tensors[name]
        if last == "lam":
            tensors[name] = torch.linspace(-9.0, 1.0, t.numel()).to(t.dtype)
        elif last == "conv":
            tensors[name] = t * 4
        elif last == "sink":
            tensors[name] = t * 20
        elif last == "vmix":
            tensors[name] = torch.tensor(0.2 + 0.1 * (i % 4), dtype=t.dtype)
        elif last in ("router", "ra", "ri"):
            tensors[name] = t * 3
