"""
Small Fuvipel configurations for the tests, as config.json dictionaries.  They differ from one another in
every size and in the order of layers: widths and head counts that are not powers of two, key and value
sizes of the delta rule that differ (and, once, agree), fewer q/k heads than value heads, rotation over
part of a head and over all of it, halves of a parallel mixer that are equally wide and that are not,
convolutions of 1 to 5 taps, layers with and without a feed-forward, a model of delta rules only.
"""


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attention(heads, kv_heads, dim, scale, rot_dims, base=10000.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "rot": {"base": base, "dims": rot_dims}}


def mixing(heads, dim, decay_rank):
    return {"heads": heads, "dim": dim, "decay_rank": decay_rank}


def parallel(left, right):
    return {"type": "parallel", "mixer": {"left": left, "right": right}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def model(vocab, width, eps, layers):
    return {"architecture": "Fuvipel", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [dict(mixer, mlp=mlp) for mixer, mlp in layers]}


# every mechanism; odd sizes; layers of both kinds with and without a feed-forward; a parallel layer first
MIXED = model(300, 96, 1e-5, [
    (parallel(attention(4, 2, 20, 0.3, 12, base=5000.0), mixing(3, 24, 10)), dense(72)),
    (delta(4, 2, 20, 24, 3), None),
    (delta(3, 3, 36, 12, 5), dense(40)),
    (parallel(attention(3, 1, 16, 0.5, 16), mixing(2, 24, 5)), None),
    (delta(2, 1, 24, 40, 1), None),
])

# delta rules only: the model needs state slots, no page
RECURRENT = model(211, 64, 1e-6, [
    (delta(6, 2, 16, 8, 2), dense(48)),
    (delta(2, 2, 40, 24, 4), None),
])

# sizes the bfloat16 kernels for a few tokens and the tensor-core attention take
WIDE = model(512, 128, 1e-6, [
    (delta(4, 2, 32, 32, 4), None),
    (parallel(attention(4, 2, 64, 0.1, 32, base=20000.0), mixing(8, 32, 32)), dense(192)),
    (delta(2, 1, 64, 128, 4), dense(96)),
    (parallel(attention(2, 2, 64, 0.2, 64), mixing(3, 64, 16)), None),
])

# heads of 128 channels, three query heads a key/value head (the tensor-core attention's other head size)
GROUPED = model(257, 128, 1e-5, [
    (parallel(attention(6, 2, 128, 0.09, 128, base=1000.0), mixing(2, 128, 8)), dense(64)),
    (delta(2, 2, 128, 64, 4), None),
])

WEIGHTS = {"std": 0.1, "unit_std": 0.25}


def steady_reads(tensors):
    """
    Makes every recurrence's q (or r) resemble its k, in place.  A state that holds one token reads out (k . q) v, which
    its norm turns into sign(k . q) v: with independent random q and k the first tokens of a model would hang on
    bfloat16's rounding of the projections wherever k . q is near zero.  Convolutions get taps of ordinary size.
    """
    for name in list(tensors):
        if name.endswith(".conv"):
            tensors[name] = tensors[name] * 4
    for name in list(tensors):
        base, _, last = name.rpartition(".")
        if last == "A_log":
            tensors[f"{base}.q"] = tensors[f"{base}.k"] + tensors[f"{base}.q"] / 4
            tensors[f"{base}.q.conv"] = tensors[f"{base}.k.conv"]
        elif last == "w0":
            tensors[f"{base}.r"] = tensors[f"{base}.k"] + tensors[f"{base}.r"] / 4
            tensors[f"{base}.mu.r"] = tensors[f"{base}.mu.k"]
            tensors[f"{base}.u"] = 0.5 + tensors[f"{base}.u"].abs()
