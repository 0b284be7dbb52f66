"""
Typed configuration of the Fuvipel decoder, read from the keys of its own config.json, and the
`ModelSpec` it turns into.

config.json: `architecture` "Fuvipel", `vocab`, `width`, `norm.eps` and `layers`, a list whose entries
give `type` (the mixer: "delta" or "parallel"), `mixer` (its sizes and constants) and `mlp` (`kind`
"dense" with `ff`, or null for a layer without a feed-forward).  A "delta" mixer holds `heads`,
`kv_heads`, `dim`, `vdim` and `conv`; a "parallel" mixer holds `left` (attention: `heads`, `kv_heads`,
`dim`, `vdim`, `scale`, `rot` with `dims` and `base`) and `right` (time mixing: `heads`, `dim`).  Layers
may come in any order and number; every size is read here and nowhere else.  Tensors: `embed`,
`final.norm`, and per layer `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`, `l<i>.mlp.*`.  The inner size of the
time mixing's decay projection is the shape of its tensors (`decay_rank`, optional, is only needed to
draw random weights).

What the design fixes stands here as constants: RMS norms with a weight on the sublayers' outputs only,
around a float32 residual stream; the delta rule has one decay a head and a silu gate, makes q and k
unit vectors with 1e-6 under the root and scales q by dim^(-1/2); the attention takes its keys as
projected for values, rotates neighbouring channels, norms every head of q and k without a weight, has a
sink of score 0 and a sigmoid output gate; the two halves of a parallel mixer are normed one by one
(`left.out`, `right.out`) and averaged; feed-forwards are up, squared relu, down; the output head is the
embedding table.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from tinyserve_llm_b200.config.duduvik import DEFAULT_MAX_POSITIONS, _get
from tinyserve_llm_b200.config.llama import ConfigError
from tinyserve_llm_b200.config.spec import (
    BlockSpec,
    GatedAttentionSpec,
    GatedDeltaRuleSpec,
    InlineRotarySpec,
    ModelSpec,
    ParallelMixerSpec,
    PartSpec,
    PlainMLPSpec,
    RunEntry,
    StreamRMSNormSpec,
    TimeMixingSpec,
)

MIXER_TYPES = ("delta", "parallel")
UNIT_EPS = 1e-6
SINK_SCORE = 0.0
BRANCH_SCALE = 0.5


@dataclass(frozen=True)
class FuvipelLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None


@dataclass(frozen=True)
class FuvipelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[FuvipelLayer, ...]
    max_positions: int
    eos_token_id: int
    raw: Mapping[str, Any]

    architecture = "Fuvipel"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "FuvipelConfig":
        layers = _get(raw, "layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: layers must be a non-empty list")
        parsed = []
        for i, layer in enumerate(layers):
            kind = layer.get("type") if isinstance(layer, Mapping) else None
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: layers[{i}].type {kind!r} is not supported; have {list(MIXER_TYPES)}")
            if not isinstance(layer.get("mixer"), Mapping):
                raise ConfigError(f"config.json: layers[{i}] lacks its mixer's sizes")
            mlp = layer.get("mlp")
            if mlp is not None and (not isinstance(mlp, Mapping) or mlp.get("kind") != "dense"):
                raise ConfigError(f"config.json: layers[{i}].mlp must be null or of kind 'dense', got {mlp!r}")
            parsed.append(FuvipelLayer(kind, layer["mixer"], mlp))
        eos = raw.get("eos_token_id")
        config = cls(vocab=_get(raw, "vocab", int), width=_get(raw, "width", int), norm_eps=_get(raw, "norm.eps", float),
                     layers=tuple(parsed), max_positions=int(raw.get("max_positions", DEFAULT_MAX_POSITIONS)),
                     eos_token_id=-1 if eos is None else int(eos), raw=raw)
        for i in range(len(parsed)):                       # every size is looked at now, not at the first step
            config.mixer_spec(i), config.feed_forward_spec(i)
        return config

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw)

    # ------------------------------------------------------------------ parts of layer i
    @staticmethod
    def _heads(where: str, m: Mapping[str, Any]) -> tuple[int, int]:
        heads, kv_heads = _get(m, "heads", int), _get(m, "kv_heads", int)
        if heads % kv_heads:
            raise ConfigError(f"config.json: {where}.heads={heads} is not a multiple of kv_heads={kv_heads}")
        return heads, kv_heads

    def _attention(self, where: str, m: Mapping[str, Any]) -> GatedAttentionSpec:
        heads, kv_heads = self._heads(where, m)
        dim, vdim = _get(m, "dim", int), _get(m, "vdim", int)
        if vdim != dim:
            raise ConfigError(f"config.json: {where}.vdim={vdim}: the values are the keys, of dim={dim}")
        dims, base = _get(m, "rot.dims", int), _get(m, "rot.base", float)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}.rot.dims={dims} must be even and at most dim={dim}")
        if base <= 0:
            raise ConfigError(f"config.json: {where}.rot.base={base} must be positive")
        return GatedAttentionSpec(hidden_size=self.width, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, value_dim=dim,
                                  scale=_get(m, "scale", float), qk_norm=True, qk_norm_scope="head", qk_norm_weight=False,
                                  qk_norm_eps=self.norm_eps, values="keys", sink=SINK_SCORE, output_gate=True,
                                  position=InlineRotarySpec(dims=dims, base=base, interleaved=True))

    def _delta_rule(self, where: str, m: Mapping[str, Any]) -> GatedDeltaRuleSpec:
        heads, kv_heads = self._heads(where, m)
        dim = _get(m, "dim", int)
        return GatedDeltaRuleSpec(hidden_size=self.width, num_heads=heads, num_kv_heads=kv_heads, key_dim=dim,
                                  value_dim=_get(m, "vdim", int), conv_taps=_get(m, "conv", int), q_scale=dim ** -0.5,
                                  unit_eps=UNIT_EPS, out_norm_eps=self.norm_eps, decay_scope="head", gate="silu")

    def mixer_spec(self, i: int) -> PartSpec:
        layer = self.layers[i]
        m, where = layer.mixer, f"layers[{i}].mixer"
        if layer.type == "delta":
            return self._delta_rule(where, m)
        left, right = _get(m, "left"), _get(m, "right")
        mixing = TimeMixingSpec(hidden_size=self.width, num_heads=_get(right, "heads", int), head_dim=_get(right, "dim", int),
                                decay_rank=int(right.get("decay_rank", 0)), out_norm_eps=self.norm_eps)
        return ParallelMixerSpec(branches=((self._attention(where + ".left", left), "left.", BRANCH_SCALE),
                                           (mixing, "right.", BRANCH_SCALE)),
                                 hidden_size=self.width, norm_names=("left.out", "right.out"), norm_eps=self.norm_eps)

    def feed_forward_spec(self, i: int) -> PartSpec | None:
        f = self.layers[i].mlp
        if f is None:
            return None
        return PlainMLPSpec(hidden_size=self.width, intermediate_size=_get(f, "ff", int), activation="relu2",
                            tensor_names=("up", "down"))


def fuvipel_model_spec(config: FuvipelConfig) -> ModelSpec:
    """One block per entry of `layers`, each run once in order with a cache entry of its own."""
    norm = StreamRMSNormSpec(size=config.width, eps=config.norm_eps, weight_name="")
    blocks = []
    for i in range(len(config.layers)):
        feed_forward = config.feed_forward_spec(i)
        blocks.append(BlockSpec(
            arrangement="post_norm_stream",
            mixer=config.mixer_spec(i),
            feed_forward=feed_forward,
            mixer_norm=None,
            feed_forward_norm=None,
            prefix=f"l{i}.",
            mixer_prefix="mix.",
            feed_forward_prefix="mlp.",
            mixer_post_norm=norm,
            feed_forward_post_norm=norm if feed_forward is not None else None,
            mixer_post_norm_prefix="norm1",
            feed_forward_post_norm_prefix="norm2",
        ))
    return ModelSpec(
        architecture=config.architecture,
        vocab_size=config.vocab,
        hidden_size=config.width,
        blocks=tuple(blocks),
        run=tuple(RunEntry(block=i, cache_entry=i) for i in range(len(blocks))),
        final_norm=norm,
        embedding_name="embed",
        final_norm_prefix="final.norm",
        lm_head_name=None,
        max_positions=config.max_positions,
        eos_token_id=config.eos_token_id,
    )
