"""
Typed configuration of the Gimotar decoder, read from the keys of its own config.json, and the
`ModelSpec` it turns into.

config.json: `architecture` "Gimotar", `vocab`, `width`, `norm.eps`, `residual_mult`, `embedding` (`scale`,
and `bigram` with `buckets`, `mul_prev`, `mul_cur`) and `layers`, a list whose entries give `type` (the mixer:
"rglru", "latent_attention" or "attention"), `mixer` (its sizes and constants) and `mlp` (`kind` "moe" with
`router.experts`, `router.top`, `expert.ff` and `shared.ff`, or null for a layer without a feed-forward).  Mixers:

* "rglru": `width`, `blocks`, `conv`.  Griffin's recurrent block.
* "latent_attention": `heads`, `dim`, `rot_dim`, `vdim`, `kv_rank`, `scale`, `rot` with `dims` (= rot_dim), `base` and
  an optional `scaling` of `factor`, `original`, `fast`, `slow` (YaRN).
* "attention": `heads`, `kv_heads`, `dim`, `vdim`, `scale`, `mask.size` (chunks), `v_mix`, `rot` with `dims`, `base`.

Layers may come in any order and number; every size is read here and nowhere else.  Tensors: `embed`, `bigram`,
`final.norm`, and per layer `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`.

What the design fixes stands here as constants: one RMS norm a layer with a weight stored around zero, whose
output both sublayers read, around a float32 residual stream; the latent attention rotates neighbouring channels,
has no query latent, a sink a head and a sigmoid gate on its concatenated heads; the attention norms every head of
q and k with plain weights and rotates by halves; of the layers with `v_mix` the first gives the values that the
others mix into theirs; the recurrence's rate constant is 8; experts are gated by silu, chosen by a router with a
bias and weighted by the softmax over the chosen logits; the output head is the embedding table.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from tinyserve_llm_b200.config.duduvik import DEFAULT_MAX_POSITIONS, _get
from tinyserve_llm_b200.config.llama import ConfigError
from tinyserve_llm_b200.config.spec import (
    BlockSpec,
    GatedAttentionSpec,
    GatedLRUSpec,
    GatedMLPSpec,
    InlineRotarySpec,
    LatentAttentionSpec,
    ModelSpec,
    PairEmbeddingSpec,
    PartSpec,
    RoutedExpertsSpec,
    RunEntry,
    StreamRMSNormSpec,
    YarnScaling,
)

MIXER_TYPES = ("rglru", "latent_attention", "attention")
DECAY_RATE = 8.0


@dataclass(frozen=True)
class GimotarLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Mapping[str, Any] | None


@dataclass(frozen=True)
class GimotarConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    embedding_scale: float
    layers: tuple[GimotarLayer, ...]
    max_positions: int
    eos_token_id: int
    raw: Mapping[str, Any]

    architecture = "Gimotar"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "GimotarConfig":
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
            if mlp is not None and mlp.get("kind") != "moe":
                raise ConfigError(f"config.json: layers[{i}].mlp.kind {mlp.get('kind')!r} is not supported; have ['moe']")
            parsed.append(GimotarLayer(kind, layer["mixer"], mlp))
        eos = raw.get("eos_token_id")
        config = cls(vocab=_get(raw, "vocab", int), width=_get(raw, "width", int), norm_eps=_get(raw, "norm.eps", float),
                     residual_mult=_get(raw, "residual_mult", float), embedding_scale=_get(raw, "embedding.scale", float),
                     layers=tuple(parsed), max_positions=int(raw.get("max_positions", DEFAULT_MAX_POSITIONS)),
                     eos_token_id=-1 if eos is None else int(eos), raw=raw)
        config.embedding_pairs()
        for i in range(len(parsed)):                       # every size is looked at now, not at the first step
            config.mixer_spec(i), config.feed_forward_spec(i)
        return config

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw)

    def embedding_pairs(self) -> PairEmbeddingSpec | None:
        if self.raw["embedding"].get("bigram") is None:
            return None
        spec = PairEmbeddingSpec(size=self.width, buckets=_get(self.raw, "embedding.bigram.buckets", int),
                                 mul_prev=_get(self.raw, "embedding.bigram.mul_prev", int),
                                 mul_cur=_get(self.raw, "embedding.bigram.mul_cur", int), name="bigram")
        if spec.buckets <= 0 or spec.mul_prev < 0 or spec.mul_cur < 0:
            raise ConfigError("config.json: embedding.bigram needs a positive number of buckets and multipliers that are not negative")
        return spec

    # ------------------------------------------------------------------ parts of layer i
    @property
    def value_source(self) -> int:
        """The first layer that mixes values, -1 if none does."""
        return next((i for i, layer in enumerate(self.layers) if layer.type == "attention" and layer.mixer.get("v_mix")), -1)

    @staticmethod
    def _rotation(where: str, m: Mapping[str, Any], dim: int, interleaved: bool) -> InlineRotarySpec | None:
        rot = m.get("rot")
        if rot is None or not rot.get("dims"):
            return None
        dims, base = _get(rot, "dims", int), _get(rot, "base", float)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}.rot.dims={dims} must be even and at most {dim}")
        if base <= 1:
            raise ConfigError(f"config.json: {where}.rot.base must be above 1, got {base}")
        yarn = None
        if rot.get("scaling"):
            sc = rot["scaling"]
            yarn = YarnScaling(factor=_get(sc, "factor", float), original=_get(sc, "original", float),
                               fast=_get(sc, "fast", float), slow=_get(sc, "slow", float))
            if yarn.factor <= 0 or yarn.original <= 0 or yarn.fast <= 0 or yarn.slow <= 0:
                raise ConfigError(f"config.json: {where}.rot.scaling needs positive factor, original, fast and slow")
        return InlineRotarySpec(dims=dims, base=base, yarn=yarn, interleaved=interleaved)

    def _latent_attention(self, where: str, m: Mapping[str, Any]) -> LatentAttentionSpec:
        rot_dim = _get(m, "rot_dim", int)
        position = self._rotation(where, m, rot_dim, interleaved=True)
        if (position.dims if position is not None else 0) != rot_dim:
            raise ConfigError(f"config.json: {where}.rot.dims must be rot_dim={rot_dim}")
        return LatentAttentionSpec(hidden_size=self.width, num_heads=_get(m, "heads", int), head_dim=_get(m, "dim", int),
                                   rot_dim=rot_dim, value_dim=_get(m, "vdim", int), q_rank=0, kv_rank=_get(m, "kv_rank", int),
                                   scale=_get(m, "scale", float), norm_eps=self.norm_eps, position=position, output_gate=True,
                                   sink=True)

    def _attention(self, i: int, where: str, m: Mapping[str, Any]) -> GatedAttentionSpec:
        heads, kv_heads, dim, vdim = (_get(m, k, int) for k in ("heads", "kv_heads", "dim", "vdim"))
        if heads % kv_heads:
            raise ConfigError(f"config.json: {where}.heads={heads} is not a multiple of kv_heads={kv_heads}")
        mix = "none"
        if m.get("v_mix"):
            mix = "source" if i == self.value_source else "mixed"
            source = self.layers[self.value_source].mixer
            if kv_heads * vdim != _get(source, "kv_heads", int) * _get(source, "vdim", int):
                raise ConfigError(f"config.json: {where} mixes its values with those of layer {self.value_source}, which has others "
                                  "than kv_heads * vdim of them")
        chunk = 0 if m.get("mask") is None else _get(m, "mask.size", int)
        return GatedAttentionSpec(hidden_size=self.width, num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, value_dim=vdim,
                                  scale=_get(m, "scale", float), qk_norm=True, qk_norm_scope="head", qk_norm_eps=self.norm_eps,
                                  chunk=chunk, position=self._rotation(where, m, dim, interleaved=False), value_mix=mix)

    def mixer_spec(self, i: int) -> PartSpec:
        layer = self.layers[i]
        m, where = layer.mixer, f"layers[{i}].mixer"
        if layer.type == "latent_attention":
            return self._latent_attention(where, m)
        if layer.type == "attention":
            return self._attention(i, where, m)
        width, blocks = _get(m, "width", int), _get(m, "blocks", int)
        if blocks <= 0 or width % blocks:
            raise ConfigError(f"config.json: {where}.width={width} is not a multiple of blocks={blocks}")
        return GatedLRUSpec(hidden_size=self.width, width=width, blocks=blocks, conv_taps=_get(m, "conv", int),
                            decay_rate=DECAY_RATE)

    def feed_forward_spec(self, i: int) -> PartSpec | None:
        f = self.layers[i].mlp
        if f is None:
            return None
        experts, top = _get(f, "router.experts", int), _get(f, "router.top", int)
        if not 0 < top <= experts:
            raise ConfigError(f"config.json: layers[{i}].mlp.router.top={top} must be between 1 and experts={experts}")
        gated = lambda ff: GatedMLPSpec(hidden_size=self.width, intermediate_size=ff, activation="silu",  # noqa: E731
                                        tensor_names=("gate", "up", "down"))
        shared = gated(_get(f, "shared.ff", int)) if f.get("shared") is not None else None
        return RoutedExpertsSpec(hidden_size=self.width, num_experts=experts, top=top, expert=gated(_get(f, "expert.ff", int)),
                                 shared=shared)


def gimotar_model_spec(config: GimotarConfig) -> ModelSpec:
    """One block per entry of `layers`, each run once in order with a cache entry of its own."""
    norm = StreamRMSNormSpec(size=config.width, eps=config.norm_eps, weight_offset=1.0, weight_name="")
    blocks = tuple(BlockSpec(
        arrangement="parallel_stream",
        mixer=config.mixer_spec(i),
        feed_forward=config.feed_forward_spec(i),
        mixer_norm=norm,
        feed_forward_norm=None,
        prefix=f"l{i}.",
        mixer_prefix="mix.",
        feed_forward_prefix="mlp.",
        mixer_norm_prefix="norm1",
        branch_scale=config.residual_mult,
    ) for i in range(len(config.layers)))
    source = config.value_source
    return ModelSpec(
        architecture=config.architecture,
        vocab_size=config.vocab,
        hidden_size=config.width,
        blocks=blocks,
        run=tuple(RunEntry(block=i, cache_entry=i) for i in range(len(blocks))),
        final_norm=norm,
        embedding_name="embed",
        final_norm_prefix="final.norm",
        lm_head_name=None,
        max_positions=config.max_positions,
        eos_token_id=config.eos_token_id,
        embedding_scale=config.embedding_scale,
        embedding_pairs=config.embedding_pairs(),
        # the layer whose values the others mix in has no use for a mixing number; a checkpoint may carry it all the same
        optional_tensors=(f"l{source}.mix.vmix",) if source >= 0 else (),
    )
