"""Configuration of decoders whose layers differ from one another: each names its mixer and its feed-forward.

``HybridConfig.from_json`` reads the ``config.json`` of the "Zikunex" design: ``layers`` lists, per layer, the mixer
``type`` with its sizes (``mixer``) and the feed-forward (``mlp``, or null for none).  Sizes that are not listed there
(low ranks, convolution taps) follow from tensor shapes when the weights are read.
"""
from __future__ import annotations

from dataclasses import dataclass, field


@dataclass
class LatentAttentionSpec:
    """Attention whose keys and values are per-head projections of one cached latent per token."""
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    kv_from: int | None = None      # layer whose cached latents this layer reads (None: its own)


@dataclass
class ChannelDeltaSpec:
    """Gated delta rule with one decay per key channel."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass
class MlstmSpec:
    """Matrix memory with exponential gates."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass
class DenseSpec:
    ff: int


@dataclass
class MoeSpec:
    experts: int
    top: int
    expert_ff: int
    groups: int = 1
    keep: int = 1
    shared_ff: int | None = None


MIXERS = {"latent_attention": LatentAttentionSpec, "channel_delta": ChannelDeltaSpec, "mlstm": MlstmSpec}


@dataclass
class LayerSpec:
    type: str
    mixer: LatentAttentionSpec | ChannelDeltaSpec | MlstmSpec
    mlp: DenseSpec | MoeSpec | None = None


@dataclass
class HybridConfig:
    vocab_size: int
    hidden_size: int
    layers: list[LayerSpec] = field(default_factory=list)
    embed_scale: float = 1.0
    rms_norm_eps: float = 1e-5
    max_position_embeddings: int = 1 << 20      # no positions enter the model: a bound for page tables only
    architecture: str = "Zikunex"

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def __post_init__(self):
        for i, layer in enumerate(self.layers):
            mx = layer.mixer
            if isinstance(mx, LatentAttentionSpec) and mx.kv_from is not None:
                j = mx.kv_from
                src = self.layers[j].mixer if 0 <= j < i else None
                if not isinstance(src, LatentAttentionSpec) or src.kv_from is not None or src.kv_rank != mx.kv_rank:
                    raise ValueError(f"layer {i}: kv_from {j} must name an earlier latent_attention layer with its own "
                                     "latents of the same rank")
            if isinstance(mx, ChannelDeltaSpec) and mx.heads % mx.kv_heads:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            mlp = layer.mlp
            if isinstance(mlp, MoeSpec):
                if mlp.experts % mlp.groups or not 0 < mlp.keep <= mlp.groups:
                    raise ValueError(f"layer {i}: experts must split into equal groups")
                if mlp.top > mlp.keep * (mlp.experts // mlp.groups):
                    raise ValueError(f"layer {i}: top exceeds the experts of the groups kept")

    @classmethod
    def from_json(cls, raw: dict) -> "HybridConfig":
        layers = []
        for i, entry in enumerate(raw["layers"]):
            kind = entry["type"]
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            spec = MIXERS[kind]
            mixer = spec(**{k: entry["mixer"][k] for k in spec.__dataclass_fields__ if k in entry["mixer"]})
            layers.append(LayerSpec(kind, mixer, _mlp_spec(entry.get("mlp"), i)))
        return cls(vocab_size=raw["vocab"], hidden_size=raw["width"], layers=layers,
                   embed_scale=float(raw["embedding"]["scale"]), rms_norm_eps=float(raw["norm"]["eps"]),
                   architecture=raw["architecture"])


def _mlp_spec(mlp: dict | None, layer: int):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return DenseSpec(mlp["ff"])
    if mlp["kind"] == "moe":
        router = mlp["router"]
        groups = router.get("groups") or {"count": 1, "keep": 1}
        shared = mlp.get("shared")
        return MoeSpec(router["experts"], router["top"], mlp["expert"]["ff"], groups["count"], groups["keep"],
                       None if shared is None else shared["ff"])
    raise ValueError(f"layer {layer}: unknown feed-forward kind {mlp['kind']!r}")
