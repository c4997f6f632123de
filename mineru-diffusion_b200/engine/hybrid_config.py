"""Configuration of decoders whose layers differ from one another: each names its mixer and its feed-forward.

``HybridConfig.from_json`` reads the ``config.json`` of the designs in ``DESIGNS``: ``layers`` lists, per layer, the mixer
``type`` with its sizes (``mixer``) and the feed-forward (``mlp``, or null for none).  Sizes that are not listed there
(low ranks) follow from tensor shapes when the weights are read.  What a design fixes for all its models -- where the norms
sit, how their weights are stored, the activation of its dense feed-forward, whether the embedding is the output matrix --
is in its ``Design`` entry.
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
class DecayScanSpec:
    """Linear recurrence with one decay per head: S <- decay S + step k v^T, read out by q.  ``decay``: the heads' fixed
    factors and plain projections (lightning attention), or None: factor and step come from a projection per token, and
    v, k and q pass a short convolution (Mamba-2).  ``kv_heads``: heads of k and q."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int = 0
    decay: list[float] | None = None
    norm_groups: int = 1


@dataclass
class WindowAttentionSpec:
    """Rotary attention with per-head q/k norms over a window, a sink, and one output gate per head; the values are the keys
    before norm and rotation."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int = 0             # 0: every key up to the query
    rot_dims: int = 0
    rot_base: float = 10000.0
    sink: bool = True


@dataclass
class ParallelSpec:
    """Two mixers side by side on the same input, added with scales."""
    left: WindowAttentionSpec
    right: DecayScanSpec
    left_scale: float
    right_scale: float


@dataclass
class DenseSpec:
    ff: int
    act: str = "relu2"          # "relu_glu": relu(gate) * up


@dataclass
class MoeSpec:
    experts: int
    top: int
    expert_ff: int
    groups: int = 1
    keep: int = 1
    shared_ff: int | None = None


Mixer = LatentAttentionSpec | ChannelDeltaSpec | MlstmSpec | DecayScanSpec | WindowAttentionSpec | ParallelSpec


def _plain(spec):
    """Reader of a mixer whose config keys are the fields of its spec."""
    return lambda mx: spec(**{k: mx[k] for k in spec.__dataclass_fields__ if k in mx})


def _lightning(mx: dict) -> DecayScanSpec:
    return DecayScanSpec(mx["heads"], mx["heads"], mx["dim"], mx["vdim"], decay=[float(d) for d in mx["decay"]])


def _mamba2(mx: dict) -> DecayScanSpec:
    return DecayScanSpec(mx["heads"], mx["groups"], mx["state"], mx["vdim"], conv=mx["conv"], norm_groups=mx["norm_groups"])


def _window_attention(mx: dict) -> WindowAttentionSpec:
    if mx["vdim"] != mx["dim"]:
        raise ValueError("values that are the keys have the keys' size")
    rot, mask = mx.get("rot"), mx.get("mask")
    return WindowAttentionSpec(mx["heads"], mx["kv_heads"], mx["dim"], float(mx["scale"]), 0 if mask is None else mask["size"],
                               **({} if rot is None else {"rot_dims": rot["dims"], "rot_base": float(rot["base"])}))


def _parallel(mx: dict) -> ParallelSpec:
    return ParallelSpec(_window_attention(mx["left"]), _mamba2(mx["right"]), float(mx["left_scale"]), float(mx["right_scale"]))


@dataclass(frozen=True)
class Design:
    """What all models of an architecture have in common."""
    mixers: dict                    # layer type -> reader of its mixer entry
    dense_act: str = "relu2"
    post_norm: bool = False         # norm of (scaled residual + sublayer) instead of a norm in front of the sublayer
    norm_offset: float = 0.0        # stored norm weights of the residual stream are offset from this
    tied_head: bool = False         # the output matrix is the embedding


DESIGNS = {
    "Zikunex": Design({"latent_attention": _plain(LatentAttentionSpec), "channel_delta": _plain(ChannelDeltaSpec),
                       "mlstm": _plain(MlstmSpec)}),
    "Nipadra": Design({"lightning": _lightning, "parallel": _parallel}, dense_act="relu_glu", post_norm=True, norm_offset=1.0,
                      tied_head=True),
}


@dataclass
class LayerSpec:
    type: str
    mixer: Mixer
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
    residual_scale: float = 1.0                 # post-norm designs: factor of the residual in front of the sum

    @property
    def design(self) -> Design:
        return DESIGNS[self.architecture]

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
            for part in parts_of(mx):
                if isinstance(part, WindowAttentionSpec):
                    if part.heads % part.kv_heads:
                        raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                    if part.rot_dims % 2 or not 0 <= part.rot_dims <= part.dim:
                        raise ValueError(f"layer {i}: the rotated dimensions must be pairs within a head")
                    if part.window < 0 or part.scale <= 0:
                        raise ValueError(f"layer {i}: window and scale must be positive")
                if isinstance(part, DecayScanSpec):
                    if part.heads % part.kv_heads or part.heads * part.vdim % part.norm_groups:
                        raise ValueError(f"layer {i}: heads and channels must split into equal groups")
                    if part.decay is not None and len(part.decay) != part.heads:
                        raise ValueError(f"layer {i}: one decay per head")
                    if part.decay is None and part.conv < 1:
                        raise ValueError(f"layer {i}: the short convolution has at least one tap")
            mlp = layer.mlp
            if isinstance(mlp, MoeSpec):
                if mlp.experts % mlp.groups or not 0 < mlp.keep <= mlp.groups:
                    raise ValueError(f"layer {i}: experts must split into equal groups")
                if mlp.top > mlp.keep * (mlp.experts // mlp.groups):
                    raise ValueError(f"layer {i}: top exceeds the experts of the groups kept")

    @classmethod
    def from_json(cls, raw: dict) -> "HybridConfig":
        design = DESIGNS[raw["architecture"]]
        layers = []
        for i, entry in enumerate(raw["layers"]):
            kind = entry["type"]
            if kind not in design.mixers:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            layers.append(LayerSpec(kind, design.mixers[kind](entry["mixer"]), _mlp_spec(entry.get("mlp"), i, design)))
        return cls(vocab_size=raw["vocab"], hidden_size=raw["width"], layers=layers,
                   embed_scale=float(raw.get("embedding", {}).get("scale", 1.0)), rms_norm_eps=float(raw["norm"]["eps"]),
                   architecture=raw["architecture"], residual_scale=float(raw["postln_alpha"]) if design.post_norm else 1.0)


def parts_of(mixer: Mixer) -> tuple:
    """The mixers a layer's mixer consists of."""
    return (mixer.left, mixer.right) if isinstance(mixer, ParallelSpec) else (mixer,)


def _mlp_spec(mlp: dict | None, layer: int, design: Design):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return DenseSpec(mlp["ff"], design.dense_act)
    if mlp["kind"] == "moe" and design.dense_act == "relu2":
        router = mlp["router"]
        groups = router.get("groups") or {"count": 1, "keep": 1}
        shared = mlp.get("shared")
        return MoeSpec(router["experts"], router["top"], mlp["expert"]["ff"], groups["count"], groups["keep"],
                       None if shared is None else shared["ff"])
    raise ValueError(f"layer {layer}: unknown feed-forward kind {mlp['kind']!r}")
