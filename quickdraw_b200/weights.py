"""Weight containers for the batch-one decode path (the data contract of the kernels).

Field names, shapes and dtypes follow the reference containers so that a checkpoint
object built for the reference can be handed to this package unchanged
(reference: quickdraw/models/weights.py:29-166).  Only the containers live here; the
arithmetic that consumes them is in the CUDA library.

NVFP4 storage (reference: quickdraw/models/weights.py:14-55):
  * ``weight``         uint8 ``[..., out, in/2]``; byte j holds input 2j in its low
                       nibble and input 2j+1 in its high nibble, each an E2M1 code
                       (bit 3 sign, bits 2:1 exponent, bit 0 mantissa);
  * ``weight_scale``   float8_e4m3fn ``[..., out, in/group_size]``;
  * ``weight_scale_2`` fp32 scalar, or ``[E]`` for an expert bank;
  * the value of weight (o, i) is ``e2m1 * weight_scale[o, i // group] * weight_scale_2``.
"""

from __future__ import annotations

import json
from dataclasses import dataclass, field, fields
from pathlib import Path

import torch

E2M1_MAGNITUDES = (0.0, 0.5, 1.0, 1.5, 2.0, 3.0, 4.0, 6.0)


@dataclass
class NVFP4Linear:
    """Weight-only FP4 projection; activations stay bf16 (W4A16)."""
    weight: torch.Tensor
    weight_scale: torch.Tensor
    weight_scale_2: torch.Tensor
    input_scale: torch.Tensor | None = None
    group_size: int = 16

    @property
    def out_features(self) -> int:
        return self.weight.shape[-2]

    @property
    def in_features(self) -> int:
        return 2 * self.weight.shape[-1]

    def nbytes(self) -> int:
        return self.weight.nbytes + self.weight_scale.nbytes + self.weight_scale_2.nbytes


@dataclass
class FP8Linear:
    """Static E4M3 projection with scalar weight and activation scales."""
    weight: torch.Tensor
    weight_scale: torch.Tensor
    input_scale: torch.Tensor | None = None

    @property
    def out_features(self) -> int:
        return self.weight.shape[0]

    @property
    def in_features(self) -> int:
        return self.weight.shape[1]


@dataclass
class GDNWeights:
    """Gated-DeltaNet mixer: fused q|k|v projection, output-gate projection z,
    decay/beta projections a/b, depthwise conv taps, per-head decay parameters,
    per-head norm gamma and the output projection."""
    in_proj_qkv: NVFP4Linear | FP8Linear
    in_proj_z: NVFP4Linear | FP8Linear
    in_proj_a: torch.Tensor
    in_proj_b: torch.Tensor
    conv1d: torch.Tensor
    A_log: torch.Tensor
    dt_bias: torch.Tensor
    norm: torch.Tensor
    out_proj: NVFP4Linear | FP8Linear


@dataclass
class FullAttnWeights:
    """GQA mixer; every q_proj head stores its query rows then its gate rows."""
    q_proj: NVFP4Linear | FP8Linear
    k_proj: NVFP4Linear | FP8Linear
    v_proj: NVFP4Linear | FP8Linear
    o_proj: NVFP4Linear | FP8Linear
    q_norm: torch.Tensor
    k_norm: torch.Tensor


@dataclass
class MoEWeights:
    """Router, expert banks (leading expert axis) and the gated shared expert."""
    router: torch.Tensor
    shared_expert_gate: torch.Tensor
    experts_gate: NVFP4Linear
    experts_up: NVFP4Linear
    experts_down: NVFP4Linear
    shared_gate: NVFP4Linear
    shared_up: NVFP4Linear
    shared_down: NVFP4Linear


@dataclass
class LayerWeights:
    idx: int
    layer_type: str
    input_layernorm: torch.Tensor
    post_attention_layernorm: torch.Tensor
    attn: GDNWeights | FullAttnWeights
    moe: MoEWeights


@dataclass
class ModelConfig:
    hidden_size: int
    num_hidden_layers: int
    layer_types: list[str]
    full_attention_interval: int
    num_attention_heads: int
    num_key_value_heads: int
    head_dim: int
    linear_num_key_heads: int
    linear_key_head_dim: int
    linear_num_value_heads: int
    linear_value_head_dim: int
    linear_conv_kernel_dim: int
    num_experts: int
    num_experts_per_tok: int
    moe_intermediate_size: int
    shared_expert_intermediate_size: int
    rms_norm_eps: float
    partial_rotary_factor: float
    rope_theta: float
    vocab_size: int

    @classmethod
    def from_json(cls, path: str | Path) -> "ModelConfig":
        """Read the ``text_config`` block of a Hugging Face ``config.json``
        (reference: quickdraw/models/weights.py:149-156)."""
        text = json.loads(Path(path).read_text())["text_config"]
        rope = text.get("rope_parameters", {})
        special = {"partial_rotary_factor": text.get("partial_rotary_factor", 0.25),
                   "rope_theta": rope.get("rope_theta", 1.0e7)}
        plain = {f.name: text[f.name] for f in fields(cls) if f.name not in special}
        return cls(**plain, **special)

    @property
    def conv_channels(self) -> int:
        return (2 * self.linear_num_key_heads * self.linear_key_head_dim
                + self.linear_num_value_heads * self.linear_value_head_dim)

    @property
    def rotary_dim(self) -> int:
        return int(self.head_dim * self.partial_rotary_factor)


@dataclass
class Checkpoint:
    """``lm_head`` is an NVFP4Linear in the published checkpoint and a bf16
    ``[vocab, hidden]`` tensor in the synthetic 36B-A3B model; both are accepted."""
    config: ModelConfig
    embed_tokens: torch.Tensor
    final_norm: torch.Tensor
    lm_head: NVFP4Linear | torch.Tensor
    layers: list[LayerWeights]
    mtp: dict[str, torch.Tensor] = field(default_factory=dict)


# ------------------------------------------------- bf16-weight hybrids (fp32 residual stream)
@dataclass
class WindowAttnConfig:
    """Sliding-window attention with sinks; ``window`` counts the token itself."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    rotary_dims: int
    rotary_base: float
    scale: float

    @property
    def span(self) -> int:
        """The most positions a query sees: rows a cache has to keep."""
        return self.window


@dataclass
class ChunkAttnConfig:
    """Attention within chunks of ``span`` positions counted from 0, with a penalty slope * distance per head and one
    added to the softmax's denominator."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    span: int
    scale: float

    def slopes(self) -> list[float]:
        return [2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads)]


@dataclass
class LatentAttnConfig:
    """Sliding-window attention whose queries, keys and values are expanded from latents; ``dim`` columns per head
    without and ``rot_dim`` with rotary positions, the latter shared by all keys of a token."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    window: int
    rotary_base: float
    scale: float

    @property
    def span(self) -> int:
        return self.window

    @property
    def rot_column(self) -> int:
        """First rotated column of a cache row: behind the latent, on a 16-byte boundary."""
        return -(-self.kv_rank // 8) * 8

    @property
    def row(self) -> int:
        """Elements of a cache row (a multiple of sixteen)."""
        return -(-(self.rot_column + self.rot_dim) // 16) * 16


@dataclass
class GLAConfig:
    """Gated linear attention; decay = sigmoid(z)^(1 / tau) per key channel."""
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass
class ChannelDeltaConfig:
    """Delta rule with one decay per head and key channel, behind short convolutions."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass
class WindowAttnWeights:
    """Names are the tensor names below ``<layer>.mix.``; all bf16."""
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    g: torch.Tensor
    o: torch.Tensor
    q_norm: torch.Tensor
    k_norm: torch.Tensor
    sink: torch.Tensor


@dataclass
class ChunkAttnWeights:
    q: torch.Tensor
    q_b: torch.Tensor
    k: torch.Tensor
    k_b: torch.Tensor
    v: torch.Tensor
    v_b: torch.Tensor
    q_norm: torch.Tensor
    k_norm: torch.Tensor
    o: torch.Tensor
    o_b: torch.Tensor


@dataclass
class LatentAttnWeights:
    dq: torch.Tensor
    dq_norm: torch.Tensor
    uq: torch.Tensor
    dkv: torch.Tensor
    dkv_norm: torch.Tensor
    uk: torch.Tensor
    uv: torch.Tensor
    g: torch.Tensor
    o: torch.Tensor


@dataclass
class GLAWeights:
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    g: torch.Tensor
    o: torch.Tensor
    a1: torch.Tensor
    a2: torch.Tensor
    a2_b: torch.Tensor
    norm: torch.Tensor


@dataclass
class ChannelDeltaWeights:
    q: torch.Tensor
    k: torch.Tensor
    v: torch.Tensor
    b: torch.Tensor
    o: torch.Tensor
    q_conv: torch.Tensor
    k_conv: torch.Tensor
    v_conv: torch.Tensor
    A_log: torch.Tensor
    dt_bias: torch.Tensor
    a1: torch.Tensor
    a2: torch.Tensor
    g1: torch.Tensor
    g2: torch.Tensor
    norm: torch.Tensor


@dataclass
class NormWeights:
    """Layer norm with weight and bias."""
    w: torch.Tensor
    b: torch.Tensor


@dataclass
class SublayerWeights:
    """What surrounds a mixer or a feed-forward: the norm before it, the residual gate
    (sigmoid(gate h + gate_b) on the result, h the normed input) and the norm after it."""
    norm: NormWeights
    gate: torch.Tensor
    gate_b: torch.Tensor
    post: NormWeights


@dataclass
class GeluMLPWeights:
    up: torch.Tensor
    down: torch.Tensor


@dataclass
class HybridLayerWeights:
    idx: int
    mixer: WindowAttnWeights | GLAWeights | ChannelDeltaWeights
    around_mixer: SublayerWeights
    mlp: GeluMLPWeights | None
    around_mlp: SublayerWeights | None
    depth: torch.Tensor          # weights of the depth average: embedding output, then every layer result


@dataclass
class HybridLayerConfig:
    mixer: WindowAttnConfig | GLAConfig | ChannelDeltaConfig
    ff: int | None


@dataclass
class FezopelConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: list[HybridLayerConfig]

    ARCHITECTURE = "Fezopel"

    def runs(self) -> list[tuple[int, None]]:
        """(layer, no pass of a loop), in the order they run."""
        return [(i, None) for i in range(len(self.layers))]

    @classmethod
    def from_json(cls, path: str | Path) -> "FezopelConfig":
        return cls.from_dict(json.loads(Path(path).read_text()))

    @classmethod
    def from_dict(cls, data: dict) -> "FezopelConfig":
        if data.get("architecture") != cls.ARCHITECTURE:
            raise ValueError(f"not a {cls.ARCHITECTURE} configuration: {data.get('architecture')!r}")
        layers = []
        for index, entry in enumerate(data["layers"]):
            m, kind = entry["mixer"], entry["type"]
            if kind == "attention":
                mixer = WindowAttnConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"],
                                         window=m["mask"]["size"], rotary_dims=m["rot"]["dims"],
                                         rotary_base=float(m["rot"]["base"]), scale=float(m["scale"]))
            elif kind == "gla":
                mixer = GLAConfig(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], tau=float(m["tau"]))
            elif kind == "channel_delta":
                mixer = ChannelDeltaConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"],
                                           conv=m["conv"])
            else:
                raise ValueError(f"layer {index}: unknown mixer {kind!r}")
            kv_heads = getattr(mixer, "kv_heads", mixer.heads)
            if mixer.heads % kv_heads:
                raise ValueError(f"layer {index}: {mixer.heads} heads do not divide among {kv_heads} key/value heads")
            mlp = entry["mlp"]
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {index}: unknown feed-forward {mlp['kind']!r}")
            layers.append(HybridLayerConfig(mixer=mixer, ff=None if mlp is None else mlp["ff"]))
        return cls(vocab_size=data["vocab"], hidden_size=data["width"], norm_eps=float(data["norm"]["eps"]), layers=layers)

    def to_dict(self) -> dict:
        """The ``config.json`` this configuration reads from."""
        layers = []
        for layer in self.layers:
            m = layer.mixer
            entry = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
            if isinstance(m, WindowAttnConfig):
                kind = "attention"
                entry |= {"kv_heads": m.kv_heads, "mask": {"size": m.window}, "scale": m.scale,
                          "rot": {"base": m.rotary_base, "dims": m.rotary_dims}}
            elif isinstance(m, GLAConfig):
                kind = "gla"
                entry |= {"tau": m.tau}
            else:
                kind = "channel_delta"
                entry |= {"kv_heads": m.kv_heads, "conv": m.conv}
            layers.append({"type": kind, "mixer": entry,
                           "mlp": None if layer.ff is None else {"kind": "dense", "ff": layer.ff}})
        return {"architecture": self.ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps}, "layers": layers}


@dataclass
class FezopelCheckpoint:
    config: FezopelConfig
    embed_tokens: torch.Tensor
    final_norm: NormWeights
    lm_head: torch.Tensor
    layers: list[HybridLayerWeights]


@dataclass
class ReGLUWeights:
    """down(relu(gate h) * (up h))."""
    gate: torch.Tensor
    up: torch.Tensor
    down: torch.Tensor


@dataclass
class PreNormLayerWeights:
    """RMS norms in front of the mixer and the feed-forward, stored as their distance from one."""
    idx: int
    mixer: LatentAttnWeights | ChunkAttnWeights
    norm1: torch.Tensor
    mlp: ReGLUWeights | None
    norm2: torch.Tensor | None


@dataclass
class PreNormLayerConfig:
    mixer: LatentAttnConfig | ChunkAttnConfig
    ff: int | None


@dataclass
class LoopConfig:
    """Layers start .. stop - 1 run ``times`` times in a row with the same weights and a history of their own each time."""
    start: int
    stop: int
    times: int


@dataclass
class DokulixConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: list[PreNormLayerConfig]
    loop: LoopConfig | None = None

    ARCHITECTURE = "Dokulix"

    def runs(self) -> list[tuple[int, int | None]]:
        """(layer, the pass that begins with it or None), in the order they run."""
        if self.loop is None:
            return [(i, None) for i in range(len(self.layers))]
        start, stop = self.loop.start, self.loop.stop
        looped = [(i, t if i == start else None) for t in range(self.loop.times) for i in range(start, stop)]
        return [(i, None) for i in range(start)] + looped + [(i, None) for i in range(stop, len(self.layers))]

    @classmethod
    def from_json(cls, path: str | Path) -> "DokulixConfig":
        return cls.from_dict(json.loads(Path(path).read_text()))

    @classmethod
    def from_dict(cls, data: dict) -> "DokulixConfig":
        if data.get("architecture") != cls.ARCHITECTURE:
            raise ValueError(f"not a {cls.ARCHITECTURE} configuration: {data.get('architecture')!r}")
        layers = []
        for index, entry in enumerate(data["layers"]):
            m, kind = entry["mixer"], entry["type"]
            if kind == "latent_attention":
                mixer = LatentAttnConfig(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=m["q_rank"],
                                         kv_rank=m["kv_rank"], window=m["mask"]["size"], rotary_base=float(m["rot"]["base"]),
                                         scale=float(m["scale"]))
                if m["rot"]["dims"] != mixer.rot_dim or mixer.rot_dim % 2:
                    raise ValueError(f"layer {index}: {m['rot']['dims']} rotated dimensions of {mixer.rot_dim}")
            elif kind == "attention":
                mixer = ChunkAttnConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], span=m["mask"]["size"],
                                        scale=float(m["scale"]))
                if mixer.heads % mixer.kv_heads:
                    raise ValueError(f"layer {index}: {mixer.heads} heads do not divide among {mixer.kv_heads} key/value heads")
            else:
                raise ValueError(f"layer {index}: unknown mixer {kind!r}")
            mlp = entry["mlp"]
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {index}: unknown feed-forward {mlp['kind']!r}")
            layers.append(PreNormLayerConfig(mixer=mixer, ff=None if mlp is None else mlp["ff"]))
        loop = data.get("loop")
        if loop is not None:
            loop = LoopConfig(start=loop["start"], stop=loop["stop"], times=loop["times"])
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 0:
                raise ValueError(f"loop over layers {loop.start} .. {loop.stop} of {len(layers)}, {loop.times} times")
        return cls(vocab_size=data["vocab"], hidden_size=data["width"], norm_eps=float(data["norm"]["eps"]), layers=layers, loop=loop)

    def to_dict(self) -> dict:
        """The ``config.json`` this configuration reads from."""
        layers = []
        for layer in self.layers:
            m = layer.mixer
            entry = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "mask": {"size": m.span}, "scale": m.scale}
            if isinstance(m, LatentAttnConfig):
                kind = "latent_attention"
                entry |= {"rot_dim": m.rot_dim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
                          "rot": {"base": m.rotary_base, "dims": m.rot_dim}}
            else:
                kind = "attention"
                entry |= {"kv_heads": m.kv_heads}
            layers.append({"type": kind, "mixer": entry, "mlp": None if layer.ff is None else {"kind": "dense", "ff": layer.ff}})
        loop = None if self.loop is None else {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return {"architecture": self.ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps}, "loop": loop, "layers": layers}


@dataclass
class DokulixCheckpoint:
    config: DokulixConfig
    embed_tokens: torch.Tensor
    final_norm: torch.Tensor
    lm_head: torch.Tensor
    layers: list[PreNormLayerWeights]
    loop_steps: torch.Tensor | None          # [times, width]: added to the stream in front of every pass


CONTAINERS = {cls.__name__: cls for cls in (
    NVFP4Linear, FP8Linear, GDNWeights, FullAttnWeights, MoEWeights, LayerWeights,
    ModelConfig, Checkpoint)}
