"""Model shapes: the Qwen3-style decoder (the reference's `ModelConfig`, flash_attn_llm/models/config.py:7-104, reduced to what
a Qwen3-style decoder needs) and the hybrid decoders, whose layers name their own mixers."""
from __future__ import annotations

from dataclasses import dataclass, fields
from typing import List, Optional, Tuple, Union


@dataclass(frozen=True)
class ModelConfig:
    num_layers: int
    hidden_size: int
    num_heads: int
    num_kv_heads: int
    head_dim: int
    intermediate_size: int
    vocab_size: int
    rms_norm_eps: float = 1e-6
    rope_theta: float = 1e6
    qk_norm: bool = True          # per-head RMSNorm on q and k (Qwen3)
    init_std: float = 0.02

    def validate(self, world: int) -> None:
        if self.num_heads % self.num_kv_heads:
            raise ValueError("num_heads must be divisible by num_kv_heads")
        for name, v in (("num_heads", self.num_heads), ("num_kv_heads", self.num_kv_heads),
                        ("intermediate_size", self.intermediate_size), ("vocab_size", self.vocab_size)):
            if v % world:
                raise ValueError(f"{name}={v} must be divisible by the tensor-parallel size {world}")
        if self.head_dim not in (64, 128, 256):
            raise ValueError("head_dim must be 64, 128 or 256")

    @classmethod
    def from_dict(cls, d: dict) -> "ModelConfig":
        cfg = cls(**{f.name: d[f.name] for f in fields(cls) if f.name in d})
        cfg.validate(1)
        return cfg


def qwen3_8b_shaped() -> ModelConfig:
    """36 layers, hidden 4096, 32 query / 8 KV heads of 128, SwiGLU 12288, vocabulary 151936."""
    return ModelConfig(num_layers=36, hidden_size=4096, num_heads=32, num_kv_heads=8, head_dim=128,
                       intermediate_size=12288, vocab_size=151936)


def tiny_config() -> ModelConfig:
    """Small shape for parity tests (same structure, divisible by 2 for TP=2)."""
    return ModelConfig(num_layers=2, hidden_size=256, num_heads=8, num_kv_heads=2, head_dim=64,
                       intermediate_size=512, vocab_size=1024)


# ---- hybrid decoders: layers with different sequence mixers ----------------------------------------------------
@dataclass(frozen=True)
class LightningSpec:
    """Decayed linear attention: per head a state [dim, vdim] with its own decay."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    def validate(self) -> None:
        _positive(self, "heads", "dim", "vdim")
        if len(self.decay) != self.heads:
            raise ValueError(f"lightning: {len(self.decay)} decays for {self.heads} heads")


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention on one cached latent row per token (`kv_rank` + `rot_dim` elements for all heads)."""
    heads: int
    dim: int                 # unrotated query / key dimensions per head
    rot_dim: int             # rotated ones
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float

    def validate(self) -> None:
        _positive(self, "heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")
        if self.rot_dim % 2:
            raise ValueError("latent_attention: rot_dim must be even")


@dataclass(frozen=True)
class MlstmSpec:
    """Matrix memory with exponential gates: per head a state [dim, vdim], a normaliser [dim] and a running maximum."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float          # both gate logits are cap tanh(. / cap)

    def validate(self) -> None:
        _positive(self, "heads", "dim", "vdim", "gate_cap")


@dataclass(frozen=True)
class Mamba2Spec:
    """State-space duality: a short convolution, per head a state [state, vdim] with a decay that depends on the token; the heads
    of a group share its input and output vectors."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                # taps of the convolution, the current token's included
    norm_groups: int         # equal parts of the output that are normed on their own

    def validate(self) -> None:
        _positive(self, "heads", "vdim", "state", "groups", "conv", "norm_groups")
        if self.heads % self.groups:
            raise ValueError(f"mamba2: {self.heads} heads are not whole groups of {self.groups}")
        if self.inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.inner} columns do not make {self.norm_groups} equal parts")

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Of the convolution: the heads' values, and the input and output vectors of every group."""
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class ChunkedAttentionSpec:
    """Grouped-query attention inside chunks of the sequence, with a distance bias per head and an element-wise output gate."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int                       # position i sees the keys from i - i % chunk on
    slopes: Tuple[float, ...]        # per head, taken off the score for every position of distance
    v_mix: bool = False              # mix in the values of the first layer that says so

    def validate(self) -> None:
        _positive(self, "heads", "kv_heads", "dim", "vdim", "chunk")
        if self.heads % self.kv_heads:
            raise ValueError("attention: heads must be divisible by kv_heads")
        if len(self.slopes) != self.heads:
            raise ValueError(f"attention: {len(self.slopes)} slopes for {self.heads} heads")


@dataclass(frozen=True)
class GeluSpec:
    """W_down gelu(W_up h), gelu in its tanh form."""
    ff: int

    def validate(self) -> None:
        _positive(self, "ff")


@dataclass(frozen=True)
class BigramSpec:
    """Embedding of (previous token, token): row (previous * mul_prev + token * mul_cur) mod buckets, row `buckets` for the first."""
    buckets: int
    mul_prev: int
    mul_cur: int

    def validate(self) -> None:
        _positive(self, "buckets")
        if not 0 <= self.mul_prev < 2 ** 31 or not 0 <= self.mul_cur < 2 ** 31:
            raise ValueError("bigram: the multipliers must be non-negative 32-bit numbers")


@dataclass(frozen=True)
class ClampedGluSpec:
    """g sigmoid(1.702 g) (u + 1) with g and u clamped at `limit`."""
    ff: int
    limit: float

    def validate(self) -> None:
        _positive(self, "ff")


@dataclass(frozen=True)
class HybridLayer:
    mixer: Union[LightningSpec, LatentAttentionSpec, MlstmSpec, Mamba2Spec, ChunkedAttentionSpec]
    mlp: Optional[Union[ClampedGluSpec, GeluSpec]]


@dataclass(frozen=True)
class HybridConfig:
    """A decoder whose layers each name their mixer and feed-forward.  The range [loop_start, loop_stop) is passed through
    `loop_times` times with shared weights; passes share nothing they keep per request, and from the second one on the residual
    first receives the token embeddings again.  `parallel`: mixer and feed-forward read (differently normed) the same residual and
    their outputs are added to it together."""
    vocab_size: int
    width: int
    layers: Tuple[HybridLayer, ...]
    norm_eps: float
    side_dim: int = 0        # per-layer width of the token side embedding (0: none)
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    parallel: bool = False
    embed_scale: float = 1.0
    bigram: Optional[BigramSpec] = None
    max_positions: int = 0   # rows of the learned position table (0: there is none)

    def validate(self) -> None:
        _positive(self, "vocab_size", "width", "loop_times")
        if not self.layers:
            raise ValueError("the model has no layers")
        if not 0 <= self.loop_start <= self.loop_stop <= len(self.layers):
            raise ValueError(f"loop {self.loop_start}..{self.loop_stop} is not inside the {len(self.layers)} layers")
        for layer in self.layers:
            layer.mixer.validate()
            if layer.mlp is not None:
                layer.mlp.validate()
        if self.bigram is not None:
            self.bigram.validate()
        if self.loop_times > 1 and (self.bigram is not None or self.max_positions or self.embed_scale != 1.0):
            raise ValueError("a loop adds the plain token embeddings again: it does not go with a scaled or summed embedding")
        values = {l.mixer.kv_heads * l.mixer.vdim for l in self.layers if isinstance(l.mixer, ChunkedAttentionSpec) and l.mixer.v_mix}
        if len(values) > 1:
            raise ValueError(f"layers that mix values must have values of the same size, got {sorted(values)}")

    def runs(self) -> List[Tuple[int, bool]]:
        """(layer index, add the embedding output first) of every layer run, in order."""
        out = [(i, False) for i in range(self.loop_start)]
        for t in range(self.loop_times):
            out += [(i, t > 0 and i == self.loop_start) for i in range(self.loop_start, self.loop_stop)]
        return out + [(i, False) for i in range(self.loop_stop, len(self.layers))]

    @classmethod
    def from_dict(cls, d: dict) -> "HybridConfig":
        loop = d.get("loop") or {}
        side = d.get("token_side") or {}
        cfg = cls(vocab_size=int(d["vocab"]), width=int(d["width"]), layers=tuple(_layer(x) for x in d["layers"]),
                  norm_eps=float(d["norm"]["eps"]), side_dim=int(side.get("dim", 0)), loop_start=int(loop.get("start", 0)),
                  loop_stop=int(loop.get("stop", 0)), loop_times=int(loop.get("times", 1)))
        cfg.validate()
        return cfg


def _positive(obj, *names) -> None:
    for n in names:
        if getattr(obj, n) <= 0:
            raise ValueError(f"{type(obj).__name__}.{n} must be positive, got {getattr(obj, n)}")


def _lightning(m: dict) -> LightningSpec:
    return LightningSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), tuple(float(x) for x in m["decay"]))


def _latent_attention(m: dict) -> LatentAttentionSpec:
    rot = m["rot"]
    if int(rot["dims"]) != int(m["rot_dim"]):
        raise ValueError("latent_attention rotates its whole rotated part: rot.dims must equal rot_dim")
    return LatentAttentionSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["q_rank"]),
                               int(m["kv_rank"]), float(m["scale"]), float(rot["base"]))


def _mlstm(m: dict) -> MlstmSpec:
    return MlstmSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))


def _mamba2(m: dict) -> Mamba2Spec:
    return Mamba2Spec(int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["conv"]), int(m["norm_groups"]))


def power_of_two_slopes(heads: int) -> Tuple[float, ...]:
    """2^(-8 (h + 1) / heads) of every head h."""
    return tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads))


def _chunked_attention(m: dict) -> ChunkedAttentionSpec:
    heads = int(m["heads"])
    return ChunkedAttentionSpec(heads, int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), int(m["mask"]["size"]),
                                power_of_two_slopes(heads), bool(m.get("v_mix", False)))


_MIXER_SPECS = {"lightning": _lightning, "latent_attention": _latent_attention}
_SABIPEL_MIXERS = {"mlstm": _mlstm, "mamba2": _mamba2, "attention": _chunked_attention}


def _clamped_glu(m: dict) -> ClampedGluSpec:
    return ClampedGluSpec(int(m["ff"]), float(m["limit"]))


def _gelu(m: dict) -> GeluSpec:
    return GeluSpec(int(m["ff"]))


def _layer(d: dict, mixers=_MIXER_SPECS, dense=_clamped_glu) -> HybridLayer:
    """`mixers`: reader of every mixer the design has; `dense`: reader of its feed-forward."""
    if d["type"] not in mixers:
        raise ValueError(f"unknown mixer {d['type']!r}; known: {sorted(mixers)}")
    mlp = d.get("mlp")
    if mlp is not None:
        if mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward {mlp['kind']!r}; known: dense")
        mlp = dense(mlp)
    return HybridLayer(mixers[d["type"]](d["mixer"]), mlp)


def sabipel_config(d: dict) -> HybridConfig:
    """Parallel layers of exponential-gate memories, state-space recurrences and chunked attention; embeddings of the token (scaled),
    of the token pair and of the position."""
    e = d["embedding"]
    b = e.get("bigram")
    bigram = BigramSpec(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b is not None else None
    cfg = HybridConfig(vocab_size=int(d["vocab"]), width=int(d["width"]), layers=tuple(_layer(x, _SABIPEL_MIXERS, _gelu) for x in d["layers"]),
                       norm_eps=float(d["norm"]["eps"]), parallel=True, embed_scale=float(e.get("scale", 1.0)), bigram=bigram,
                       max_positions=int(d["max_positions"]))
    cfg.validate()
    return cfg
