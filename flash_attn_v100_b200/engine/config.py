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
class ClampedGluSpec:
    """g sigmoid(1.702 g) (u + 1) with g and u clamped at `limit`."""
    ff: int
    limit: float

    def validate(self) -> None:
        _positive(self, "ff")


@dataclass(frozen=True)
class HybridLayer:
    mixer: Union[LightningSpec, LatentAttentionSpec]
    mlp: Optional[ClampedGluSpec]


@dataclass(frozen=True)
class HybridConfig:
    """A decoder whose layers each name their mixer and feed-forward.  The range [loop_start, loop_stop) is passed through
    `loop_times` times with shared weights; passes share nothing they keep per request, and from the second one on the residual
    first receives the token embeddings again."""
    vocab_size: int
    width: int
    layers: Tuple[HybridLayer, ...]
    norm_eps: float
    side_dim: int = 0        # per-layer width of the token side embedding (0: none)
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1

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


_MIXER_SPECS = {"lightning": _lightning, "latent_attention": _latent_attention}


def _layer(d: dict) -> HybridLayer:
    if d["type"] not in _MIXER_SPECS:
        raise ValueError(f"unknown mixer {d['type']!r}; known: {sorted(_MIXER_SPECS)}")
    mlp = d.get("mlp")
    if mlp is not None:
        if mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward {mlp['kind']!r}; known: dense")
        mlp = ClampedGluSpec(int(mlp["ff"]), float(mlp["limit"]))
    return HybridLayer(_MIXER_SPECS[d["type"]](d["mixer"]), mlp)
