"""Seeded random-initialised weights, generated full-size and sliced per tensor-parallel rank.

Sharding follows the reference's rules (flash_attn_llm/parallel/tensor_parallel.py:129-146
`chunk(tp_size, dim)[rank]`; shard specs flash_attn_llm/weights/mapper.py:149-184): q/k/v/gate/up are
column-parallel (output rows split; q and k/v by head, so that rank r owns KV heads
[r*H_KV/ws, ...) and the matching query heads, tensor_parallel.py:451-457), o/down are row-parallel
(input columns split), embeddings replicated, the LM head split over the vocabulary.
Every rank draws the same full matrix from the same seed and keeps its slice, so any tensor-parallel
size reproduces the same model.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .config import (ChunkedAttentionSpec, ClampedGluSpec, HybridConfig, LatentAttentionSpec, LightningSpec, Mamba2Spec, MlstmSpec,
                     ModelConfig)


def _randn(shape, gen, std, device, dtype):
    return (torch.randn(shape, generator=gen, device=gen.device, dtype=torch.float32) * std).to(dtype).to(device)


def make_full_layer(cfg: ModelConfig, layer: int, seed: int, gen_device, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    g = torch.Generator(device=gen_device).manual_seed(seed * 100003 + layer)
    H, D = cfg.hidden_size, cfg.head_dim
    return {
        "wq": _randn((cfg.num_heads * D, H), g, cfg.init_std, gen_device, dtype),
        "wk": _randn((cfg.num_kv_heads * D, H), g, cfg.init_std, gen_device, dtype),
        "wv": _randn((cfg.num_kv_heads * D, H), g, cfg.init_std, gen_device, dtype),
        "wo": _randn((H, cfg.num_heads * D), g, cfg.init_std, gen_device, dtype),
        "wg": _randn((cfg.intermediate_size, H), g, cfg.init_std, gen_device, dtype),
        "wu": _randn((cfg.intermediate_size, H), g, cfg.init_std, gen_device, dtype),
        "wd": _randn((H, cfg.intermediate_size), g, cfg.init_std, gen_device, dtype),
        # norm weights: 1 + small noise so that parity tests exercise them
        "ln1": (1.0 + _randn((H,), g, cfg.init_std, gen_device, torch.float32)).to(dtype),
        "ln2": (1.0 + _randn((H,), g, cfg.init_std, gen_device, torch.float32)).to(dtype),
        "qn": (1.0 + _randn((D,), g, cfg.init_std, gen_device, torch.float32)).to(dtype),
        "kn": (1.0 + _randn((D,), g, cfg.init_std, gen_device, torch.float32)).to(dtype),
    }


def make_full_globals(cfg: ModelConfig, seed: int, gen_device, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    g = torch.Generator(device=gen_device).manual_seed(seed * 100003 + 99991)
    return {
        "embed": _randn((cfg.vocab_size, cfg.hidden_size), g, cfg.init_std, gen_device, dtype),
        "lm_head": _randn((cfg.vocab_size, cfg.hidden_size), g, cfg.init_std, gen_device, dtype),
        "final_ln": (1.0 + _randn((cfg.hidden_size,), g, cfg.init_std, gen_device, torch.float32)).to(dtype),
    }


def shard_layer(cfg: ModelConfig, full: Dict[str, torch.Tensor], rank: int, world: int, device) -> Dict[str, torch.Tensor]:
    D = cfg.head_dim
    ql, kl = cfg.num_heads // world, cfg.num_kv_heads // world
    il = cfg.intermediate_size // world
    q0, k0, i0 = rank * ql * D, rank * kl * D, rank * il
    out = {
        # fused column-parallel projection: my q heads, my k heads, my v heads
        "wqkv": torch.cat([full["wq"][q0:q0 + ql * D], full["wk"][k0:k0 + kl * D], full["wv"][k0:k0 + kl * D]]).contiguous(),
        "wo": full["wo"][:, q0:q0 + ql * D].contiguous(),                       # row-parallel
        "wgu": torch.cat([full["wg"][i0:i0 + il], full["wu"][i0:i0 + il]]).contiguous(),
        "wd": full["wd"][:, i0:i0 + il].contiguous(),                           # row-parallel
        "ln1": full["ln1"], "ln2": full["ln2"], "qn": full["qn"], "kn": full["kn"],
    }
    return {k: v.to(device) for k, v in out.items()}


def make_rank_weights(cfg: ModelConfig, rank: int, world: int, seed: int, device, gen_device=None,
                      dtype=torch.bfloat16):
    """Weights of one rank: {'layers': [dict per layer], 'embed', 'lm_head' (vocab shard), 'final_ln'}."""
    cfg.validate(world)
    gen_device = gen_device or device
    layers: List[Dict[str, torch.Tensor]] = []
    for l in range(cfg.num_layers):
        full = make_full_layer(cfg, l, seed, gen_device, dtype)
        layers.append(shard_layer(cfg, full, rank, world, device))
        del full
    glob = make_full_globals(cfg, seed, gen_device, dtype)
    vl = cfg.vocab_size // world
    return {
        "layers": layers,
        "embed": glob["embed"].to(device),
        "lm_head": glob["lm_head"][rank * vl:(rank + 1) * vl].contiguous().to(device),
        "final_ln": glob["final_ln"].to(device),
    }


def rank_weights_from_tensors(cfg: ModelConfig, tensors: Dict[str, torch.Tensor], rank: int, world: int, device):
    """The same per-rank dictionary from named full-size tensors: 'embed', 'lm_head', 'final_ln' and 'l<i>.<name>' with
    the names of `make_full_layer`."""
    cfg.validate(world)
    layers = []
    for l in range(cfg.num_layers):
        pre = f"l{l}."
        full = {k[len(pre):]: t.to(torch.bfloat16) for k, t in tensors.items() if k.startswith(pre)}
        layers.append(shard_layer(cfg, full, rank, world, device))
    vl = cfg.vocab_size // world
    get = lambda n: tensors[n].to(torch.bfloat16)
    return {"layers": layers, "embed": get("embed").to(device), "final_ln": get("final_ln").to(device),
            "lm_head": get("lm_head")[rank * vl:(rank + 1) * vl].contiguous().to(device)}


# ---- hybrid decoders -------------------------------------------------------------------------------------------
def _mixer_shapes(m, W: int) -> Dict[str, tuple]:
    if isinstance(m, LightningSpec):
        kd, vd = m.heads * m.dim, m.heads * m.vdim
        return {"q": (kd, W), "k": (kd, W), "v": (vd, W), "g": (vd, W), "o": (W, vd), "norm": (vd,)}
    if isinstance(m, LatentAttentionSpec):
        H = m.heads
        return {"dq": (m.q_rank, W), "dq.norm": (m.q_rank,), "uq": (H * (m.dim + m.rot_dim), m.q_rank),
                "dkv": (m.kv_rank + m.rot_dim, W), "dkv.norm": (m.kv_rank,), "uk": (H * m.dim, m.kv_rank),
                "uv": (H * m.vdim, m.kv_rank), "g": (H, W), "o": (W, H * m.vdim)}
    if isinstance(m, MlstmSpec):
        kd, vd, H = m.heads * m.dim, m.heads * m.vdim, (m.heads,)
        return {"q": (kd, W), "k": (kd, W), "v": (vd, W), "g": (vd, W), "o": (W, vd), "norm": (vd,),
                "i": H + (W,), "i.b": H, "f": H + (W,), "f.b": H}
    if isinstance(m, Mamba2Spec):
        H = (m.heads,)
        return {"in": (m.inner + m.channels + m.heads, W), "conv": (m.channels, m.conv), "conv.b": (m.channels,), "dt_bias": H, "A_log": H,
                "D": H, "norm": (m.inner,), "o": (W, m.inner)}
    if isinstance(m, ChunkedAttentionSpec):
        qd, kd, vd = m.heads * m.dim, m.kv_heads * m.dim, m.heads * m.vdim
        out = {"q": (qd, W), "k": (kd, W), "v": (m.kv_heads * m.vdim, W), "q.norm": (qd,), "k.norm": (kd,), "g": (vd, W), "o": (W, vd)}
        return dict(out, vmix=()) if m.v_mix else out
    raise TypeError(type(m))


def hybrid_tensor_shapes(cfg: HybridConfig) -> Dict[str, tuple]:
    """Name and shape of every tensor of the model."""
    W = cfg.width
    out = {"embed": (cfg.vocab_size, W), "final.norm": (W,)}
    if cfg.bigram is not None:
        out["bigram"] = (cfg.bigram.buckets + 1, W)
    if cfg.max_positions:
        out["pos"] = (cfg.max_positions, W)
    if cfg.side_dim:
        out["side.embed"] = (cfg.vocab_size, len(cfg.layers) * cfg.side_dim)
    for i, layer in enumerate(cfg.layers):
        pre = f"l{i}."
        out[pre + "norm1"] = (W,)
        out.update({pre + "mix." + k: s for k, s in _mixer_shapes(layer.mixer, W).items()})
        if layer.mlp is not None:
            F = layer.mlp.ff
            gate = {pre + "mlp.gate": (F, W)} if isinstance(layer.mlp, ClampedGluSpec) else {}
            out.update({pre + "norm2": (W,), **gate, pre + "mlp.up": (F, W), pre + "mlp.down": (W, F)})
        if cfg.side_dim:
            out.update({pre + "side.gate": (cfg.side_dim, W), pre + "side.proj": (W, cfg.side_dim), pre + "side.norm": (W,)})
    return out


def random_hybrid_tensors(cfg: HybridConfig, seed: int, device="cpu", dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Seeded random tensors: matrices N(0, 1 / inputs), norm weights 1 + N(0, 0.1^2), embeddings N(0, 1); gate biases 3 + N(0, 0.1^2)
    (forget) and N(0, 0.1^2), step biases around softplus^-1(0.05), decay rates 1 to 16, mixing weights 1 / 2."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in hybrid_tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g, device=device)
        if len(shape) == 0:
            t = torch.tensor(0.5)
        elif name.endswith((".f.b", ".i.b", ".conv.b")):
            t = 0.1 * t + (3.0 if name.endswith(".f.b") else 0.0)
        elif name.endswith(".dt_bias"):
            t = 0.1 * t - 3.0
        elif name.endswith(".A_log"):
            t = torch.rand(shape, generator=g, device=device) * 2.77
        elif len(shape) == 1:
            t = 1.0 + 0.1 * t
        elif name not in ("embed", "side.embed", "bigram", "pos"):
            t = t / shape[1] ** 0.5
        out[name] = t.to(dtype)
    return out


def _stack(mats, multiple: int = 8):
    """Several [n_i, inputs] matrices as one, every block padded with zero rows to a multiple of `multiple` (so that the
    columns of the product stay 16-byte aligned); returns the matrix and the first row of every block."""
    rows, at, n = [], [], 0
    for w in mats:
        at.append(n)
        pad = -w.size(0) % multiple
        rows.append(w)
        if pad:
            rows.append(torch.zeros((pad, w.size(1)), dtype=w.dtype, device=w.device))
        n += w.size(0) + pad
    return torch.cat(rows).contiguous(), tuple(at)


def hybrid_weights(cfg: HybridConfig, tensors: Dict[str, torch.Tensor], dtype, device):
    """The model's tensors in the layout the decoder runs: projections of the same input stacked into one matrix.
    {'embed', 'side_embed', 'bigram', 'pos', 'final_norm', 'layers': [dict per layer]}.  In parallel layers the output projections of
    mixer and feed-forward are one matrix over their activations side by side."""
    want = hybrid_tensor_shapes(cfg)
    unused = {f"l{i}.mix.vmix" for i in range(len(cfg.layers))}           # of a layer that does not mix values
    missing, extra = sorted(set(want) - set(tensors)), sorted(set(tensors) - set(want) - unused)
    if missing or extra:
        raise ValueError(f"tensors do not fit the configuration: missing {missing[:5]}, unknown {extra[:5]}")
    for name, shape in want.items():
        if tuple(tensors[name].shape) != shape:
            raise ValueError(f"{name} has shape {tuple(tensors[name].shape)}, the configuration says {shape}")

    def get(name):
        return tensors[name].to(device=device, dtype=dtype).contiguous()

    layers = []
    for i, layer in enumerate(cfg.layers):
        m, pre = layer.mixer, f"l{i}."
        mix = lambda n: get(pre + "mix." + n)
        f32 = lambda n: tensors[pre + "mix." + n].to(device=device, dtype=torch.float32).contiguous()
        lw = {"norm1": get(pre + "norm1")}
        if isinstance(m, LightningSpec):
            lw["w_in"], lw["in_at"] = _stack([mix(n) for n in ("q", "k", "v", "g")])
            lw["norm"], lw["w_out"] = mix("norm"), mix("o")
            lw["decay"] = torch.tensor(m.decay, dtype=torch.float32, device=device)
        elif isinstance(m, MlstmSpec):
            lw["w_in"], lw["in_at"] = _stack([mix(n) for n in ("q", "k", "v", "g", "i", "f")])
            lw["norm"], lw["w_out"], lw["bias_i"], lw["bias_f"] = mix("norm"), mix("o"), mix("i.b"), mix("f.b")
        elif isinstance(m, Mamba2Spec):
            lw["w_in"], _ = _stack([mix("in")])
            lw["conv_w"], lw["conv_b"] = mix("conv").t().contiguous(), mix("conv.b")
            lw["dt_bias"], lw["a_log"], lw["skip"] = f32("dt_bias"), f32("A_log"), f32("D")
            lw["norm"], lw["w_out"] = mix("norm"), mix("o")
        elif isinstance(m, ChunkedAttentionSpec):
            lw["w_in"], lw["in_at"] = _stack([mix(n) for n in ("q", "k", "v", "g")])
            lw["q_norm"], lw["k_norm"], lw["w_out"] = mix("q.norm"), mix("k.norm"), mix("o")
            lw["lambda"] = float(tensors[pre + "mix.vmix"].float()) if m.v_mix else 0.0
            lw["slopes"] = torch.tensor(m.slopes, dtype=torch.float32, device=device)
        else:
            dkv = mix("dkv")
            lw["w_in"], lw["in_at"] = _stack([mix("dq"), dkv[:m.kv_rank], dkv[m.kv_rank:], mix("g")])
            lw["q_norm"], lw["kv_norm"], lw["w_uq"], lw["w_out"] = mix("dq.norm"), mix("dkv.norm"), mix("uq"), mix("o")
            uk, uv = mix("uk"), mix("uv")
            lw["w_ukv"] = torch.cat([uk, uv]).contiguous()             # expansion of the latents (prompts)
            lw["w_uk"] = lw["w_ukv"][:m.heads * m.dim].view(m.heads, m.dim, m.kv_rank)       # per head (decode)
            lw["w_uv"] = lw["w_ukv"][m.heads * m.dim:].view(m.heads, m.vdim, m.kv_rank)
        if layer.mlp is not None:
            lw["norm2"] = get(pre + "norm2")
            if isinstance(layer.mlp, ClampedGluSpec):
                lw["w_gu"] = torch.cat([get(pre + "mlp.gate"), get(pre + "mlp.up")]).contiguous()
            else:
                lw["w_up"] = get(pre + "mlp.up")
            if cfg.parallel:
                lw["w_out"] = torch.cat([lw["w_out"], get(pre + "mlp.down")], dim=1).contiguous()
            else:
                lw["w_down"] = get(pre + "mlp.down")
        if cfg.side_dim:
            lw["side_gate"], lw["side_proj"], lw["side_norm"] = (get(pre + "side." + n) for n in ("gate", "proj", "norm"))
        layers.append(lw)
    return {"embed": get("embed"), "side_embed": get("side.embed") if cfg.side_dim else None,
            "bigram": get("bigram") if cfg.bigram is not None else None, "pos": get("pos") if cfg.max_positions else None,
            "final_norm": get("final.norm"), "layers": layers}
