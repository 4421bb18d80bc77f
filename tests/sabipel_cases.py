"""Small Sabipel decoders for the tests: configurations (as the dictionaries of a config.json) and seeded random weights."""
import torch


def mlstm(heads, dim, vdim, cap=10.0):
    return "mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def mamba2(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return "mamba2", {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def attention(heads, kv_heads, dim, vdim, size, v_mix=True, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                         "mask": {"size": size}, "v_mix": v_mix}


def config(layers, vocab=160, width=96, eps=1e-5, scale=3.0, bigram=(101, 17, 5), positions=700):
    """layers: (mixer, ff or None)."""
    return {"architecture": "Sabipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "max_positions": positions,
            "embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))},
            "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (t, m), ff in layers]}


def small_config():
    """Sizes the tensor-core kernels take, all different; every mixer twice; layers without a feed-forward; an attention layer without
    value mixing ahead of the first that mixes."""
    return config([(attention(6, 3, 40, 24, 64, v_mix=False), 80), (mlstm(3, 32, 48), 112), (mamba2(4, 24, 40, groups=2, conv=4, norm_groups=2), None),
                   (attention(4, 2, 24, 16, 50), 64), (mamba2(6, 8, 16, groups=1, conv=2, norm_groups=3), 48), (mlstm(2, 64, 16, cap=4.0), None),
                   (attention(8, 2, 16, 16, 33), 40)])


def odd_config():
    """Sizes that only the general kernels take (nothing a multiple of eight); one tap, one group per head."""
    return config([(mlstm(3, 9, 13), 27), (attention(3, 1, 10, 14, 37), 30), (mamba2(3, 5, 7, groups=3, conv=1, norm_groups=5), None),
                   (mamba2(2, 11, 6, groups=1, conv=5), 21), (attention(5, 1, 6, 14, 29), None)], vocab=77, width=50, scale=0.5, bigram=(7, 3, 0))


def wide_config():
    """Heads of the sizes real models have: two heads per tile, 128 columns, more than one column tile, more than eight query heads per
    key."""
    return config([(mamba2(8, 64, 128, groups=2, conv=4, norm_groups=2), 64), (mlstm(2, 128, 256), 96), (attention(12, 1, 128, 64, 80), 64),
                   (mlstm(2, 128, 128), 64), (attention(4, 1, 64, 64, 128), None)], width=128)


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Seeded random weights: forget gates and decays spread from closed to open, so that states of every length of memory occur."""
    from flash_attn_v100_b200.engine.config import sabipel_config
    from flash_attn_v100_b200.engine.weights import hybrid_tensor_shapes
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in hybrid_tensor_shapes(sabipel_config(cfg)).items():
        t = torch.randn(shape, generator=g)
        if name.endswith(".vmix"):
            t = torch.tensor(0.25 + 0.5 * torch.rand((), generator=g).item())
        elif name.endswith(".f.b"):
            t = 2.0 + 2.0 * t
        elif name.endswith((".i.b", ".conv.b", ".D")):
            t = 0.5 * t
        elif name.endswith(".dt_bias"):
            t = t - 2.0
        elif name.endswith(".A_log"):
            t = 0.7 * t
        elif len(shape) == 1:
            t = 1.0 + 0.2 * t
        elif name.endswith(".conv"):
            t = t / shape[1] ** 0.5
        elif name == "pos":
            t = 0.5 * t
        elif name not in ("embed", "bigram"):
            t = t / shape[1] ** 0.5
        out[name] = t.to(dtype)
    return out


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(2000 + seed)).tolist()


def model(cfg, w, dtype=torch.float32, device="cuda"):
    from flash_attn_v100_b200.engine import HybridDecoder, hybrid_weights
    from flash_attn_v100_b200.engine.config import sabipel_config
    c = sabipel_config(cfg)
    return HybridDecoder(c, hybrid_weights(c, w, dtype, device), device)


def write_model(cfg, w, folder):
    import json
    import os
    from flash_attn_v100_b200.engine import safetensors
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    safetensors.save_file(w, os.path.join(folder, "model.safetensors"))
