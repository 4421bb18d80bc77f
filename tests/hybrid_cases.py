"""Small hybrid decoders for the tests: configurations (as the dictionaries of a config.json) and seeded random weights."""
import torch


def lightning(heads, dim, vdim, decay=None):
    if decay is None:
        decay = [1.0 - 2.0 ** (-1.5 - 1.7 * h) for h in range(heads)]
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, base=1000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
            "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}


def layer(mixer, ff=None, limit=1.5):
    return {"type": "latent_attention" if "kv_rank" in mixer else "lightning", "mixer": mixer,
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers, vocab=160, width=96, side=8, loop=None, eps=1e-5):
    c = {"architecture": "Berilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if side:
        c["token_side"] = {"dim": side}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def small_config():
    """Sizes the tensor-core kernels take, all different; a loop in the middle; a layer without a feed-forward."""
    return config([layer(lightning(3, 32, 48), 80), layer(latent(3, 40, 16, 56, 48, 64), None),
                   layer(lightning(2, 72, 96), 112, 0.7), layer(latent(5, 24, 8, 16, 72, 40, base=50.0), 64)],
                  loop=(1, 3, 3))


def odd_config():
    """Sizes that only the general kernels take (nothing a multiple of eight)."""
    return config([layer(latent(3, 10, 6, 14, 22, 18), 30), layer(lightning(3, 9, 13), 27), layer(lightning(1, 5, 34), None)],
                  vocab=77, width=50, side=5, loop=(0, 2, 2))


def plain_config():
    """No loop, no token side input."""
    return config([layer(lightning(4, 16, 16), 48), layer(latent(2, 16, 16, 16, 32, 24), 48)], side=0)


def weights(cfg, seed=0, dtype=torch.bfloat16):
    from flash_attn_v100_b200.engine.config import HybridConfig
    from flash_attn_v100_b200.engine.weights import hybrid_tensor_shapes
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in hybrid_tensor_shapes(HybridConfig.from_dict(cfg)).items():
        t = torch.randn(shape, generator=g)
        if len(shape) == 1:
            t = 1.0 + 0.2 * t
        elif not name.endswith("embed"):
            t = t / shape[1] ** 0.5
        out[name] = t.to(dtype)
    return out


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def model(cfg, w, dtype=torch.float32, device="cuda"):
    from flash_attn_v100_b200.engine import HybridDecoder, hybrid_weights
    from flash_attn_v100_b200.engine.config import HybridConfig
    c = HybridConfig.from_dict(cfg)
    return HybridDecoder(c, hybrid_weights(c, w, dtype, device), device)


def write_model(cfg, w, folder):
    import json
    import os
    from flash_attn_v100_b200.engine import safetensors
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    safetensors.save_file(w, os.path.join(folder, "model.safetensors"))
