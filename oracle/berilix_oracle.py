"""Plain CPU restatement of the Berilix decoder, one function per mechanism.  TEST INFRASTRUCTURE ONLY.

Token-by-token recurrences, full score matrices, no cache, no fusion, no code shared with the engine.  It takes the
model description as the plain dictionary of a config.json and the weights as a name -> tensor dictionary, and works in
the floating-point type it is asked for (float64 unless told otherwise).

Notation: x is the residual row of a token, h a normed row, p a position, d a decay, S a state matrix.
"""
from __future__ import annotations

import math

import torch


def rms_scale(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_scale(x, eps) * w


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(vec, positions, base, dims):
    """Rotary embedding of the first `dims` entries of the last axis: entry i pairs with entry i + dims/2 and the pair
    turns by p * base^(-2i/dims).  vec [T, ..., n], positions [T]."""
    half = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=vec.dtype)
    a = positions.to(vec.dtype)[:, None] * f[None, :]
    a = a.reshape([a.shape[0]] + [1] * (vec.dim() - 2) + [half])
    u, v = vec[..., :half], vec[..., half:dims]
    return torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), vec[..., dims:]], dim=-1)


def linear_attention_scan(q, k, v, decay, state=None):
    """S <- d S + k v^T, o = S^T q, one token after the other.  q, k [T, H, K], v [T, H, V], decay [H];
    returns o [T, H, V] and the final state [H, K, V]."""
    T, H, K = q.shape
    V = v.shape[-1]
    s = torch.zeros(H, K, V, dtype=q.dtype) if state is None else state.clone()
    out = torch.empty(T, H, V, dtype=q.dtype)
    d = decay.to(q.dtype)[:, None, None]
    for t in range(T):
        s = d * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (s * q[t][:, :, None]).sum(1)
    return out, s


def lightning_mixer(h, w, pre, m, eps, state=None):
    """Decayed linear attention.  Returns the mixer's output and the state it leaves behind."""
    T, H, K, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[pre + "q"].T).reshape(T, H, K)
    k = silu(h @ w[pre + "k"].T).reshape(T, H, K)
    v = silu(h @ w[pre + "v"].T).reshape(T, H, V)
    o, s = linear_attention_scan(q, k, v, torch.tensor(m["decay"], dtype=torch.float64), state)
    o = rms_norm(o.reshape(T, H * V), w[pre + "norm"], eps) * sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T, s


def causal_attention(q, k, v, scale):
    """q, k [T, H, K], v [T, H, V]: softmax over the keys at and before each query."""
    T = q.shape[0]
    s = torch.einsum("thd,shd->hts", q, k) * scale
    s = s.masked_fill(torch.triu(torch.ones(T, T, dtype=torch.bool), 1), float("-inf"))
    s = torch.exp(s - s.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    return torch.einsum("hts,shv->thv", s, v)


def latent_attention_mixer(h, w, pre, m, eps, positions):
    """Attention whose keys and values are expanded from one low-rank row per token plus one rotated key part that all
    heads share."""
    T, H, K, R, V, L = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    q = (rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T).reshape(T, H, K + R)
    down = h @ w[pre + "dkv"].T
    c = rms_norm(down[:, :L], w[pre + "dkv.norm"], eps)
    kr = rotate(down[:, L:], positions, base, R)
    qr = rotate(q[..., K:], positions, base, R)
    q = torch.cat([q[..., :K], qr], -1)
    k = torch.cat([(c @ w[pre + "uk"].T).reshape(T, H, K), kr[:, None, :].expand(T, H, R)], -1)
    v = (c @ w[pre + "uv"].T).reshape(T, H, V)
    o = causal_attention(q, k, v, m["scale"])
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ w[pre + "o"].T


def clamped_glu(h, w, pre, limit):
    """Gated feed-forward with both branches clamped and the linear branch shifted by one."""
    g = torch.clamp(h @ w[pre + "gate"].T, max=limit)
    u = torch.clamp(h @ w[pre + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T


def token_side_input(x, w, pre, e, eps):
    """What a layer adds for the token itself: e is the layer's part of the token's side embedding."""
    y = (gelu_tanh(x @ w[pre + "gate"].T) * e) @ w[pre + "proj"].T
    return rms_norm(y, w[pre + "norm"], eps)


def layer_runs(cfg):
    """Order in which the layers run: (layer, the embedding output is added first)."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, False) for i in range(a)]
    for t in range(times):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


@torch.no_grad()
def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """tokens: list of ids of ONE sequence -> logits [T, vocab].  `layers_out` (a list) receives the residual rows
    after every layer run."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    tok = torch.as_tensor(tokens, dtype=torch.long)
    pos = torch.arange(tok.numel())
    x0 = w["embed"][tok]
    x = x0.clone()
    side = cfg.get("token_side")
    for i, again in layer_runs(cfg):
        layer, pre = cfg["layers"][i], f"l{i}."
        if again:
            x = x + x0
        h = rms_norm(x, w[pre + "norm1"], eps)
        if layer["type"] == "lightning":
            x = x + lightning_mixer(h, w, pre + "mix.", layer["mixer"], eps)[0]
        elif layer["type"] == "latent_attention":
            x = x + latent_attention_mixer(h, w, pre + "mix.", layer["mixer"], eps, pos)
        else:
            raise ValueError(layer["type"])
        if layer["mlp"] is not None:
            x = x + clamped_glu(rms_norm(x, w[pre + "norm2"], eps), w, pre + "mlp.", layer["mlp"]["limit"])
        if side is not None:
            n = side["dim"]
            x = x + token_side_input(x, w, pre + "side.", w["side.embed"][tok][:, i * n:(i + 1) * n], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


@torch.no_grad()
def greedy_generate(cfg, weights, prompt, max_new_tokens, dtype=torch.float64):
    """Greedy continuation of one prompt (the whole sequence is run again for every token)."""
    toks, rows = list(prompt), []
    for _ in range(max_new_tokens):
        logits = forward(cfg, weights, toks, dtype)[-1]
        rows.append(logits)
        toks.append(int(logits.argmax()))
    return toks[len(prompt):], torch.stack(rows)
