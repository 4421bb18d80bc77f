"""Plain CPU restatement of the Sabipel decoder, one function per mechanism.  TEST INFRASTRUCTURE ONLY.

Token-by-token recurrences, full score matrices, no cache, no fusion, no code shared with the engine.  It takes the
model description as the plain dictionary of a config.json and the weights as a name -> tensor dictionary, and works in
the floating-point type it is asked for (float64 unless told otherwise).

Notation: x is the residual row of a token, h a normed row, p a position, S a state matrix, n a normaliser, m the running
maximum of the log weights.
"""
from __future__ import annotations

import math

import torch


def rms_scale(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_scale(x, eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    """log(1 + e^z), without overflow."""
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def log_sigmoid(z):
    return -softplus(-z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- embedding -----------------------------------------------------------------------------------------------
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table for every token of a sequence; its first token has the row behind the buckets."""
    rows = []
    for t, tok in enumerate(tokens):
        rows.append(buckets if t == 0 else (int(tokens[t - 1]) * mul_prev + int(tok) * mul_cur) % buckets)
    return torch.tensor(rows, dtype=torch.long)


def embedding(cfg, w, tokens):
    e = cfg["embedding"]
    tok = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][tok] * e["scale"]
    b = e["bigram"]
    x = x + w["bigram"][bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])]
    return x + w["pos"][: len(tokens)]


# ---- matrix memory with exponential gates ----------------------------------------------------------------------
def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def mlstm_scan(q, k, v, i, f, state=None):
    """q, k [T, H, K], v [T, H, V], log gates i, f [T, H]; returns o [T, H, V] and the state (S, n, m)."""
    T, H, K = q.shape
    V = v.shape[-1]
    if state is None:
        S, n, m = (torch.zeros(s, dtype=q.dtype) for s in ((H, K, V), (H, K), (H,)))
    else:
        S, n, m = (s.clone() for s in state)
    out = torch.empty(T, H, V, dtype=q.dtype)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        num = (S * q[t][:, :, None]).sum(1)
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = num / den[:, None]
    return out, (S, n, m)


def mlstm_mixer(h, w, pre, mix, eps, state=None):
    T, H, K, V, cap = h.shape[0], mix["heads"], mix["dim"], mix["vdim"], mix["gate_cap"]
    q = (h @ w[pre + "q"].T).reshape(T, H, K) * K ** -0.5
    k = (h @ w[pre + "k"].T).reshape(T, H, K)
    v = (h @ w[pre + "v"].T).reshape(T, H, V)
    i = soft_cap(h @ w[pre + "i"].T + w[pre + "i.b"], cap)
    f = log_sigmoid(soft_cap(h @ w[pre + "f"].T + w[pre + "f.b"], cap))
    o, state = mlstm_scan(q, k, v, i, f, state)
    o = rms_scale(o, eps).reshape(T, H * V) * w[pre + "norm"] * sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T, state


# ---- state-space duality -----------------------------------------------------------------------------------------
def causal_conv(u, w, b, before=None):
    """Per-channel convolution of u [T, C] with w [C, taps] (last column: the current token) and bias b; `before`
    [taps - 1, C] are the inputs ahead of the first token (zeros by default)."""
    taps = w.shape[1]
    if before is None:
        before = torch.zeros(taps - 1, u.shape[1], dtype=u.dtype)
    ext = torch.cat([before, u])
    out = b.expand(u.shape[0], -1).clone()
    for j in range(taps):
        out = out + ext[j:j + u.shape[0]] * w[:, j]
    return out


def ssd_scan(x, B, C, dt, A_log, D, state=None):
    """x [T, H, V], B, C [T, G, N], dt [T, H] (after softplus); returns y [T, H, V] and the state [H, N, V]."""
    T, H, V = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, V, dtype=x.dtype) if state is None else state.clone()
    y = torch.empty_like(x)
    group = torch.tensor([h // (H // G) for h in range(H)])
    for t in range(T):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][group][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t][group][:, :, None]).sum(1) + D[:, None] * x[t]
    return y, S


def mamba2_mixer(h, w, pre, mix, eps):
    T, H, V, N, G, parts = h.shape[0], mix["heads"], mix["vdim"], mix["state"], mix["groups"], mix["norm_groups"]
    inner = H * V
    z, u, dt = torch.split(h @ w[pre + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    u = silu(causal_conv(u, w[pre + "conv"], w[pre + "conv.b"]))
    x, B, C = torch.split(u, [inner, G * N, G * N], dim=1)
    dt = softplus(dt + w[pre + "dt_bias"])
    y, _ = ssd_scan(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), dt, w[pre + "A_log"], w[pre + "D"])
    y = y.reshape(T, inner) * silu(z)
    y = rms_scale(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * w[pre + "norm"]
    return y @ w[pre + "o"].T


# ---- chunked attention with a distance bias ------------------------------------------------------------------------
def slopes(heads, dtype):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=dtype)


def chunk_mask(T, size):
    """[T, T]: query i sees key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def biased_attention(q, k, v, scale, size):
    """q [T, H, K], k [T, G, K], v [T, G, V]; the distance times the head's slope is taken off the score."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    k, v = k.repeat_interleave(rep, 1), v.repeat_interleave(rep, 1)
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(q.dtype)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale - slopes(H, q.dtype)[:, None, None] * dist
    s = s.masked_fill(~chunk_mask(T, size), float("-inf"))
    s = torch.exp(s - s.max(-1, keepdim=True).values)
    return torch.einsum("hij,jhd->ihd", s / s.sum(-1, keepdim=True), v)


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention_mixer(h, w, pre, mix, eps, v_first):
    """Returns the mixer's output and the values of the first value-mixing layer (`v_first`, or this layer's own)."""
    T, H, G, K, V = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = rms_norm(h @ w[pre + "q"].T, w[pre + "q.norm"], eps).reshape(T, H, K)
    k = rms_norm(h @ w[pre + "k"].T, w[pre + "k.norm"], eps).reshape(T, G, K)
    v = h @ w[pre + "v"].T
    if mix.get("v_mix"):
        if v_first is None:
            v_first = v
        else:
            v = mix_values(v, v_first, w[pre + "vmix"])
    o = biased_attention(q, k, v.reshape(T, G, V), mix["scale"], mix["mask"]["size"]).reshape(T, H * V)
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T, v_first


def dense(h, w, pre):
    return gelu_tanh(h @ w[pre + "up"].T) @ w[pre + "down"].T


@torch.no_grad()
def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """tokens: list of ids of ONE sequence -> logits [T, vocab].  `layers_out` (a list) receives the residual rows
    after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embedding(cfg, w, list(tokens))
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        h = rms_norm(x, w[pre + "norm1"], eps)
        if layer["type"] == "mlstm":
            y = mlstm_mixer(h, w, pre + "mix.", layer["mixer"], eps)[0]
        elif layer["type"] == "mamba2":
            y = mamba2_mixer(h, w, pre + "mix.", layer["mixer"], eps)
        elif layer["type"] == "attention":
            y, v_first = attention_mixer(h, w, pre + "mix.", layer["mixer"], eps, v_first)
        else:
            raise ValueError(layer["type"])
        if layer["mlp"] is not None:
            y = y + dense(rms_norm(x, w[pre + "norm2"], eps), w, pre + "mlp.")
        x = x + y
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
