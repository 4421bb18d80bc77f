"""Decoder whose layers each name their sequence mixer and feed-forward (`HybridConfig`).

A layer run is x += mixer(norm1(x)); x += mlp(norm2(x)); x += rmsnorm(proj(gelu(gate x) * side[token])) — the last two only
where the configuration has them — or, in parallel layers, x += mixer(norm1(x)) + mlp(norm2(x)) of the same x: one kernel norms x
with both weights, and the two output projections are one product over the activations of mixer and feed-forward side by side.
The residual x is fp32 throughout; h, the activations and the cached rows are the model's type (bfloat16, or float32 with
every product in 32 bits).  Matrix products go to cuBLAS through torch; everything between them is libfa_b200_rows,
libfa_b200_hybrid and libfa_b200_mixers.  An update of x is not applied by a kernel of its own: it is left pending and the next
norm's kernel adds it.

Mixers are classes with the same four members (see `LightningMixer`), looked up by the type of their spec; what a mixer keeps
between calls is described by `store` and lives in `HybridCache.stores`, one entry per layer run.
"""
from __future__ import annotations

import itertools
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from .. import hybrid_ops as hops
from .. import mixer_ops as mops
from .. import row_ops as rops
from ..kv_cache import BLOCK_SIZE, HybridCache
from .config import ChunkedAttentionSpec, GeluSpec, HybridConfig, LatentAttentionSpec, LightningSpec, Mamba2Spec, MlstmSpec
from .model import GreedyHead, Segments

GLU_ALPHA, GLU_SHIFT = 1.702, 1.0      # g sigmoid(1.702 g) (u + 1)
NORMALISER_EPS = 1e-6                  # added to the denominator of the exponential-gate memory

# Prompts of at least this many tokens per sequence run on the prompt attention kernels; shorter portions and decode steps work
# on the pages, row by row.
PROMPT_TOKENS = 32


@dataclass
class Pieces:
    """A pass's sequences cut at the borders of chunks: what a piece's queries see are keys of the piece, all before their own."""
    cu_q: torch.Tensor                   # [n + 1] int32
    cu_kv: torch.Tensor                  # [n + 1] int32; a piece's keys begin at its chunk's first position
    seq: torch.Tensor                    # [n] int32
    key0: torch.Tensor                   # [n] int32, position of the first key
    max_q: int
    total_kv: int
    fresh: bool                          # all keys are tokens of this pass


@dataclass
class Step:
    """One pass over the packed tokens of a batch: whole prompts, portions of prompts, or one token per sequence."""
    tokens: torch.Tensor                 # [T] int64
    positions: torch.Tensor              # [T] int32, place in the token's sequence (= its cache slot)
    starts: torch.Tensor                 # [n_seq] int32, position of the sequence's first token in this pass
    cu: Optional[torch.Tensor]           # [n_seq + 1] int32; None: one token per sequence
    tok_seq: torch.Tensor                # [T] int32, sequence of every token
    state_rows: torch.Tensor             # [n_seq] int32, state slot of every sequence
    block_table: torch.Tensor            # [n_seq, max_blocks] int32
    lens: Optional[List[int]]            # host: new tokens per sequence (None: one each)
    past: Optional[List[int]]            # host: cached tokens per sequence (prompts only)
    cu_kv: Optional[torch.Tensor]        # [n_seq + 1] int32 offsets of all the sequences' keys (prompts only)
    status: torch.Tensor
    values_first: Optional[torch.Tensor] = None      # [T, n] values of the first layer that mixes values
    _pieces: Dict[int, Pieces] = field(default_factory=dict)

    def sequences(self) -> mops.Sequences:
        return mops.Sequences(self.state_rows, self.starts, self.cu, max(self.lens) if self.cu is not None else 1)

    def pieces(self, chunk: int) -> Pieces:
        """The prompts of this pass cut at multiples of `chunk` positions."""
        if chunk not in self._pieces:
            cu_q, cu_kv, seq, key0 = [0], [0], [], []
            for i, (past, n) in enumerate(zip(self.past, self.lens)):
                at = past
                while at < past + n:
                    first = at - at % chunk
                    end = min(first + chunk, past + n)
                    cu_q.append(cu_q[-1] + end - at)
                    cu_kv.append(cu_kv[-1] + end - first)
                    seq.append(i)
                    key0.append(first)
                    at = end
            dev = self.tokens.device
            put = torch.tensor(cu_q + cu_kv + seq + key0, dtype=torch.int32).to(dev)
            n = len(seq)
            t = torch.split(put, [n + 1, n + 1, n, n])
            self._pieces[chunk] = Pieces(*(x.contiguous() for x in t), max(b - a for a, b in zip(cu_q, cu_q[1:])), cu_kv[-1], cu_q == cu_kv)
        return self._pieces[chunk]


def linear(h, w):
    return h @ w.t()


class LightningMixer:
    """Decayed linear attention; keeps a fp32 state per request."""

    def __init__(self, spec: LightningSpec, w: dict, eps: float):
        self.spec, self.w, self.eps = spec, w, eps

    @staticmethod
    def store(spec: LightningSpec):
        return ("state", spec.heads, spec.dim, spec.vdim)

    def rope_key(self):
        return None

    def mix(self, h, store, step: Step, rope, out=None):
        """The mixer's activations [T, n] ahead of the output projection, in `out` (rows at any stride) if that is given."""
        s, w = self.spec, self.w
        z = linear(h, w["w_in"])                                     # q | k | v | output gate
        o = hops.lightning(z, w["in_at"][:3], s.heads, s.dim, s.vdim, w["decay"], store, step.state_rows, step.starts, step.status,
                           cu_seqlens=step.cu, max_len=max(step.lens) if step.cu is not None else 1)
        at = w["in_at"][3]
        return rops.gated_norm(o, z[:, at:at + s.heads * s.vdim], w["norm"], self.eps, out=out)


class LatentAttentionMixer:
    """Attention on cached latent rows; keeps `kv_rank` + `rot_dim` elements per token."""

    # Prompts expand the latents into per-head keys and values; shorter portions and decode steps work in the latent space,
    # where nothing has to be computed for the keys.

    def __init__(self, spec: LatentAttentionSpec, w: dict, eps: float):
        self.spec, self.w, self.eps = spec, w, eps
        self.can_expand = w["w_in"].is_cuda and hops.latent_prefill_supported(spec.dim, spec.rot_dim, spec.vdim, spec.scale, w["w_in"].dtype)

    @staticmethod
    def store(spec: LatentAttentionSpec):
        return ("latent", spec.kv_rank + spec.rot_dim)

    def rope_key(self):
        return self.spec.rot_base, self.spec.rot_dim

    def mix(self, h, store, step: Step, rope, out=None):
        o = self._attend(h, store, step, rope)
        return o if out is None else out.copy_(o)

    def _attend(self, h, store, step: Step, rope):
        s, w = self.spec, self.w
        cos, sin = rope
        T, H = h.size(0), s.heads
        z = linear(h, w["w_in"])                                     # query latent | latent | shared key part | head gates
        at = w["in_at"]
        gate = z[:, at[3]:at[3] + H]
        expand = self.can_expand and step.cu is not None and T >= PROMPT_TOKENS * len(step.lens)
        fresh = expand and not any(step.past)
        cq, c, kr = hops.latent_prep(z, at[0], s.q_rank, at[1], s.kv_rank, at[2], s.rot_dim, w["q_norm"], w["kv_norm"], self.eps, cos, sin,
                                     store, step.block_table, step.tok_seq, step.positions, step.status, contiguous_kv=fresh)
        q = linear(cq, w["w_uq"])
        if expand:
            if not fresh:                                            # this pass's rows are in the pages too
                c, kr = hops.latent_gather(store, step.block_table, step.cu_kv, sum(step.past) + T, s.kv_rank, s.rot_dim, step.status)
            hops.rotate_heads_(q, cos, sin, H, s.dim + s.rot_dim, s.dim, s.rot_dim)
            o = hops.latent_prefill(q, linear(c, w["w_ukv"]), kr, gate, step.cu, step.cu_kv, max(step.lens), H, s.dim, s.vdim, s.scale,
                                    step.status)
            return o
        q = q.view(T, H, s.dim + s.rot_dim)
        # scores and values in the latent space: q W_uk against the cached latents, the weighted latent times W_uv
        q_abs = torch.empty((T, H, s.kv_rank), dtype=h.dtype, device=h.device)
        torch.bmm(q[..., :s.dim].transpose(0, 1), w["w_uk"], out=q_abs.transpose(0, 1))
        lat = hops.latent_attention(q_abs, q, s.dim, cos, sin, store, step.block_table, step.tok_seq, step.positions, gate, s.kv_rank,
                                    s.rot_dim, s.scale, step.status)
        o = torch.empty((T, H, s.vdim), dtype=h.dtype, device=h.device)
        torch.bmm(lat.transpose(0, 1), w["w_uv"].transpose(1, 2), out=o.transpose(0, 1))
        return o.view(T, H * s.vdim)


class MlstmMixer:
    """Matrix memory with exponential gates; keeps a fp32 state, a normaliser and a running maximum per request."""

    def __init__(self, spec: MlstmSpec, w: dict, eps: float):
        self.spec, self.w, self.eps = spec, w, eps
        self.one_kernel = w["w_in"].is_cuda and mops.recurrence_step_supported(spec.dim, spec.vdim)

    @staticmethod
    def store(spec: MlstmSpec):
        H, f32 = spec.heads, torch.float32
        return "slots", ((H, spec.dim, spec.vdim), f32), ((2, H, spec.dim), f32), ((2, H), f32)

    def rope_key(self):
        return None

    def mix(self, h, store, step: Step, rope, out=None):
        s, w = self.spec, self.w
        state, norm, m = store
        z = linear(h, w["w_in"])                                     # q | k | v | output gate | input gate | forget gate
        q, k, v, g, i, f = w["in_at"]
        seqs, scale = step.sequences(), dict(q_scale=s.dim ** -0.5, norm_eps=NORMALISER_EPS)
        if step.cu is None and self.one_kernel:
            o = mops.max_gate_step(z, (q, k, v), s.heads, s.dim, s.vdim, i, f, w["bias_i"], w["bias_f"], s.gate_cap, state, norm, m, seqs,
                                   step.status, **scale)
        else:
            la, b, floor, n0 = mops.max_gates(z, i, f, w["bias_i"], w["bias_f"], s.gate_cap, m, norm, seqs, step.status)
            o = mops.recurrence(z, (q, k, v), s.heads, s.heads, s.dim, s.vdim, la, b, state, seqs, step.status, floor=floor, n0=n0, norm=norm, **scale)
        return rops.gated_norm(o, z[:, g:g + s.heads * s.vdim], w["norm"], self.eps, group=s.vdim, out=out)


class Mamba2Mixer:
    """State-space recurrence behind a short convolution; keeps a fp32 state and the convolution's last inputs per request."""

    def __init__(self, spec: Mamba2Spec, w: dict, eps: float):
        self.spec, self.w, self.eps = spec, w, eps
        self.one_kernel = w["w_in"].is_cuda and mops.recurrence_step_supported(spec.state, spec.vdim)

    @staticmethod
    def store(spec: Mamba2Spec):
        return "slots", ((spec.heads, spec.state, spec.vdim), torch.float32), ((spec.conv, spec.channels), None)

    def rope_key(self):
        return None

    def mix(self, h, store, step: Step, rope, out=None):
        s, w = self.spec, self.w
        state, ring = store
        z = linear(h, w["w_in"])                                     # gate | x | B | C | step size
        seqs, off_dt = step.sequences(), s.inner + s.channels
        if step.cu is None and self.one_kernel:
            y = mops.ssd_step(z, s.inner, s.heads, s.groups, s.state, s.vdim, off_dt, w["dt_bias"], w["a_log"], w["skip"], w["conv_w"], w["conv_b"],
                              ring, state, seqs, step.status)
        else:
            u = mops.conv_silu(z, s.inner, w["conv_w"], w["conv_b"], ring, seqs, step.tok_seq, step.positions, step.status)
            la, b = mops.step_gates(z, off_dt, w["dt_bias"], w["a_log"])
            at_b = s.inner
            at_c = at_b + s.groups * s.state
            y = mops.recurrence(u, (at_c, at_b, 0), s.heads, s.groups, s.state, s.vdim, la, b, state, seqs, step.status, skip=w["skip"])
        return rops.gated_norm(y, z[:, :s.inner], w["norm"], self.eps, group=s.inner // s.norm_groups, silu_first=True, out=out)


class ChunkedAttentionMixer:
    """Grouped-query attention inside chunks of the sequence; keeps keys and (mixed) values per token."""

    def __init__(self, spec: ChunkedAttentionSpec, w: dict, eps: float):
        self.spec, self.w, self.eps = spec, w, eps
        self.prompt_kernel = w["w_in"].is_cuda and mops.kv_prefill_supported(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.scale,
                                                                             w["w_in"].dtype)

    @staticmethod
    def store(spec: ChunkedAttentionSpec):
        return "kv", spec.kv_heads, spec.dim, spec.vdim, spec.chunk

    def rope_key(self):
        return None

    def mix(self, h, store, step: Step, rope, out=None):
        s, w = self.spec, self.w
        z = linear(h, w["w_in"])                                     # q | k | v | output gate
        at = w["in_at"]
        gate = z[:, at[3]:at[3] + s.heads * s.vdim]
        first = None
        if s.v_mix:
            first = step.values_first
            if first is None:
                step.values_first = z[:, at[2]:at[2] + s.kv_heads * s.vdim]
        pages = mops.Pages(*store, step.block_table, step.tok_seq, step.positions, step.status)
        pieces = None
        if self.prompt_kernel and step.cu is not None and h.size(0) >= PROMPT_TOKENS * len(step.lens):
            pieces = step.pieces(s.chunk)
        q, k, v = mops.kv_prep(pages, z, at[:3], s.heads, w["q_norm"], w["k_norm"], self.eps, v_first=first, lam=w["lambda"],
                               contiguous_kv=pieces is not None and pieces.fresh)
        if pieces is None:
            return mops.kv_attention(pages, q, s.heads, s.chunk, s.scale, slopes=w["slopes"], gate=gate, out=out)
        if not pieces.fresh:                                         # this pass's rows are in the pages too
            k, v = mops.kv_gather(pages, s.heads, pieces.seq, pieces.key0, pieces.cu_kv, pieces.total_kv)
        return mops.kv_prefill(q, k, v, pieces.cu_q, pieces.cu_kv, pieces.max_q, s.heads, s.kv_heads, s.scale, w["slopes"], step.status, gate=gate,
                               out=out)


MIXERS = {LightningSpec: LightningMixer, LatentAttentionSpec: LatentAttentionMixer, MlstmSpec: MlstmMixer, Mamba2Spec: Mamba2Mixer,
          ChunkedAttentionSpec: ChunkedAttentionMixer}


class HybridDecoder(GreedyHead):
    """Single-GPU decoder with the interface `GenerationRunner` drives (see `TPDecoder`)."""

    supports_portions = True     # a prompt may be prefilled in several passes

    def __init__(self, cfg: HybridConfig, weights, device="cuda"):
        cfg.validate()
        self.cfg, self.w = cfg, weights
        self.rank, self.world, self.group, self.comm = 0, 1, None, None
        self.device = torch.device(device)
        self.dtype = weights["embed"].dtype
        self.vl = cfg.vocab_size
        self.max_positions = cfg.max_positions
        if self.device.type == "cuda":
            # 32-bit products stay 32-bit, and the partial sums of a bfloat16 product are added up in 32 bits
            torch.backends.cuda.matmul.allow_tf32 = False
            torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        self.mixers = [MIXERS[type(l.mixer)](l.mixer, lw, cfg.norm_eps) for l, lw in zip(cfg.layers, weights["layers"])]
        self.runs = cfg.runs()
        self._rope_f = {}
        for m in self.mixers:
            key = m.rope_key()
            if key is not None and key not in self._rope_f:
                base, dims = key
                i = torch.arange(0, dims, 2, dtype=torch.float64)
                self._rope_f[key] = (float(base) ** (-i / dims)).to(device=self.device, dtype=torch.float32)
        self._iota = torch.arange(1, dtype=torch.int32, device=self.device)
        self.layer_hook = None     # called with the residual after every layer run (inspection and tests)

    # ---- what GenerationRunner asks for ----------------------------------------------------------------
    def make_cache(self, max_batch: int, max_seq_len: int, num_blocks: int = 0) -> HybridCache:
        specs = [self.mixers[i].store(self.cfg.layers[i].mixer) for i, _ in self.runs]
        if self.cfg.bigram is not None:
            specs.append(("slots", ((), torch.int32)))               # the last token of every request
        per_seq = (max_seq_len + BLOCK_SIZE - 1) // BLOCK_SIZE
        return HybridCache(specs, num_blocks or max_batch * per_seq, max_batch, per_seq, self.device, self.dtype)

    def check_errors(self) -> None:
        """Raise if a kernel of this model recorded an error on the device (its cache holds the status word)."""

    def _range(self, n):
        if self._iota.numel() < n:
            self._iota = torch.arange(n, dtype=torch.int32, device=self.device)
        return self._iota[:n]

    def rope_tables(self, positions):
        """fp32 cos / sin [T, dims / 2] of every rotation the layers use."""
        out = {}
        for key, f in self._rope_f.items():
            a = torch.outer(positions.float(), f)
            out[key] = (a.cos(), a.sin())
        return out

    def forward(self, token_ids, positions, kv: HybridCache, block_table, slots, max_blocks, *, cu_seqlens=None, max_seqlen=0,
                seq_lens_after=None, seg=None, state_rows=None, want=None, lens=None, past=None):
        """Arguments as `TPDecoder.forward`, and: `state_rows` [n_seq] table rows of the sequences (default 0 .. n_seq - 1), `lens` /
        `past` (prompts: new and cached tokens per sequence, on the host), `want` rows of the packed tokens whose hidden state is
        returned (default: the last of every sequence)."""
        n_seq = slots.numel()
        seg = seg or Segments(capture=False)
        prompt = cu_seqlens is not None
        if prompt and lens is None:
            c = cu_seqlens.tolist()
            lens = [b - a for a, b in zip(c, c[1:])]
        if prompt and past is None:
            past = [int(p) for p in slots.tolist()]
        rows = self._range(n_seq) if state_rows is None else state_rows
        if prompt:
            tok_seq = torch.repeat_interleave(torch.arange(n_seq, dtype=torch.int32),
                                              torch.tensor(lens)).to(self.device, non_blocking=True)
        else:
            tok_seq = self._range(n_seq)
        cu_kv = cu_seqlens
        if prompt and any(past):
            cu_kv = torch.tensor(list(itertools.accumulate((p + n for p, n in zip(past, lens)), initial=0)), dtype=torch.int32).to(self.device)
        step = Step(token_ids, positions, slots, cu_seqlens, tok_seq, rows, block_table, lens, past, cu_kv, kv.status)
        if prompt and want is None:
            want = (cu_seqlens[1:] - 1).long()
        out = {}
        seg.run(lambda: out.update(hidden=self._pass(step, kv, want)))
        return out["hidden"]

    def _embedding(self, step: Step, kv: HybridCache):
        """Arguments of the norm that sets x to the embedding output."""
        cfg, w = self.cfg, self.w
        more = []
        if cfg.bigram is not None:
            b = cfg.bigram
            more.append((w["bigram"], rops.bigram_rows(step.tokens, step.starts, step.state_rows, kv.stores[len(self.runs)][0], b.buckets, b.mul_prev,
                                                       b.mul_cur, step.status, cu_seqlens=step.cu)))
        if cfg.max_positions:
            more.append((w["pos"], step.positions))
        return dict(embed=w["embed"], tokens=step.tokens, init=True, embed_scale=cfg.embed_scale, more=more)

    def _mlp_act(self, h, lw, mlp, out=None):
        """The feed-forward's activations ahead of its output projection."""
        if isinstance(mlp, GeluSpec):
            return rops.gelu(linear(h, lw["w_up"]), out=out)
        act = rops.clamped_glu(linear(h, lw["w_gu"]), mlp.limit, GLU_ALPHA, GLU_SHIFT)
        return act if out is None else out.copy_(act)

    def _parallel_layer(self, i, x, store, step, rope, pend):
        """mixer(norm1(x)) + mlp(norm2(x)), x with `pend` applied."""
        lw, mixer, mlp = self.w["layers"][i], self.mixers[i], self.cfg.layers[i].mlp
        if mlp is None:
            h = rops.residual_norm(x, lw["norm1"], self.cfg.norm_eps, **pend)
            return linear(mixer.mix(h, store, step, rope), lw["w_out"])
        h, h2 = rops.residual_norm(x, lw["norm1"], self.cfg.norm_eps, w2=lw["norm2"], **pend)
        n = lw["w_out"].size(1)                                      # activations of the mixer, then of the feed-forward
        act = torch.empty((x.size(0), (n + 7) // 8 * 8), dtype=self.dtype, device=self.device)[:, :n]
        mixer.mix(h, store, step, rope, out=act[:, :n - mlp.ff])
        self._mlp_act(h2, lw, mlp, out=act[:, n - mlp.ff:])
        return linear(act, lw["w_out"])

    def _pass(self, step: Step, kv: HybridCache, want):
        cfg, w, eps = self.cfg, self.w, self.cfg.norm_eps
        T = step.tokens.numel()
        x = torch.empty((T, cfg.width), dtype=torch.float32, device=self.device)
        rope = self.rope_tables(step.positions)
        pend = self._embedding(step, kv)                # the update of x that the next norm applies
        for r, (i, again) in enumerate(self.runs):
            lw, mixer, mlp = w["layers"][i], self.mixers[i], cfg.layers[i].mlp
            if again:
                pend = dict(pend, embed=w["embed"], tokens=step.tokens)
            if cfg.parallel:
                pend = dict(delta=self._parallel_layer(i, x, kv.stores[r], step, rope.get(mixer.rope_key()), pend))
            else:
                h = rops.residual_norm(x, lw["norm1"], eps, **pend)
                pend = dict(delta=linear(mixer.mix(h, kv.stores[r], step, rope.get(mixer.rope_key())), lw["w_out"]))
                if mlp is not None:
                    h = rops.residual_norm(x, lw["norm2"], eps, **pend)
                    pend = dict(delta=linear(self._mlp_act(h, lw, mlp), lw["w_down"]))
            if cfg.side_dim:
                xt = rops.residual_norm(x, None, eps, **pend)
                y = rops.side_gate(linear(xt, lw["side_gate"]), w["side_embed"], step.tokens, i * cfg.side_dim)
                pend = dict(delta=linear(y, lw["side_proj"]), delta_w=lw["side_norm"])
            if self.layer_hook is not None:
                rops.residual_norm(x, None, eps, **pend, out=False)
                pend = {}
                self.layer_hook(x)
        if want is not None:
            if want.numel() == 0:
                return torch.empty((0, cfg.width), dtype=self.dtype, device=self.device)
            x = x[want].contiguous()
            if "delta" in pend:
                pend = dict(pend, delta=pend["delta"][want].contiguous())
        return rops.residual_norm(x, w["final_norm"], eps, **pend)

    def logits(self, hidden):
        """fp32 logits; the output matrix is the embedding table."""
        if hidden.dtype == torch.float32:
            return hidden @ self.w["embed"].t()
        return torch.mm(hidden, self.w["embed"].t(), out_dtype=torch.float32)
