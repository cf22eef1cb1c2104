"""Attention through a latent: per token the cache holds one row, a normed low-rank latent c and one rotated key part
shared by all heads, instead of keys and values per head.  A head's unrotated key is W_uk c and its value W_uv c, so
the score q . (W_uk c) is formed as (W_uk^T q) . c and the output as W_uv (sum_j p_j c_j): every head attends over the
same cached rows, and keys and values per head are never made.  Causal, with an optional sliding window, an optional
learned sink per head in the softmax's denominator, and an optional gate per token and head.  A layer may have rows of its
own or read those of another layer's run (its run's ``cache_of``).
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..kernels.limits import latent_refusal
from ..weights.manifest import MATRIX, NORM_WEIGHT, VECTOR, TensorSpec
from .base import KVSpec, Mixer, take_weight
from .linear import _check_true_fp32, filled_rows, kernel_modules as linear_modules, linear
from .registry import register_mixer


PROMPT_KERNEL_MIN_TOKENS = 17      # whole prompts of at least this many tokens (the longest of the step) take the
                                   # tensor-core kernel; shorter ones are scored against the latents like single tokens


class LatentAttention(Mixer):
    """params: hidden_size, heads, dim (unrotated query/key size per head), rot_dim (rotated size), vdim, kv_rank,
    q_rank (0: q = W_q h, without a low rank), scale, window (0: none), sink (bool), head_gate (bool), shared_rows (bool),
    norm_eps, names (optional overrides).

    c_q = RMSnorm(W_dq h); q = W_uq c_q (or q = W_q h), head by head [dim | rot_dim].  W_dkv h = [kv_rank latent, RMS-normed ->
    c | rot_dim rotated key part].  The position encoding turns neighbouring pairs of the rotated parts of q and k.
    score = (q_plain . W_uk c + q_rot . k_rot) * scale; softmax over the visible keys (and the sink); value W_uv c.
    ``head_gate``: a sigmoid gate per token and head (W_g h) on the heads' outputs, ahead of W_o.  ``shared_rows``: the layer
    has no W_dkv and writes no rows; its run reads the rows of another layer's run, whose latent and rotation have the same
    sizes, through keys, values and queries of its own."""

    NAMES = {"q_down": "dq", "q_norm": "dq.norm", "q_up": "uq", "kv_down": "dkv", "kv_norm": "dkv.norm", "k_up": "uk",
             "v_up": "uv", "sink": "sink", "out": "o", "q": "q", "gate": "g"}

    def __init__(self, spec, runtime, position=None):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.heads = int(p["hidden_size"]), int(p["heads"])
        self.dim, self.rot_dim, self.vdim = int(p["dim"]), int(p["rot_dim"]), int(p["vdim"])
        self.kv_rank, self.q_rank = int(p["kv_rank"]), int(p.get("q_rank", 0) or 0)
        self.scale = float(p["scale"])
        self.window = int(p.get("window", 0) or 0)
        self.has_sink, self.head_gate = bool(p.get("sink", False)), bool(p.get("head_gate", False))
        self.shared_rows = bool(p.get("shared_rows", False))
        self.eps = float(p["norm_eps"])
        self.names = {**self.NAMES, **dict(p.get("names", {}))}
        self.position = position
        rotated = getattr(position, "rotary_dim", 0) if position is not None else 0
        if rotated > self.rot_dim:
            raise ValueError(f"latent attention '{self.prefix}': the rotation covers {rotated} values, the rotated part has {self.rot_dim}")
        refusal = latent_refusal(self.kv_rank, self.rot_dim)
        if refusal:
            raise ValueError(f"latent attention '{self.prefix}': {refusal}")

    def tensors(self):
        n, px, D, H = self.names, self.prefix, self.hidden, self.heads
        n_q = H * (self.dim + self.rot_dim)
        if self.q_rank:
            out = [TensorSpec(px + n["q_down"], (self.q_rank, D), MATRIX),
                   TensorSpec(px + n["q_norm"], (self.q_rank,), VECTOR, NORM_WEIGHT),
                   TensorSpec(px + n["q_up"], (n_q, self.q_rank), MATRIX)]
        else:
            out = [TensorSpec(px + n["q"], (n_q, D), MATRIX)]
        if not self.shared_rows:
            out += [TensorSpec(px + n["kv_down"], (self.kv_rank + self.rot_dim, D), MATRIX),
                    TensorSpec(px + n["kv_norm"], (self.kv_rank,), VECTOR, NORM_WEIGHT)]
        out += [TensorSpec(px + n["k_up"], (H * self.dim, self.kv_rank), MATRIX),
                TensorSpec(px + n["v_up"], (H * self.vdim, self.kv_rank), MATRIX),
                TensorSpec(px + n["out"], (D, H * self.vdim), MATRIX)]
        if self.head_gate:
            out.append(TensorSpec(px + n["gate"], (H, D), MATRIX))
        if self.has_sink:
            out.append(TensorSpec(px + n["sink"], (H,), VECTOR))
        return out

    def bind(self, weights):
        n, px, H = self.names, self.prefix, self.heads
        # one projection for everything that reads the mixer's input: (q) | (latent and rotated key part) | (gate)
        parts = ([] if self.q_rank else ["q"]) + ([] if self.shared_rows else ["kv_down"]) + (["gate"] if self.head_gate else [])
        self.w_in = filled_rows([take_weight(weights, px + n[k]) for k in parts]) if parts else None
        self.dkv_col0 = 0 if self.q_rank else H * (self.dim + self.rot_dim)
        self.gate_col0 = self.dkv_col0 + (0 if self.shared_rows else self.kv_rank + self.rot_dim)
        self.w_out = weights[px + n["out"]]
        if self.q_rank:
            self.w_q_down, self.w_q_up = weights[px + n["q_down"]], weights[px + n["q_up"]]
            self.q_norm_w = weights[px + n["q_norm"]].to(torch.float32).contiguous()
        self.kv_norm_w = None if self.shared_rows else weights[px + n["kv_norm"]].to(torch.float32).contiguous()
        self.w_k_up_flat, self.w_v_up_flat = weights[px + n["k_up"]], weights[px + n["v_up"]]
        self.w_k_up = weights[px + n["k_up"]].view(H, self.dim, self.kv_rank)                    # q_plain @ this: W_uk^T q
        self.w_v_up_t = weights[px + n["v_up"]].view(H, self.vdim, self.kv_rank).transpose(1, 2)   # latent @ this: W_uv c
        self.sink = weights[px + n["sink"]].to(torch.float32).contiguous() if self.has_sink else None

    def kernel_modules(self):
        mods = ["attention_latent", "elementwise", "rope_kv", *linear_modules(self.runtime.dtype)]
        if ops.latent_prefill_fits(self.runtime.dtype, self.dim, self.rot_dim, self.vdim, self.kv_rank):
            mods.append("attention_latent_mma")
        return tuple(mods)

    def kv_spec(self):
        return KVSpec(1, self.kv_rank + self.rot_dim, self.window, values=False)

    def _per_head(self, a, b):
        """Batched over heads: a [H, T, n] @ b [H, n, m] -> float32 [H, T, m] (a library product, 32-bit sums)."""
        if a.dtype == torch.bfloat16:
            return torch.bmm(a, b, out_dtype=torch.float32)
        _check_true_fp32()
        return torch.bmm(a, b)

    def forward(self, x, ctx, cache):
        dtype, H = self.runtime.dtype, self.heads
        proj = linear(x, self.w_in) if self.w_in is not None else None
        q = proj if not self.q_rank else linear(ops.rmsnorm(linear(x, self.w_q_down), self.q_norm_w, self.eps, dtype), self.w_q_up)
        dkv = None if self.shared_rows else proj
        gate = proj if self.head_gate else None
        cos = sin = None
        if self.position is not None:
            cos, sin = self.position.prepare(ctx)
        table = ctx.page_tables[cache.group_id]
        rows_key = ("latent_rows", cache.k_pool.data_ptr())     # this step's rows of a layer, for the layers that read them too
        if (ctx.all_start and ctx.max_new >= PROMPT_KERNEL_MIN_TOKENS and (not self.shared_rows or rows_key in ctx.shared)
                and ops.latent_prefill_fits(dtype, self.dim, self.rot_dim, self.vdim, self.kv_rank)):
            # whole prompts: keys and values per head from the prompt's own latents (two library products with bfloat16
            # results), then the usual attention on the tensor cores
            q_heads, rows = ops.latent_prep(q, dkv, self.kv_norm_w, cos, sin, ctx, table, cache.k_pool, H, self.dim,
                                            self.rot_dim, self.kv_rank, self.eps, store=cache.writable, whole_heads=True,
                                            dkv_col0=self.dkv_col0)
            if self.shared_rows:
                rows = ctx.shared[rows_key]
            else:
                ctx.shared[rows_key] = rows
            c = rows[:, :self.kv_rank]
            att = ops.latent_prefill(q_heads, torch.mm(c, self.w_k_up_flat.t()), rows, torch.mm(c, self.w_v_up_flat.t()), ctx,
                                     self.sink, self.scale, self.window, H, self.dim, self.rot_dim, self.vdim, gate=gate,
                                     gate_col0=self.gate_col0)
            return linear(att, self.w_out)
        q_plain, q_rot = ops.latent_prep(q, dkv, self.kv_norm_w, cos, sin, ctx, table, cache.k_pool, H, self.dim,
                                         self.rot_dim, self.kv_rank, self.eps, store=cache.writable, dkv_col0=self.dkv_col0)
        q_abs = self._per_head(q_plain, self.w_k_up)
        latent = ops.latent_attention(q_abs, q_rot, cache.k_pool, table, ctx, self.sink, self.scale, self.window)
        values = self._per_head(latent, self.w_v_up_t)                                             # [H, T, vdim]
        return linear(ops.latent_heads_out(values, dtype, gate, self.gate_col0), self.w_out)


register_mixer("latent_attention", LatentAttention)
