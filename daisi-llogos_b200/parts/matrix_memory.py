"""A matrix-valued memory per head, written under exponential gates (mLSTM), as a mixer with a fixed-size state.

Per head, with ``q = W_q h / sqrt(dim)``, ``k = W_k h``, ``v = W_v h`` and the logarithms of the two gates

    i = cap tanh((w_i . h + b_i) / cap),     f = logsigmoid(cap tanh((w_f . h + b_f) / cap)),

the memory S [dim, vdim], its normaliser n [dim] and a running maximum m (all zero before a sequence) follow

    m' = max(f + m, i),   S' = e^(f + m - m') S + e^(i - m') k v^T,   n' = e^(f + m - m') n + e^(i - m') k,
    o = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6).

Every head's o is divided by its root mean square (eps inside the root), the concatenated heads are multiplied by a weight
vector and by ``sigmoid(W_g h)``, and ``W_o`` projects them.  All projections of h are one product; ``ops.matrix_memory`` adds its
float32 partial sums and does the rest up to the output product in float32.  Carrying m beside S keeps every exponential at
most one; because S e^m and n e^m are linear in what was before, a prompt runs in pieces side by side that are joined by
their sums of f and their own maxima, and not token by token.  The cache keeps S, n and m per sequence in float32.
"""
from __future__ import annotations

import torch

from ..kernels.linear import linear
from .base import Branch, Mixer, MultiNeed, StateNeed, TensorDecl, as_f32, register_part

DENOMINATOR_EPS = 1e-6      # added to the read-out's denominator


class MatrixMemory(Mixer):
    """params: hidden_size, num_heads, head_dim, value_dim, gate_cap, norm_eps.  Tensors: ``q_proj``, ``k_proj``, ``v_proj``,
    ``g_proj``, ``i_gate``, ``f_gate``, ``o_proj`` (weights), ``i_gate.bias``, ``f_gate.bias`` [heads], ``norm.weight``
    [heads value_dim]."""

    SCORES_PAIRS = False        # no (query, key) pairs: the cost of a token does not grow with what came before

    _IN = ("q_proj.weight", "k_proj.weight", "v_proj.weight", "g_proj.weight", "i_gate.weight", "f_gate.weight")

    def __init__(self, params, prefix, env):
        super().__init__(params, prefix, env)
        p = params
        self.hidden = int(p["hidden_size"])
        self.nh = int(p["num_heads"])
        self.hd = int(p["head_dim"])
        self.vd = int(p.get("value_dim") or self.hd)
        for what, v in (("num_heads", self.nh), ("head_dim", self.hd), ("value_dim", self.vd)):
            if v <= 0:
                raise ValueError(f"matrix_memory: {what} must be positive, got {v}")
        self.cap = float(p["gate_cap"])
        if not self.cap > 0:
            raise ValueError(f"matrix_memory: gate_cap must be positive, got {self.cap}")
        self.eps = float(p["norm_eps"])
        fits = getattr(env.ops, "matrix_memory_supported", None)
        if fits is not None and not fits(self.hd, self.vd):
            raise ValueError(f"matrix_memory: a head's state of {self.hd} rows does not fit a block")
        self.w_in = self.w_o = self.b_i = self.b_f = self.norm_w = None

    def tensors(self):
        qk, v = self.nh * self.hd, self.nh * self.vd
        rows = dict(zip(self._IN, (qk, qk, v, v, self.nh, self.nh)))
        t = {name: TensorDecl((n, self.hidden)) for name, n in rows.items()}
        t.update({"i_gate.bias": TensorDecl((self.nh,), "bias"), "f_gate.bias": TensorDecl((self.nh,), "bias"),
                  "norm.weight": TensorDecl((v,), "norm"), "o_proj.weight": TensorDecl((self.hidden, v))})
        return t

    def bind(self, tensors):
        ws = [tensors[n] for n in self._IN]
        if len({w.dtype for w in ws}) != 1:
            raise ValueError(f"{self.prefix}: the input projections are stored with different types")
        self.w_in = torch.cat(ws, dim=0).contiguous()                               # rows: q | k | v | g | i | f
        self.w_o = tensors["o_proj.weight"]
        self.b_i, self.b_f = as_f32(tensors["i_gate.bias"], self.env), as_f32(tensors["f_gate.bias"], self.env)
        self.norm_w = as_f32(tensors["norm.weight"], self.env)

    def cache_need(self):
        return MultiNeed.of(memory=StateNeed((self.nh, self.hd, self.vd), torch.float32),
                            normaliser=StateNeed((self.nh, self.hd), torch.float32),
                            maximum=StateNeed((self.nh,), torch.float32))

    def forward(self, x, ctx, cache) -> Branch:
        ops = ctx.ops
        n = x.shape[0]
        qk, v = self.nh * self.hd, self.nh * self.vd
        rows = linear(ctx, x, self.w_in, "memory.in", torch.float32)
        out = ctx.buffer("memory.out", (n, v))
        piece, pieces, cols = ops.matrix_memory_plan(self.hd, self.vd, self.nh, ctx.n_seqs, ctx.max_count)
        carry = raw = aside = None
        if pieces > 1:
            carry = ctx.buffer("memory.carry", (ctx.n_seqs, pieces, self.nh, self.hd * self.vd + self.hd + ops.MEMORY_CARRY_EXTRA),
                               torch.float32)
        if cols < self.vd:
            raw = ctx.buffer("memory.raw", (n, v), torch.float32)
            if carry is None:
                aside = ctx.buffer("memory.next", (ctx.n_seqs, self.nh, self.hd + 1), torch.float32)
        ops.matrix_memory(rows, q_col=0, k_col=qk, v_col=2 * qk, g_col=2 * qk + v, i_col=2 * (qk + v), f_col=2 * (qk + v) + self.nh,
                          n_heads=self.nh, dim=self.hd, vdim=self.vd, i_bias=self.b_i, f_bias=self.b_f, gate_cap=self.cap,
                          q_scale=float(self.hd) ** -0.5, denom_eps=DENOMINATOR_EPS, eps=self.eps, norm_w=self.norm_w,
                          state_s=cache["memory"].state, state_n=cache["normaliser"].state, state_m=cache["maximum"].state,
                          slots=ctx.slots, cu_tokens=ctx.cu_tokens, out=out, cols=cols, carry=carry, piece=piece, raw=raw, next_nm=aside)
        return Branch(linear(ctx, out, self.w_o, "memory.proj", torch.float32))


register_part("mixer", "matrix_memory", MatrixMemory)
