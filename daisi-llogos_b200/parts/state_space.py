"""A state-space recurrence with a scalar decay per head and step (Mamba-2), as a mixer with a fixed-size state.

One product of the mixer's input gives ``z | x | B | C | dt`` (``heads value_dim``, the same, ``groups state_size`` twice, and ``heads``
numbers).  x, B and C together pass a short causal convolution per channel with a bias, and silu.  Per head, with
``d = softplus(dt + dt_bias)`` and the B and C of the head's group (head h: group ``h // (heads / groups)``),

    S_t = exp(-exp(A_log) d_t) S_{t-1} + d_t B_t x_t^T        (S is [state_size, value_dim], zero before a sequence)
    y_t = S_t^T C_t + D x_t

and ``W_o`` projects ``N(y silu(z))``, where N divides each of ``norm_groups`` equal parts of the row by its own root mean square and
multiplies by a weight.  The cache keeps S and the convolution's last ``taps - 1`` inputs per sequence in float32.

``ops.causal_conv`` adds the product's partial sums and leaves x, B, C in the compute type; ``ops.state_space`` takes dt's and z's
sums as float32, walks the recurrence (in bfloat16 prompt steps in chunks on the tensor cores) and applies the gate;
``ops.part_rmsnorm`` norms for the output product.  Step sizes, decays, the state, the gate and the norm are float32 whatever the compute type.
"""
from __future__ import annotations

import torch

from ..kernels.linear import linear
from .base import Branch, Mixer, MultiNeed, StateNeed, TensorDecl, as_f32, register_part


class StateSpace(Mixer):
    """params: hidden_size, num_heads, value_dim, state_size, groups, conv_taps, norm_groups, norm_eps.  Tensors: ``in_proj.weight`` [2
    heads value_dim + 2 groups state_size + heads, hidden], ``conv.weight`` [channels, taps] and ``conv.bias`` [channels] (channels =
    heads value_dim + 2 groups state_size), ``dt_bias``, ``A_log``, ``D`` [heads], ``norm.weight`` [heads value_dim], ``o_proj.weight``
    [hidden, heads value_dim]."""

    SCORES_PAIRS = False        # no (query, key) pairs: the cost of a token does not grow with what came before

    def __init__(self, params, prefix, env):
        super().__init__(params, prefix, env)
        p = params
        self.hidden = int(p["hidden_size"])
        self.nh, self.vd = int(p["num_heads"]), int(p["value_dim"])
        self.state_size, self.groups = int(p["state_size"]), int(p["groups"])
        self.taps = int(p["conv_taps"])
        self.norm_groups, self.eps = int(p["norm_groups"]), float(p["norm_eps"])
        for what in ("num_heads", "value_dim", "state_size", "groups", "norm_groups"):
            if int(p[what]) <= 0:
                raise ValueError(f"state_space: {what} must be positive, got {p[what]}")
        self.inner = self.nh * self.vd
        self.channels = self.inner + 2 * self.groups * self.state_size
        if self.nh % self.groups:
            raise ValueError(f"state_space: {self.nh} heads do not split into {self.groups} groups")
        if self.inner % self.norm_groups:
            raise ValueError(f"state_space: {self.inner} elements do not split into {self.norm_groups} equal parts")
        limit = getattr(env.ops, "CONV_MAX_TAPS", None)
        if self.taps < 1 or (limit is not None and self.taps > limit):
            raise ValueError(f"state_space: {self.taps} convolution taps (1 to {limit})")
        fits = getattr(env.ops, "state_space_supported", None)
        if fits is not None and not fits(self.state_size, self.vd):
            raise ValueError(f"state_space: a head's state of {self.state_size} x {self.vd} elements does not fit a block")
        self.w_in = self.w_o = self.w_conv = self.b_conv = self.dt_bias = self.a_log = self.d_skip = self.norm_w = None

    def tensors(self):
        return {"in_proj.weight": TensorDecl((self.inner + self.channels + self.nh, self.hidden)),
                "conv.weight": TensorDecl((self.channels, self.taps), "conv"), "conv.bias": TensorDecl((self.channels,), "bias"),
                "dt_bias": TensorDecl((self.nh,), "rate"), "A_log": TensorDecl((self.nh,), "bias"), "D": TensorDecl((self.nh,), "norm"),
                "norm.weight": TensorDecl((self.inner,), "norm"), "o_proj.weight": TensorDecl((self.hidden, self.inner))}

    def bind(self, tensors):
        self.w_in, self.w_o = tensors["in_proj.weight"], tensors["o_proj.weight"]
        self.w_conv, self.b_conv = as_f32(tensors["conv.weight"], self.env), as_f32(tensors["conv.bias"], self.env)
        self.dt_bias, self.a_log = as_f32(tensors["dt_bias"], self.env), as_f32(tensors["A_log"], self.env)
        self.d_skip, self.norm_w = as_f32(tensors["D"], self.env), as_f32(tensors["norm.weight"], self.env)

    def cache_need(self):
        state = StateNeed((self.nh, self.state_size, self.vd), torch.float32)
        if self.taps > 1:
            return MultiNeed.of(state=state, conv=StateNeed((self.taps - 1, self.channels), torch.float32))
        return state

    def forward(self, x, ctx, cache) -> Branch:
        ops = ctx.ops
        n = x.shape[0]
        conv_state = None
        if self.taps > 1:
            cache, conv_state = cache["state"], cache["conv"].state
        rows = linear(ctx, x, self.w_in, "ssm.in", torch.float32)                   # [P, N, z | x | B | C | dt]
        mixed = ctx.buffer("ssm.mixed", (n, self.channels))
        wide = mixed.dtype == torch.float32
        ops.causal_conv(rows, self.inner, self.w_conv, conv_state, ctx.slots, ctx.cu_tokens, ctx.seq_of_token, ctx.len_before,
                        mixed if wide else None, bias=self.b_conv, out2=None if wide else mixed, act="silu")
        gated = ctx.buffer("ssm.gated", (n, self.inner), torch.float32)
        ops.state_space(mixed, rows, z_col=0, dt_col=self.inner + self.channels, dt_bias=self.dt_bias, a_log=self.a_log,
                        d_skip=self.d_skip, n_heads=self.nh, groups=self.groups, n_state=self.state_size, vdim=self.vd,
                        state=cache.state, slots=ctx.slots, cu_tokens=ctx.cu_tokens, out=gated, max_count=ctx.max_count)
        out = ctx.buffer("ssm.out", (n, self.inner))
        ops.part_rmsnorm(gated, self.norm_w, self.norm_groups, self.eps, out)
        return Branch(linear(ctx, out, self.w_o, "ssm.proj", torch.float32))


register_part("mixer", "state_space", StateSpace)
