"""A plain, slow implementation of the Penasun decoder, for tests only: whole sequences, no cache, float64,
one function per mechanism, and no code shared with the library under test (it reads config.json's keys and
looks tensors up by name on its own).

The design in this file's notation (T tokens, width D, token ids ``tok``):

* ``N(x, w) = x / sqrt(mean(x^2) + eps) * w``; a layer is ``x <- x + mixer(N(x, norm1))`` and, where it has a
  feed-forward, ``x <- x + ff(N(x, norm2))``; ``x`` starts as ``embed[tok]``, the logits are ``embed N(x, final.norm)``.
* mixer "mamba2": ``[z | x | B | C | dt] = W_in h``; the columns of x, B and C pass ``silu(conv)``, a causal convolution
  per channel with a bias (last column: the current token); per head ``d = softplus(dt + dt_bias)``,
  ``S <- exp(-exp(A_log) d) S + d B x^T`` from S = 0, ``y = S^T C + D x``, where head h reads the B and C of group
  ``floor(h groups / heads)``; ``y silu(z)`` is divided by its root mean square in ``norm_groups`` equal parts, multiplied by
  ``norm`` and projected by ``W_o``.
* mixer "attention": q, k, v with biases; a query head and a key head hold two maps of ``dim`` elements each, one after
  the other; q times ``1 + coef ln(floor((p + 1) / every) + 1)``; for each map a causal softmax of ``scale q . k`` over the
  same values gives ``a1`` and ``a2``; ``lam = exp(lq1 . lk1) - exp(lq2 . lk2) + diff``; ``o = a1 - lam a2`` divided by its root
  mean square per head, times ``1 - diff``; ``W_o`` with a bias.
* feed-forward "moe": ``s = softmax(router h)`` over the experts and the identity experts; choice scores ``s + correction``;
  consecutive groups, the ``keep`` groups of largest best choice score stay; the ``top`` largest choice scores among them
  are chosen, weighted by ``scale s``; an expert is ``down(g sigmoid(1.702 g) (u + 1))`` with ``g = min(gate h, limit)``
  and ``u = clamp(up h, -limit, limit)``; an identity expert returns h.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Sequence, Tuple

import torch

F64 = torch.float64


# ---- mechanisms ---------------------------------------------------------------------------------

def linear(x, w, b=None):
    y = x.to(F64) @ w.to(F64).t()
    return y if b is None else y + b.to(F64)


def unit_rms(x, eps):
    x = x.to(F64)
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight.to(F64)


def silu(x):
    return x * torch.sigmoid(x)


def causal_conv(u: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """u: [T, channels]; out_t = bias + sum_j weight[:, taps - 1 - j] u_{t - j}, zeros before the first token."""
    u, weight = u.to(F64), weight.to(F64)
    taps = weight.shape[1]
    out = bias.to(F64).expand_as(u).clone()
    for j in range(taps):
        shifted = torch.zeros_like(u)
        if j < u.shape[0]:
            shifted[j:] = u[:u.shape[0] - j]
        out += weight[:, taps - 1 - j] * shifted
    return out


def state_space(x, b, c, dt, a_log, d_skip, state=None) -> Tuple[torch.Tensor, torch.Tensor]:
    """x: [T, heads, vdim]; b, c: [T, groups, N]; dt: [T, heads] (already softplus).  ``(y [T, heads, vdim], last S
    [heads, N, vdim])``, token by token."""
    t, heads, vdim = x.shape
    groups, n = b.shape[1:]
    of = torch.arange(heads) // (heads // groups)
    s = torch.zeros(heads, n, vdim, dtype=F64) if state is None else state.to(F64).clone()
    rate, skip = torch.exp(a_log.to(F64)), d_skip.to(F64)[:, None]
    ys = []
    for i in range(t):
        decay = torch.exp(-rate * dt[i])
        s = decay[:, None, None] * s + (dt[i][:, None] * b[i, of])[:, :, None] * x[i][:, None, :]
        ys.append((s * c[i, of][:, :, None]).sum(1) + skip * x[i])
    return torch.stack(ys), s


def gated_group_norm(y, z, weight, parts, eps) -> torch.Tensor:
    """``y silu(z)``, then each of ``parts`` equal parts of a row by its own root mean square, then the weight."""
    v = y.to(F64) * silu(z.to(F64))
    return unit_rms(v.view(v.shape[0], int(parts), -1), eps).reshape(v.shape) * weight.to(F64)


def mamba2(h, w, p, mx, eps) -> torch.Tensor:
    t = h.shape[0]
    heads, vdim, n, groups = int(mx["heads"]), int(mx["vdim"]), int(mx["state"]), int(mx["groups"])
    inner, gn = heads * vdim, groups * n
    rows = linear(h, w[p + "in"])
    z, mixed, dt = rows[:, :inner], rows[:, inner:2 * inner + 2 * gn], rows[:, 2 * inner + 2 * gn:]
    mixed = silu(causal_conv(mixed, w[p + "conv"], w[p + "conv.b"]))
    x, b, c = mixed[:, :inner], mixed[:, inner:inner + gn], mixed[:, inner + gn:]
    step = torch.nn.functional.softplus(dt + w[p + "dt_bias"].to(F64), threshold=1e9)
    y, _ = state_space(x.reshape(t, heads, vdim), b.reshape(t, groups, n), c.reshape(t, groups, n), step, w[p + "A_log"], w[p + "D"])
    y = gated_group_norm(y.reshape(t, inner), z, w[p + "norm"], mx["norm_groups"], eps)
    return linear(y, w[p + "o"])


def query_temperature(positions: torch.Tensor, temp: Optional[dict]) -> torch.Tensor:
    if not temp:
        return torch.ones(positions.shape, dtype=F64)
    return 1.0 + float(temp["coef"]) * torch.log(torch.floor((positions.to(F64) + 1.0) / int(temp["every"])) + 1.0)


def two_maps(q, k, v, scale) -> Tuple[torch.Tensor, torch.Tensor]:
    """q: [T, heads, 2, dim], k: [T, kv, 2, dim], v: [T, kv, vdim]: both maps' outputs [T, heads, vdim]."""
    t, heads = q.shape[:2]
    of = torch.arange(heads) // (heads // k.shape[1])
    mask = torch.ones(t, t, dtype=torch.bool).tril()
    out = []
    for m in range(2):
        s = torch.einsum("ihd,jhd->hij", q[:, :, m], k[:, of, m]) * scale
        out.append(torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~mask, -math.inf), -1), v[:, of]))
    return out[0], out[1]


def difference_factor(lq1, lk1, lq2, lk2, diff) -> float:
    dot = lambda a, b: float((a.to(F64) * b.to(F64)).sum())                        # noqa: E731
    return math.exp(dot(lq1, lk1)) - math.exp(dot(lq2, lk2)) + float(diff)


def attention(h, w, p, mx, eps) -> torch.Tensor:
    t = h.shape[0]
    heads, kv, dim, vdim = (int(mx[x]) for x in ("heads", "kv_heads", "dim", "vdim"))
    q = linear(h, w[p + "q"], w[p + "q.b"]).view(t, heads, 2, dim)
    k = linear(h, w[p + "k"], w[p + "k.b"]).view(t, kv, 2, dim)
    v = linear(h, w[p + "v"], w[p + "v.b"]).view(t, kv, vdim)
    q = q * query_temperature(torch.arange(t), mx.get("q_temp"))[:, None, None, None]
    a1, a2 = two_maps(q, k, v, float(mx["scale"]))
    diff = float(mx["diff"])
    lam = difference_factor(*(w[p + x] for x in ("lq1", "lk1", "lq2", "lk2")), diff)
    o = unit_rms(a1 - lam * a2, eps) * (1.0 - diff)
    return linear(o.reshape(t, heads * vdim), w[p + "o"], w[p + "o.b"])


def expert(x, w, p, limit) -> torch.Tensor:
    limit = math.inf if limit is None else float(limit)
    g = linear(x, w[p + "gate"]).clamp(max=limit)
    u = linear(x, w[p + "up"]).clamp(min=-limit, max=limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1.0), w[p + "down"])


def route(h, w_router, correction, rt) -> Tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """``(chosen [T, top], weights [T, top], margin [T])``; the margin says by how much the closest decision (a group kept or
    not, an expert chosen or not) was taken, in choice scores."""
    s = torch.softmax(linear(h, w_router), -1)
    c = s + correction.to(F64)
    t, e = c.shape
    margin = torch.full((t,), math.inf, dtype=F64)
    gr = rt.get("groups")
    if gr:
        count, keep = int(gr["count"]), int(gr["keep"])
        best = c.view(t, count, e // count).max(-1).values
        order, idx = best.sort(-1, descending=True)
        if keep < count:
            margin = torch.minimum(margin, order[:, keep - 1] - order[:, keep])
        stays = torch.zeros(t, count, dtype=torch.bool).scatter_(1, idx[:, :keep], True)
        c = c.masked_fill(~stays.repeat_interleave(e // count, 1), -math.inf)
    top = int(rt["top"])
    v, chosen = c.sort(-1, descending=True)
    if top < e:
        margin = torch.minimum(margin, v[:, top - 1] - v[:, top])
    chosen = chosen[:, :top]
    return chosen, s.gather(1, chosen) * float(rt.get("scale") or 1.0), margin


def mixture(h, w, p, ml, margins: Optional[list] = None) -> torch.Tensor:
    rt = ml["router"]
    h = h.to(F64)
    chosen, weight, margin = route(h, w[p + "router"], w[p + "correction"], rt)
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in range(int(rt["experts"]) + int(rt.get("identity") or 0)):
        t, j = (chosen == e).nonzero(as_tuple=True)
        if len(t):
            y = expert(h[t], w, p + f"e{e}.", ml["expert"].get("limit")) if e < int(rt["experts"]) else h[t]
            out.index_add_(0, t, y * weight[t, j][:, None])
    return out


# ---- the model ----------------------------------------------------------------------------------

MIXERS = {"mamba2": mamba2, "attention": attention}


def forward(w: Dict[str, torch.Tensor], cfg: dict, tokens: Sequence[int], layers_out: Optional[list] = None,
            margins: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence; ``layers_out`` receives x after every layer, ``margins`` every router's
    margins (``route``)."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"].to(F64)[torch.as_tensor(list(tokens), dtype=torch.long)]
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[lay["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", lay["mixer"], eps)
        if lay.get("mlp"):
            x = x + mixture(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", lay["mlp"], margins)
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(rms_norm(x, w["final.norm"], eps), w["embed"])


def generate(w, cfg, prompt, n_new) -> List[int]:
    """Greedy continuation, the whole sequence again for every token."""
    out = list(prompt)
    for _ in range(n_new):
        out.append(int(forward(w, cfg, out)[-1].argmax()))
    return out[len(prompt):]
