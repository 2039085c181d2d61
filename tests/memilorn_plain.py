"""A plain, slow implementation of the Memilorn decoder, for tests only: whole sequences, no cache, float64,
one function per mechanism, and no code shared with the library under test (it reads config.json's keys and
looks tensors up by name on its own).

The design in this file's notation (T tokens, width D, token ids ``tok``):

* ``L(x, w) = (x - mean) / sqrt(var + eps) * w`` with the population variance; ``U(x) = x / sqrt(mean(x^2) + eps)``.
* a layer: ``x <- x + ls1 * mixer(L(x, norm1))``, then, where it has a feed-forward, ``x <- x + ls2 * ff(L(x, norm2))``
  (``ls1`` and ``ls2`` are vectors of the width).
* the run order: layers ``start .. stop-1`` run ``times`` times; before the second and every later round the
  embedding's row ``embed[tok]`` is added to x once.
* mixer "mlstm": per head ``q = dim^-1/2 W_q h``, ``k = W_k h``, ``v = W_v h``, ``i = cap tanh((w_i . h + b_i) / cap)``,
  ``f = logsigmoid(cap tanh((w_f . h + b_f) / cap))``; from S = 0, n = 0, m = 0:
  ``m' = max(f + m, i)``, ``S' = e^{f + m - m'} S + e^{i - m'} k v^T``, ``n' = e^{f + m - m'} n + e^{i - m'} k``,
  ``o = S'^T q / (max(|n' . q|, e^{-m'}) + 1e-6)``; the output is ``W_o ([U(o)] * norm * sigmoid(W_g h))``.
* mixer "latent_attention": ``c = U(W_dkv h) * dkv.norm``; per head ``k = W_uk,h c``, ``v = W_uv,h c``; causal softmax of
  ``scale q . k``; every head's output times ``sigmoid(w_g,h . h)``; ``W_o``.
* mixer "attention": grouped-query heads, neighbouring elements of the first ``rot.dims`` rotated, scores
  ``s_h = cap tanh(scale q . k / cap)``, mixed over heads by ``talk``: ``s'_h = sum_g talk[h, g] s_g``; causal softmax whose
  denominator has one more summand ``e^{sink_h}``; every head's output times ``sigmoid(w_g,h . h)``; ``W_o``.
* feed-forward "moe": ``s = sigmoid(router h)``, the ``top`` largest; ``sum_e expert_e(s_e h)`` (the weight is on the input)
  plus ``shared(h)``; an expert is ``down(g sigmoid(1.702 g) (u + 1))`` with ``g = min(gate h, limit)`` and
  ``u = clamp(up h, -limit, limit)``.
* output: ``embed L(x, final.norm)``.
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


def layer_norm(x, weight, eps):
    x = x.to(F64)
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight.to(F64)


def unit_rms(x, eps):
    x = x.to(F64)
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x: [T, heads, d]; element 2i of the first ``rot.dims`` turns with element 2i + 1."""
    x = x.to(F64).clone()
    if not rot:
        return x
    dims = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims)
    ang = positions.to(F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., 0:dims:2].clone(), x[..., 1:dims:2].clone()
    x[..., 0:dims:2] = u * c - v * s
    x[..., 1:dims:2] = v * c + u * s
    return x


def head_gates(h, w):
    return torch.sigmoid(linear(h, w))


def mixed_scores(scores: torch.Tensor, cap, talk: Optional[torch.Tensor]) -> torch.Tensor:
    """scores: [H, T, S], already scaled; the cap, then every head's scores as a mixture of all heads'."""
    if cap:
        scores = float(cap) * torch.tanh(scores / float(cap))
    if talk is not None:
        scores = torch.einsum("hg,gts->hts", talk.to(F64), scores)
    return scores


def sink_softmax(scores: torch.Tensor, hidden: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """scores: [H, T, S]; ``hidden`` marks keys that a query does not see; ``sink``: [H] or None."""
    s = scores.masked_fill(hidden, -math.inf)
    if sink is None:
        return torch.softmax(s, dim=-1)
    extra = sink.to(F64)[:, None, None].expand(s.shape[0], s.shape[1], 1)
    return torch.softmax(torch.cat([s, extra], dim=-1), dim=-1)[..., :-1]


def attention(h, w, p, mx, pos=None, probs_out: Optional[list] = None) -> torch.Tensor:
    t = h.shape[0]
    heads, kvh, dim, vdim = int(mx["heads"]), int(mx["kv_heads"]), int(mx["dim"]), int(mx["vdim"])
    pos = torch.arange(t) if pos is None else pos
    q = rotate_neighbours(linear(h, w[p + "q"]).view(t, heads, dim), pos, mx.get("rot"))
    k = rotate_neighbours(linear(h, w[p + "k"]).view(t, kvh, dim), pos, mx.get("rot"))
    v = linear(h, w[p + "v"]).view(t, kvh, vdim)
    rep = heads // kvh
    k, v = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = mixed_scores(torch.einsum("thd,shd->hts", q, k) * float(mx["scale"]), mx.get("softcap"), w.get(p + "talk"))
    i = torch.arange(t)
    pr = sink_softmax(s, i[None, :] > i[:, None], w.get(p + "sink"))
    if probs_out is not None:
        probs_out.append(pr)
    out = torch.einsum("hts,shd->thd", pr, v) * head_gates(h, w[p + "g"])[:, :, None]
    return linear(out.reshape(t, heads * vdim), w[p + "o"])


def latent_attention(h, w, p, mx, eps, probs_out: Optional[list] = None) -> torch.Tensor:
    t = h.shape[0]
    heads, dim, vdim = int(mx["heads"]), int(mx["dim"]), int(mx["vdim"])
    q = linear(h, w[p + "q"]).view(t, heads, dim)
    c = unit_rms(linear(h, w[p + "dkv"]), eps) * w[p + "dkv.norm"].to(F64)
    k = linear(c, w[p + "uk"]).view(t, heads, dim)
    v = linear(c, w[p + "uv"]).view(t, heads, vdim)
    i = torch.arange(t)
    pr = sink_softmax(torch.einsum("thd,shd->hts", q, k) * float(mx["scale"]), i[None, :] > i[:, None], None)
    if probs_out is not None:
        probs_out.append(pr)
    out = torch.einsum("hts,shd->thd", pr, v) * head_gates(h, w[p + "g"])[:, :, None]
    return linear(out.reshape(t, heads * vdim), w[p + "o"])


def log_gates(h, w, p, cap) -> Tuple[torch.Tensor, torch.Tensor]:
    """``(i, f)``, each [T, heads]: the logarithms of the input and the forget gate."""
    cap = float(cap)
    i = cap * torch.tanh(linear(h, w[p + "i"], w[p + "i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh(linear(h, w[p + "f"], w[p + "f.b"]) / cap))
    return i, f


def matrix_memory(q, k, v, i, f, state=None):
    """The recurrence, token by token.  q, k: [T, H, d] (q already scaled), v: [T, H, e], i, f: [T, H].
    Returns the outputs [T, H, e] and the last ``(S, n, m)``."""
    t, heads, d = q.shape
    if state is None:
        state = (torch.zeros(heads, d, v.shape[-1], dtype=F64), torch.zeros(heads, d, dtype=F64), torch.zeros(heads, dtype=F64))
    s, n, m = state
    out = torch.zeros(t, heads, v.shape[-1], dtype=F64)
    for x in range(t):
        new = torch.maximum(f[x] + m, i[x])
        keep, take = torch.exp(f[x] + m - new), torch.exp(i[x] - new)
        s = keep[:, None, None] * s + take[:, None, None] * k[x][:, :, None] * v[x][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[x]
        m = new
        dots = (n * q[x]).sum(-1).abs()
        out[x] = torch.einsum("hde,hd->he", s, q[x]) / (torch.maximum(dots, torch.exp(-m)) + 1e-6)[:, None]
    return out, (s, n, m)


def mlstm(h, w, p, mx, eps) -> torch.Tensor:
    t = h.shape[0]
    heads, dim, vdim = int(mx["heads"]), int(mx["dim"]), int(mx["vdim"])
    q = linear(h, w[p + "q"]).view(t, heads, dim) * dim ** -0.5
    k = linear(h, w[p + "k"]).view(t, heads, dim)
    v = linear(h, w[p + "v"]).view(t, heads, vdim)
    i, f = log_gates(h, w, p, mx["gate_cap"])
    o, _ = matrix_memory(q, k, v, i, f)
    o = unit_rms(o, eps).reshape(t, heads * vdim) * w[p + "norm"].to(F64) * torch.sigmoid(linear(h, w[p + "g"]))
    return linear(o, w[p + "o"])


def expert(x, w, p, limit) -> torch.Tensor:
    limit = float(limit)
    g = linear(x, w[p + "gate"]).clamp(max=limit)
    u = linear(x, w[p + "up"]).clamp(min=-limit, max=limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1.0), w[p + "down"])


def route(h, w_router, top) -> Tuple[torch.Tensor, torch.Tensor]:
    """``(experts, scores)``, each [T, top]: the largest sigmoids, as they are."""
    s, c = torch.sigmoid(linear(h, w_router)).topk(int(top), dim=-1)
    return c, s


def route_margin(h, w_router, top) -> torch.Tensor:
    """[T]: by how much the last chosen expert's logit beats the next one's (infinite where nothing is left out)."""
    z = linear(h, w_router)
    if int(top) == z.shape[-1]:
        return torch.full((z.shape[0],), math.inf, dtype=F64)
    v = z.topk(int(top) + 1, dim=-1).values
    return v[:, -2] - v[:, -1]


def mixture(h, w, p, ml, margins: Optional[list] = None) -> torch.Tensor:
    chosen, score = route(h, w[p + "router"], ml["router"]["top"])
    if margins is not None:
        margins.append(route_margin(h, w[p + "router"], ml["router"]["top"]))
    out = torch.zeros_like(h, dtype=F64)
    for e in range(int(ml["router"]["experts"])):
        t, j = (chosen == e).nonzero(as_tuple=True)
        if len(t):
            out.index_add_(0, t, expert(h[t] * score[t, j][:, None], w, p + f"e{e}.", ml["expert"]["limit"]))
    if ml.get("shared"):
        out = out + expert(h, w, p + "shared.", ml["shared"]["limit"])
    return out


# ---- the model ----------------------------------------------------------------------------------

def run_order(cfg: dict) -> List[Tuple[int, bool]]:
    """``(layer, whether the embedding's row is added ahead of it)`` in the order the layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    order = [(i, False) for i in range(start)]
    for r in range(times):
        order += [(i, r > 0 and i == start) for i in range(start, stop)]
    return order + [(i, False) for i in range(stop, n)]


def forward(w: Dict[str, torch.Tensor], cfg: dict, tokens: Sequence[int], layers_out: Optional[list] = None,
            margins: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence; ``layers_out`` receives x after every layer that runs, ``margins`` every
    router's margins (``route_margin``)."""
    eps = float(cfg["norm"]["eps"])
    e = w["embed"].to(F64)[torch.as_tensor(list(tokens), dtype=torch.long)]
    x = e.clone()
    for i, again in run_order(cfg):
        if again:
            x = x + e
        lay, p = cfg["layers"][i], f"l{i}."
        h, mx = layer_norm(x, w[p + "norm1"], eps), lay["mixer"]
        if lay["type"] == "mlstm":
            y = mlstm(h, w, p + "mix.", mx, eps)
        elif lay["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", mx, eps)
        else:
            y = attention(h, w, p + "mix.", mx)
        x = x + y * w[p + "ls1"].to(F64)
        if lay.get("mlp"):
            x = x + mixture(layer_norm(x, w[p + "norm2"], eps), w, p + "mlp.", lay["mlp"], margins) * w[p + "ls2"].to(F64)
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(layer_norm(x, w["final.norm"], eps), w["embed"])


def generate(w, cfg, prompt, n_new) -> List[int]:
    """Greedy continuation, the whole sequence again for every token."""
    out = list(prompt)
    for _ in range(n_new):
        out.append(int(forward(w, cfg, out)[-1].argmax()))
    return out[len(prompt):]
