"""Small Penasun configurations with random weights for the tests: written as a model folder (config.json and
model.safetensors under the design's tensor names) so that the library loads them as it loads any checkpoint."""
import json
import os

import torch


def mamba(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def attention(heads, kv_heads, dim, vdim, scale=None, diff=0.5, temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(scale if scale is not None else dim ** -0.5),
         "diff": diff}
    if temp:
        m["q_temp"] = dict(zip(("coef", "every"), temp))
    return {"type": "attention", "mixer": m}


def moe(experts, top, ff, limit=1.5, identity=0, groups=None, scale=1.0):
    r = {"experts": experts, "top": top, "identity": identity, "scale": float(scale)}
    if groups:
        r["groups"] = dict(zip(("count", "keep"), groups))
    return {"kind": "moe", "router": r, "expert": {"ff": ff, "limit": float(limit)}}


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def config(layers, *, vocab, width, eps=1e-5):
    return {"architecture": "Penasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def _mixed():
    ls = [
        layer(mamba(6, 10, 12, 3, 4, 4), moe(7, 3, 24, 1.2, identity=3, groups=(5, 3), scale=1.7)),
        layer(attention(4, 2, 12, 20, scale=0.4, diff=0.3, temp=(0.25, 37)), moe(5, 2, 32, 2.5, identity=1, groups=(3, 2), scale=2.2)),
        layer(mamba(3, 24, 20, 1, 2, 1), None),
        layer(attention(6, 3, 8, 16, diff=0.75, temp=(0.6, 90)), moe(3, 2, 16, 0.7, identity=5, groups=(2, 1))),
        layer(mamba(4, 8, 40, 2, 3, 8), moe(4, 4, 16, 0.9)),
    ]
    return config(ls, vocab=179, width=88)


def _tensor():
    # sizes that the tensor-core kernels take: both maps of a key head together 64, 128, 80 and 48 elements beside values of that
    # size, and one layer whose values have another; states in steps of 16 rows and 8 columns; experts in steps of 8
    ls = [
        layer(attention(4, 2, 32, 64, scale=0.3, diff=0.4, temp=(0.3, 64)), moe(6, 2, 64, 1.0, identity=2, groups=(4, 2), scale=1.5)),
        layer(mamba(4, 32, 64, 2, 4, 2), moe(4, 2, 128, 2.0, identity=4)),
        layer(attention(4, 1, 64, 128, diff=0.6, temp=(0.2, 50)), None),
        layer(mamba(6, 16, 16, 3, 3, 3), moe(8, 3, 32, 1.5, identity=1, groups=(3, 2), scale=2.0)),
        layer(attention(6, 2, 24, 48, diff=0.2), moe(4, 1, 48, 0.9, identity=1)),
        layer(mamba(2, 64, 128, 1, 4, 2), None),
        layer(attention(3, 3, 40, 80, scale=0.2, diff=0.8, temp=(0.4, 100)), None),
        layer(mamba(5, 8, 144, 1, 2, 5), moe(4, 2, 64, 1.0, identity=2, groups=(2, 1))),
        layer(attention(2, 1, 16, 48, diff=0.5), None),
    ]
    return config(ls, vocab=310, width=128, eps=1e-6)


def _odd():
    # sizes that fit no vector access and no tensor-core tile; one head; one tap; more taps than a short step has tokens; no
    # temperature; a mixture without identity experts, one whose every expert is chosen, one of a single expert, one of which
    # all groups are kept; a state of one row
    ls = [
        layer(mamba(1, 7, 10, 1, 1, 1), moe(3, 3, 10, 1.0)),
        layer(attention(3, 1, 5, 6, diff=0.0), moe(1, 1, 6, 0.9, identity=1, scale=3.0)),
        layer(mamba(3, 5, 1, 3, 6, 3), moe(1, 1, 5, 1.1)),
        layer(attention(1, 1, 6, 20, diff=0.9, temp=(1.1, 1)), None),
        layer(mamba(2, 9, 33, 2, 4, 2), moe(2, 2, 7, 2.0, identity=2, groups=(2, 2), scale=0.5)),
    ]
    return config(ls, vocab=101, width=50, eps=1e-4)


# Every size differs between the configurations and from one layer to the next; none is a size of a published model.
CONFIGS = {"mixed": _mixed(), "tensor": _tensor(), "odd": _odd()}

RESERVED = 8      # see random_weights(steady_routing=True)


def random_weights(cfg, seed, *, steady_routing=False):
    """bfloat16-valued tensors by the design's names.  Spreads are chosen so that activations stay of order one, that states forget
    within tens or within hundreds of tokens, that clamps bite, that the two maps differ, and that corrections change choices and make
    most choice scores negative.

    ``steady_routing``: which experts a token gets hangs on the token alone, for comparisons in bfloat16 where the
    router's input is rounded.  The last ``RESERVED`` elements of the width hold a code of the token that no sublayer turns
    (the output projections are zero there; an identity expert only stretches it), and the routers read those elements only."""
    g = torch.Generator().manual_seed(seed)

    def normal(shape, std, mean=0.0):
        return (mean + std * torch.randn(shape, generator=g)).to(torch.bfloat16)

    d, v = cfg["width"], cfg["vocab"]
    w = {"embed": normal((v, d), 1.0), "final.norm": normal((d,), 0.1, 1.0)}
    w["final.norm"] = (w["final.norm"].float() * 0.2).to(torch.bfloat16)
    if steady_routing:
        code = 1.0 + torch.rand((v, RESERVED), generator=g)
        sign = torch.where(torch.rand((v, RESERVED), generator=g) < 0.5, -1.0, 1.0)
        w["embed"][:, -RESERVED:] = (1.5 * code * sign).to(torch.bfloat16)
        w["final.norm"][-RESERVED:] = 0.0
    for i, lay in enumerate(cfg["layers"]):
        m, p = lay["mixer"], f"l{i}."
        q = p + "mix."
        w[p + "norm1"] = normal((d,), 0.1, 1.0)
        h, dv = m["heads"], m["vdim"]
        inner = h * dv
        if lay["type"] == "mamba2":
            channels = inner + 2 * m["groups"] * m["state"]
            w[q + "in"] = normal((inner + channels + h, d), 1.2 * d ** -0.5)
            w[q + "conv"], w[q + "conv.b"] = normal((channels, m["conv"]), m["conv"] ** -0.5), normal((channels,), 0.3)
            w[q + "dt_bias"] = normal((h,), 1.0, -2.0)
            w[q + "A_log"] = normal((h,), 1.5, -0.5)
            w[q + "D"], w[q + "norm"] = normal((h,), 0.5, 1.0), normal((inner,), 0.2, 1.0)
            w[q + "o"] = normal((d, inner), inner ** -0.5)
        else:
            kv, dq = m["kv_heads"], 2 * m["dim"]
            w[q + "q"], w[q + "k"] = normal((h * dq, d), 1.5 * d ** -0.5), normal((kv * dq, d), 1.5 * d ** -0.5)
            w[q + "v"] = normal((kv * dv, d), d ** -0.5)
            for n, rows in (("q", h * dq), ("k", kv * dq), ("v", kv * dv)):
                w[q + n + ".b"] = normal((rows,), 0.5)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[q + n] = normal((m["dim"],), 0.6 * m["dim"] ** -0.25)
            w[q + "o"], w[q + "o.b"] = normal((d, inner), inner ** -0.5), normal((d,), 0.3)
            if steady_routing:
                w[q + "o.b"][-RESERVED:] = 0.0
        if steady_routing:
            w[q + "o"][-RESERVED:] = 0.0
        ml = lay.get("mlp")
        if not ml:
            continue
        w[p + "norm2"] = normal((d,), 0.1, 1.0)
        e_n, ff = ml["router"]["experts"], ml["expert"]["ff"]
        routed = e_n + ml["router"].get("identity", 0)
        if steady_routing:
            router = torch.zeros((routed, d))
            router[:, -RESERVED:] = torch.randn((routed, RESERVED), generator=g)
            w[p + "mlp.router"] = router.to(torch.bfloat16)
            w[p + "norm2"][-RESERVED:] = 1.0
        else:
            w[p + "mlp.router"] = normal((routed, d), 1.5 * d ** -0.5)
        w[p + "mlp.correction"] = normal((routed,), 0.3, -0.4)
        for e in range(e_n):
            w[p + f"mlp.e{e}.gate"] = normal((ff, d), 1.5 * d ** -0.5)
            w[p + f"mlp.e{e}.up"] = normal((ff, d), 1.5 * d ** -0.5)
            w[p + f"mlp.e{e}.down"] = normal((d, ff), ff ** -0.5)
            if steady_routing:
                w[p + f"mlp.e{e}.down"][-RESERVED:] = 0.0
    return w


def write_model(llogos, folder, cfg, seed, weights=None, **kw):
    os.makedirs(folder, exist_ok=True)
    w = weights if weights is not None else random_weights(cfg, seed, **kw)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    llogos.weights.write_safetensors(os.path.join(folder, "model.safetensors"), w, {"format": "pt"})
    return w
