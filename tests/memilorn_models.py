"""Small Memilorn configurations with random weights for the tests: written as a model folder (config.json and
model.safetensors under the design's tensor names) so that the library loads them as it loads any checkpoint."""
import json
import os

import torch


def mlstm(heads, dim, vdim, cap=12.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": float(cap)}}


def latent(heads, dim, vdim, rank, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank,
                                                  "scale": float(scale if scale is not None else dim ** -0.5)}}


def attention(heads, kv_heads, dim, vdim, rot=None, base=10000.0, scale=None, cap=20.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(scale if scale is not None else dim ** -0.5)}
    if cap:
        m["softcap"] = float(cap)
    if rot:
        m["rot"] = {"base": base, "dims": rot}
    return {"type": "attention", "mixer": m}


def moe(experts, top, ff, limit=1.5, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": float(limit)}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": float(shared[1])}
    return m


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def config(layers, *, vocab, width, eps=1e-5, loop=None):
    c = {"architecture": "Memilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def _mixed():
    ls = [
        layer(attention(4, 2, 16, 24, 8, base=500.0, scale=0.3, cap=5.0), moe(6, 2, 24, 1.2, shared=(40, 0.8))),
        layer(mlstm(3, 16, 40, cap=8.0), moe(5, 1, 32, 2.5, shared=(16, 3.0))),
        layer(latent(5, 24, 16, 32, scale=0.25), None),
        layer(mlstm(2, 32, 8, cap=15.0), moe(4, 3, 16, 0.7)),
        layer(attention(6, 3, 8, 8, 2, base=30.0, cap=1.5), moe(3, 3, 24, 1.0, shared=(8, 5.0))),
    ]
    return config(ls, vocab=179, width=88, loop=(1, 4, 3))


def _tensor():
    # sizes that the tensor-core kernels take: heads in steps of 16, a latent of 64 and of 128 elements, experts in steps of 8
    ls = [
        layer(latent(4, 32, 48, 128), moe(8, 2, 64, 1.0, shared=(96, 1.5))),
        layer(mlstm(2, 64, 128, cap=10.0), moe(4, 1, 128, 2.0, shared=(64, 1.0))),
        layer(attention(8, 2, 64, 32, 32, base=250000.0, scale=0.15, cap=30.0), moe(8, 3, 32, 1.5)),
        layer(latent(6, 16, 16, 64), moe(6, 2, 48, 0.9, shared=(32, 2.0))),
        layer(attention(5, 5, 32, 80, 32, base=9000.0, cap=10.0), None),
        layer(attention(6, 1, 128, 128, 64, base=1000.0, scale=0.1, cap=50.0), moe(4, 2, 64, 1.0)),
    ]
    return config(ls, vocab=310, width=128, eps=1e-6, loop=(0, 2, 2))


def _odd():
    # sizes that fit no vector access and no tensor-core tile; one head; no rotation; no loop; more values than keys; every
    # expert chosen; a mixer whose sizes are all one number; no cap on the scores
    ls = [
        layer(mlstm(1, 10, 7, cap=3.0), moe(3, 3, 10, 1.0, shared=(6, 0.5))),
        layer(attention(3, 1, 10, 6, 6, base=77.0, cap=0.0), moe(2, 1, 6, 0.9)),
        layer(latent(1, 9, 14, 11), moe(1, 1, 5, 1.1, shared=(5, 1.1))),
        layer(attention(1, 1, 12, 20, cap=2.0), None),
        layer(mlstm(5, 6, 6, cap=20.0), None),
    ]
    return config(ls, vocab=101, width=50, eps=1e-4)


# Every size differs between the configurations and from one layer to the next; none is a size of a published model.
CONFIGS = {"mixed": _mixed(), "tensor": _tensor(), "odd": _odd()}

RESERVED = 8      # see random_weights(steady_routing=True)


def random_weights(cfg, seed, *, steady_routing=False):
    """bfloat16-valued tensors by the design's names.  Spreads are chosen so that activations stay of order one, that gates open and
    close, that clamps and caps bite, and that the talking heads mix.

    ``steady_routing``: which experts a token gets hangs on the token alone, for comparisons in bfloat16 where the
    router's input is rounded.  The last ``RESERVED`` elements of the width hold a code of the token that no sublayer changes
    (the layer scales are zero there), the routers read those elements only, and their rows sum to zero, so that neither
    the mean that a layer norm takes off nor its divisor (nor the embedding added once more) changes an order."""
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

    def scale():
        t = normal((d,), 0.2, 0.6)
        if steady_routing:
            t[-RESERVED:] = 0.0
        return t

    for i, lay in enumerate(cfg["layers"]):
        m, p = lay["mixer"], f"l{i}."
        w[p + "norm1"], w[p + "ls1"] = normal((d,), 0.1, 1.0), scale()
        h, dq, dv = m["heads"], m["dim"], m["vdim"]
        if lay["type"] == "mlstm":
            for n, rows in (("q", h * dq), ("k", h * dq), ("v", h * dv), ("g", h * dv)):
                w[p + "mix." + n] = normal((rows, d), 1.2 * d ** -0.5)
            w[p + "mix.i"], w[p + "mix.f"] = normal((h, d), 1.5 * d ** -0.5), normal((h, d), d ** -0.5)
            w[p + "mix.i.b"], w[p + "mix.f.b"] = normal((h,), 1.0, -0.5), normal((h,), 2.0, 4.0)
            w[p + "mix.norm"] = normal((h * dv,), 0.2, 1.0)
        elif lay["type"] == "latent_attention":
            r = m["kv_rank"]
            w[p + "mix.q"], w[p + "mix.dkv"] = normal((h * dq, d), 1.5 * d ** -0.5), normal((r, d), d ** -0.5)
            w[p + "mix.dkv.norm"] = normal((r,), 0.1, 1.0)
            w[p + "mix.uk"], w[p + "mix.uv"] = normal((h * dq, r), 1.5 * r ** -0.5), normal((h * dv, r), r ** -0.5)
            w[p + "mix.g"] = normal((h, d), 1.5 * d ** -0.5)
        else:
            kv = m["kv_heads"]
            w[p + "mix.q"], w[p + "mix.k"] = normal((h * dq, d), 1.5 * d ** -0.5), normal((kv * dq, d), 1.5 * d ** -0.5)
            w[p + "mix.v"], w[p + "mix.g"] = normal((kv * dv, d), d ** -0.5), normal((h, d), 1.5 * d ** -0.5)
            w[p + "mix.sink"] = normal((h,), 1.0, 1.0)
            w[p + "mix.talk"] = (torch.eye(h) + 0.5 * torch.randn((h, h), generator=g)).to(torch.bfloat16)
        w[p + "mix.o"] = normal((d, h * dv), 1.5 * (h * dv) ** -0.5)
        ml = lay.get("mlp")
        if not ml:
            continue
        w[p + "norm2"], w[p + "ls2"] = normal((d,), 0.1, 1.0), scale()
        e_n, ff = ml["router"]["experts"], ml["expert"]["ff"]
        if steady_routing:
            router = torch.zeros((e_n, d))
            # entries of plus or minus one (and zero) sum to exactly nothing, also in bfloat16
            for e in range(e_n):
                perm = torch.randperm(RESERVED, generator=g)
                k = 1 + int(torch.randint(0, RESERVED // 2, (1,), generator=g))
                router[e, d - RESERVED + perm[:k]] = 1.0
                router[e, d - RESERVED + perm[k:2 * k]] = -1.0
            w[p + "mlp.router"] = router.to(torch.bfloat16)
            w[p + "norm2"][-RESERVED:] = 1.0
        else:
            w[p + "mlp.router"] = normal((e_n, d), 1.5 * d ** -0.5)
        for e in range(e_n):
            w[p + f"mlp.e{e}.gate"] = normal((ff, d), 1.5 * d ** -0.5)
            w[p + f"mlp.e{e}.up"] = normal((ff, d), 1.5 * d ** -0.5)
            w[p + f"mlp.e{e}.down"] = normal((d, ff), ff ** -0.5)
        if ml.get("shared"):
            sf = ml["shared"]["ff"]
            w[p + "mlp.shared.gate"], w[p + "mlp.shared.up"] = normal((sf, d), 1.5 * d ** -0.5), normal((sf, d), 1.5 * d ** -0.5)
            w[p + "mlp.shared.down"] = normal((d, sf), sf ** -0.5)
    return w


def write_model(llogos, folder, cfg, seed, weights=None, **kw):
    os.makedirs(folder, exist_ok=True)
    w = weights if weights is not None else random_weights(cfg, seed, **kw)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    llogos.weights.write_safetensors(os.path.join(folder, "model.safetensors"), w, {"format": "pt"})
    return w
