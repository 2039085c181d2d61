"""The Memilorn decoder on the GPU against the plain implementation in memilorn_plain.py, in float32 and bfloat16: every
mechanism's kernel alone; whole prompts; prompts against token-by-token decoding; prompts in portions down to two tokens;
batches of unequal requests against each alone, with slots, pages and state rows used again; a far key among hundreds in
both attentions, and one that only another head's scores find; what a memory wrote long ago; the first tokens; long
decoding; sizes that differ from layer to layer; greedy generation through the library's entry point."""
import math

import pytest
import torch

import memilorn_models as MM
import memilorn_plain as MP

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
IDS = ["f32", "bf16"]
F64 = torch.float64

# float32: every logit within 1e-4 of the request's largest |logit|.  bfloat16, relative to the root mean square of all
# compared logits: the root-mean-square error of every position within 1e-1 and of the positions on average within
# 3.5e-2, every logit within 1.5e-1 of the largest.  The models of one layer that are made to show a fault (TIGHT) stay
# within 2.5e-2 and 5e-2.
TOL = {torch.float32: (1e-4, 1e-4, 1e-4), torch.bfloat16: (1e-1, 3.5e-2, 1.5e-1)}
TIGHT = {torch.float32: (1e-4, 1e-4, 1e-4), torch.bfloat16: (2.5e-2, 2.5e-2, 5e-2)}
MARGIN = 0.05          # bfloat16: no router of a compared sequence decides by less than this (in logits)


def ops_module():
    from importlib import import_module
    return import_module("daisi-llogos_b200.kernels.ops")


def close(got, ref, dtype, what=(), tol=TOL):
    got = got.detach().to("cpu", F64).reshape(ref.shape)
    rms_tol, mean_tol, max_tol = tol[dtype]
    per_position = (got - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
    rms, mean = float(per_position.max()), float(per_position.mean())
    worst = float((got - ref).abs().max() / ref.abs().max())
    if per_position.numel() < 16:
        mean_tol = rms_tol
    assert rms <= rms_tol and mean <= mean_tol and worst <= max_tol, (*what, "rms", rms, "mean", mean, "max", worst)


def near(got, ref, tol, what=""):
    err = float((got.detach().to("cpu", F64) - ref.to(F64)).abs().max() / max(1.0, float(ref.abs().max())))
    assert err <= tol, (what, err)


@pytest.fixture(scope="module")
def models(llogos, tmp_path_factory):
    """(name, dtype) -> (folder, config, weights as float tensors); bfloat16 takes routers that read a code of the token
    (``steady_routing``), float32 routers that hang on everything."""
    out = {}
    for i, (name, cfg) in enumerate(MM.CONFIGS.items()):
        for dtype in DTYPES:
            d = str(tmp_path_factory.mktemp(f"memilorn_{name}_{IDS[DTYPES.index(dtype)]}"))
            w = MM.write_model(llogos, d, cfg, seed=370 + i, steady_routing=dtype == torch.bfloat16)
            out[name, dtype] = (d, cfg, {k: v.float() for k, v in w.items()})
    return out


@pytest.fixture(scope="module")
def engines(llogos, models):
    kept = {}

    def get(name, dtype, graphs=True, max_tokens=64 * 40):
        key = (name, dtype, graphs, max_tokens)
        if key not in kept:
            model = llogos.weights.load_model(models[name, dtype][0], dtype=dtype, device="cuda:0")
            kept[key] = llogos.engine.Engine(model, max_tokens=max_tokens, use_graphs=graphs)
        return kept[key]
    return get


_refs, _tokens, _pools = {}, {}, {}


def sequence(models, name, dtype, n, seed):
    """(tokens, plain logits) of a random sequence.  In bfloat16 the sequence is drawn again, without the tokens that met a
    close call in a router, until no router decides by less than ``MARGIN``."""
    key = (name, dtype, n, seed)
    if key in _tokens:
        return _tokens[key], _refs[key]
    _, cfg, w = models[name, dtype]
    pool = _pools.setdefault((name, dtype), list(range(cfg["vocab"])))
    for attempt in range(40):
        g = torch.Generator().manual_seed(seed * 1000 + attempt)
        toks = [pool[i] for i in torch.randint(0, len(pool), (n,), generator=g).tolist()]
        margins = []
        ref = MP.forward(w, cfg, toks, margins=margins)
        if dtype != torch.bfloat16 or not margins:
            break
        worst = torch.stack(margins).min(0).values
        if float(worst.min()) > MARGIN:
            break
        bad = {toks[i] for i in torch.nonzero(worst <= 1.5 * MARGIN).flatten().tolist()}
        pool[:] = [t for t in pool if t not in bad]
        assert len(pool) > 20, "too few tokens are left whose routing is steady"
    else:
        raise AssertionError("no sequence without a close call in a router was found")
    _tokens[key], _refs[key] = toks, ref
    return toks, ref


def layout(counts, before, slots):
    """Device tensors of a step's packed layout: (slots, cu_tokens, seq_of_token, len_before, positions)."""
    I = lambda xs: torch.tensor(list(xs), dtype=torch.int32, device="cuda")
    cu = [0]
    for c in counts:
        cu.append(cu[-1] + c)
    seq = [b for b, c in enumerate(counts) for _ in range(c)]
    pos = [p for lb, c in zip(before, counts) for p in range(lb, lb + c)]
    return I(slots), I(cu), I(seq), I(before), I(pos)


# ---- mechanisms alone --------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("hidden", [50, 72, 90, 1024, 4100])
def test_layer_norm_without_a_bias_and_sets_with_gains(dtype, hidden):
    ops = ops_module()
    g = torch.Generator().manual_seed(hidden)
    n = 9
    res = torch.randn(n, hidden, generator=g) + 3.0
    t1, t2, t3 = (torch.randn(s, n, hidden, generator=g) for s in (2, 1, 3))
    k1, k3, w = (torch.randn(hidden, generator=g) for _ in range(3))
    for gains, scale in (([k1, None, k3], 1.0), ([None, k1, None], -0.5), (None, 1.0)):
        ks = gains or [None] * 3
        total = sum(t.double().sum(0) * (1.0 if k is None else k.double()) for t, k in zip((t1, t2, t3), ks))
        want = res.double() + scale * total
        for rows in (None, [7, 0, 3]):
            idx = slice(None) if rows is None else rows
            dev = res.clone().cuda()
            out = torch.empty(n if rows is None else len(rows), hidden, dtype=dtype, device="cuda")
            kw = {} if gains is None else {"gains": [None if k is None else k.cuda() for k in gains]}
            ops.add_layernorm(dev, [t.cuda() for t in (t1, t2, t3)], scale, w.cuda(), None, 1e-5, out,
                              None if rows is None else torch.tensor(rows, dtype=torch.int32, device="cuda"), **kw)
            near(dev[idx], want[idx], 1e-5, "sum")
            near(out, MP.layer_norm(want[idx], w, 1e-5), 2e-5 if dtype == torch.float32 else 1e-2, "norm")


def _form_of(g, u, alpha, limit, off):
    g = g.clamp(max=limit)
    return g * torch.sigmoid(alpha * g) * (u.clamp(-limit, limit) + off)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("n,hidden,inner", [(1, 64, 40), (9, 128, 96), (70, 72, 200), (300, 128, 272), (600, 256, 64), (20, 50, 14)])
def test_gated_product_in_a_clamped_form(llogos, dtype, n, hidden, inner):
    """The dense gated product (few rows, many rows, sizes no tensor core takes) with gate and up values on both sides of the clamps."""
    from importlib import import_module
    linear = import_module("daisi-llogos_b200.kernels.linear")
    ctx_mod = import_module("daisi-llogos_b200.engine.context")
    ops = ops_module()
    g = torch.Generator().manual_seed(n)
    x = torch.randn(n, hidden, generator=g).to(dtype)
    wg, wu = ((1.5 * hidden ** -0.5 * torch.randn(inner, hidden, generator=g)).to(dtype) for _ in range(2))

    class Ctx:
        pass
    ctx = Ctx()
    ctx.ops = ops
    ws = ctx_mod.Workspace(torch.device("cuda"))
    ctx.buffer = lambda name, shape, dt=None, zero=False: ws.get(name, tuple(shape), dt or dtype, zero)
    for alpha, limit, off in ((1.702, 0.9, 1.0), (0.5, 2.5, 0.0)):
        out = torch.empty(n, inner, dtype=dtype, device="cuda")
        linear.gated_linear(ctx, x.cuda(), linear.gated_layout(wg.cuda(), wu.cuda()), out, form=ops.GateForm(alpha, limit, off))
        want = _form_of(MP.linear(x, wg), MP.linear(x, wu), alpha, limit, off)
        near(out, want, 2e-5 if dtype == torch.float32 else 1e-2, (alpha, limit))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("n,n_exp,top,hidden,inner", [(1, 4, 1, 64, 32), (40, 5, 2, 72, 48), (37, 3, 3, 50, 10), (600, 2, 1, 128, 192), (300, 2, 2, 64, 136)])
def test_experts_with_the_weight_on_their_input(llogos, dtype, n, n_exp, top, hidden, inner):
    """Routing by sigmoids as they are, the layout with every row's weight, the gated product in its clamped form and the plain
    sum, as the feed-forward part runs them (tiles of 32 rows, and of 128 for the grouped tcgen05 product)."""
    from importlib import import_module
    base = import_module("daisi-llogos_b200.parts.base")
    moe = import_module("daisi-llogos_b200.parts.moe")
    ctx_mod = import_module("daisi-llogos_b200.engine.context")
    ops = ops_module()
    g = torch.Generator().manual_seed(n + n_exp)
    env = base.BuildEnv(dtype=dtype, device=torch.device("cuda"), ops=ops, encodings={})
    params = {"hidden_size": hidden, "num_experts": n_exp, "top": top, "expert_size": inner, "score": "sigmoid", "normalize": False,
              "weight_on": "input", "activation": "clamped", "gate_alpha": 1.702, "up_offset": 1.0, "limit": 0.7, "shared_size": 24,
              "shared_params": {"activation": "clamped", "gate_alpha": 1.702, "up_offset": 1.0, "limit": 1.9}}
    part = moe.MoeFeedForward(params, "", env)
    w = {}
    for name, d in part.tensors().items():
        w[name] = (1.5 * d.shape[-1] ** -0.5 * torch.randn(d.shape, generator=g)).to(dtype)
    if dtype == torch.bfloat16:                   # no close calls: the routers' logits are whole numbers apart
        w["router.weight"] = torch.zeros(n_exp, hidden, dtype=dtype)
        for e in range(n_exp):
            w["router.weight"][e, e] = 1.0
    part.bind({k: v.cuda() for k, v in w.items()})
    x = torch.randn(n, hidden, generator=g)
    if dtype == torch.bfloat16:
        x[:, :n_exp] = torch.stack([torch.randperm(n_exp, generator=g) for _ in range(n)]).float() * 0.5 - 1.0
    x = x.to(dtype)

    class Ctx:
        pass
    ctx = Ctx()
    ctx.ops, ctx.dtype = ops, dtype
    ws = ctx_mod.Workspace(torch.device("cuda"))
    ctx.buffer = lambda name, shape, dt=None, zero=False: ws.get(name, tuple(shape), dt or dtype, zero)
    got = part.forward(x.cuda(), ctx).data.sum(0)
    names = {"router": w["router.weight"]}
    for i in range(n_exp):
        for what in ("gate", "up", "down"):
            names[f"e{i}.{what}"] = w[f"experts.{i}.{what}_proj.weight"]
    for what in ("gate", "up", "down"):
        names[f"shared.{what}"] = w[f"shared:{what}_proj.weight"]
    ml = {"router": {"experts": n_exp, "top": top}, "expert": {"ff": inner, "limit": 0.7}, "shared": {"ff": 24, "limit": 1.9}}
    near(got, MP.mixture(x.double(), names, "", ml), 3e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("n_exp,top", [(8, 3), (9, 2), (6, 6), (40, 1)])
def test_routing_by_sigmoids_as_they_are(n_exp, top):
    ops = ops_module()
    g = torch.Generator().manual_seed(n_exp)
    n, hidden = 50, 40
    h, wr = torch.randn(n, hidden, generator=g), torch.randn(n_exp, hidden, generator=g) * 0.4
    idx, wt = MP.route(h, wr, top)
    rule = ops.RouterRule("sigmoid", weight_scale=1.0, normalize=False)
    for way in ("route", "topk"):
        choice = torch.empty(n, top, dtype=torch.int32, device="cuda")
        weight = torch.empty(n, top, device="cuda")
        if way == "route":
            ops.moe_route(h.cuda(), wr.cuda(), None, choice, weight, rule)
        else:
            z = h @ wr.t()
            ops.moe_topk(torch.stack([0.3 * z, 0.7 * z]).contiguous().cuda(), None, choice, weight, rule)
        assert torch.equal(choice.cpu().long(), idx), way
        near(weight, wt, 1e-5, way)


MEMORY_SIZES = [(3, 16, 24, (5, 1, 9)), (2, 32, 40, (300, 1, 130)), (2, 64, 300, (5, 2, 1)), (5, 6, 6, (129, 128)), (1, 128, 128, (3, 140)),
                (1, 200, 72, (17, 270)), (2, 10, 7, (1, 1, 1)), (2, 10, 300, (4, 70, 1))]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("nh,dim,vdim,counts", MEMORY_SIZES)
def test_matrix_memory_in_one_walk_and_in_pieces(dtype, nh, dim, vdim, counts):
    """Every cut of a head's columns that the kernel takes, with and without pieces, from states that earlier tokens left; gates
    that open wide, close, and forget fast."""
    ops = ops_module()
    g = torch.Generator().manual_seed(dim + vdim)
    n, lead = sum(counts), 3
    qk, vv = nh * dim, nh * vdim
    cols_of = [lead, lead + qk, lead + 2 * qk, lead + 2 * qk + vv, lead + 2 * qk + 2 * vv, lead + 2 * qk + 2 * vv + nh]
    width = cols_of[-1] + nh
    rows = torch.randn(2, n, width, generator=g)
    rows[:, :, cols_of[4]:] *= 4.0
    ib, fb = torch.randn(nh, generator=g), torch.randn(nh, generator=g) + 3.0
    nw = torch.randn(vv, generator=g)
    cap = 9.0
    s0, n0 = torch.randn(len(counts) + 1, nh, dim, vdim, generator=g), torch.randn(len(counts) + 1, nh, dim, generator=g)
    m0 = torch.randn(len(counts) + 1, nh, generator=g)
    slots = list(range(len(counts) - 1, -1, -1))
    sl, cu, _, _, _ = layout(counts, [0] * len(counts), slots)
    x = rows.double().sum(0)
    part = lambda i, w_: x[:, cols_of[i]:cols_of[i] + w_]
    q, k, v = part(0, qk).reshape(n, nh, dim) * dim ** -0.5, part(1, qk).reshape(n, nh, dim), part(2, vv).reshape(n, nh, vdim)
    i = cap * torch.tanh((part(4, nh) + ib) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((part(5, nh) + fb) / cap))
    refs, o = [], 0
    for b, c in enumerate(counts):
        st = tuple(t[slots[b]].double() for t in (s0, n0, m0))
        y, last = MP.matrix_memory(q[o:o + c], k[o:o + c], v[o:o + c], i[o:o + c], f[o:o + c], st)
        y = MP.unit_rms(y, 1e-5).reshape(c, vv) * nw.double() * torch.sigmoid(part(3, vv)[o:o + c])
        refs.append((y, last))
        o += c
    lib_cols = sorted({vdim} | {c for c in (64, 32, 8) if c < vdim} | {ops.matrix_memory_plan(dim, vdim, nh, len(counts), max(counts))[2]})
    fits = ops._lib("matrix_memory").llg_matrix_memory_fits
    for cols in [c for c in lib_cols if fits(dim, c)]:
        for piece in (0, 128, 64, 20):
            pieces = piece > 0
            S, N, M = s0.clone().cuda(), n0.clone().cuda(), m0.clone().cuda()
            out = torch.empty(n, vv, dtype=dtype, device="cuda")
            carry = torch.empty(len(counts), -(-max(counts) // piece), nh, dim * vdim + dim + 3, device="cuda") if pieces else None
            raw = torch.empty(n, vv, device="cuda") if cols < vdim else None
            nxt = torch.empty(len(counts), nh, dim + 1, device="cuda") if cols < vdim and not pieces else None
            ops.matrix_memory(rows.cuda(), q_col=cols_of[0], k_col=cols_of[1], v_col=cols_of[2], g_col=cols_of[3], i_col=cols_of[4],
                              f_col=cols_of[5], n_heads=nh, dim=dim, vdim=vdim, i_bias=ib.cuda(), f_bias=fb.cuda(), gate_cap=cap,
                              q_scale=dim ** -0.5, denom_eps=1e-6, eps=1e-5, norm_w=nw.cuda(), state_s=S, state_n=N, state_m=M,
                              slots=sl, cu_tokens=cu, out=out, cols=cols, carry=carry, piece=piece, raw=raw, next_nm=nxt)
            o = 0
            for b, c in enumerate(counts):
                y, (s, nn, m) = refs[b]
                what = (cols, piece, b)
                near(out[o:o + c], y, 2e-4 if dtype == torch.float32 else 2e-2, ("memory", *what))
                near(S[slots[b]], s, 1e-4, ("S", *what))
                near(N[slots[b]], nn, 1e-4, ("n", *what))
                near(M[slots[b]], m, 1e-5, ("m", *what))
                o += c
            assert torch.equal(S[len(counts)].cpu(), s0[len(counts)]) and torch.equal(M[len(counts)].cpu(), m0[len(counts)])


def _paged(k, v, lens, ring, gen, dtype):
    """Pages (with what an earlier owner left in them) that hold the first ``lens[b]`` keys and values of every sequence, in a
    shuffled order; slots are shuffled too.  Returns (k_pages, v_pages, page_table, slots)."""
    b_n, nkv, hd, vd = len(lens), k[0].shape[1], k[0].shape[2], v[0].shape[2]
    n_pages = b_n * ring + 3
    kp = torch.randn(n_pages, nkv, 64, hd, generator=gen).to(dtype)
    vp = torch.randn(n_pages, nkv, 64, vd, generator=gen).to(dtype)
    order = torch.randperm(n_pages, generator=gen).tolist()
    slots = torch.randperm(b_n, generator=gen).tolist()
    table = torch.zeros(b_n, ring, dtype=torch.int32)
    for b in range(b_n):
        for j in range(ring):
            table[slots[b], j] = order.pop()
        for p in range(lens[b]):
            page = int(table[slots[b], p // 64])
            kp[page, :, p % 64] = k[b][p].to(dtype)
            vp[page, :, p % 64] = v[b][p].to(dtype)
    return kp.cuda(), vp.cuda(), table.cuda(), slots


def _mixed_attention(q, k, v, scale, cap, talk, sink, gate, first):
    """q: [T, H, d] at the last T of the S positions of k, v [S, G, .]; ``first(p)``: the first position a query at p sees."""
    t, s_n, rep = q.shape[0], k.shape[0], q.shape[1] // k.shape[1]
    kk, vv = k.double().repeat_interleave(rep, dim=1), v.double().repeat_interleave(rep, dim=1)
    s = MP.mixed_scores(torch.einsum("thd,shd->hts", q.double(), kk) * scale, cap, talk)
    pos = torch.arange(s_n - t, s_n)
    j = torch.arange(s_n)
    hidden = (j[None, :] > pos[:, None]) | (j[None, :] < torch.tensor([first(int(p)) for p in pos])[:, None])
    return (torch.einsum("hts,shd->thd", MP.sink_softmax(s, hidden, sink), vv) * gate.double()[:, :, None]).reshape(t, -1)


MIX_SIZES = [(4, 2, 16, 24, 5.0), (6, 1, 128, 128, 50.0), (8, 2, 64, 32, 30.0), (5, 5, 32, 80, 10.0), (3, 1, 10, 6, 0.0), (1, 1, 12, 20, 2.0),
             (16, 4, 128, 64, 20.0), (24, 8, 64, 64, 15.0), (7, 7, 48, 16, 8.0), (32, 8, 32, 32, 25.0), (12, 4, 16, 48, 3.0),
             (32, 8, 128, 128, 50.0), (40, 8, 128, 64, 50.0), (16, 16, 128, 128, 9.0), (48, 2, 16, 16, 5.0), (2, 1, 64, 112, 4.0)]


@pytest.mark.parametrize("dtype,tensor_cores", [(torch.float32, False), (torch.bfloat16, True), (torch.bfloat16, False)],
                         ids=["f32", "bf16", "bf16-cuda-cores"])
@pytest.mark.parametrize("window,chunked", [(0, False), (70, False), (50, True)])
@pytest.mark.parametrize("nh,nkv,hd,vd,cap", MIX_SIZES)
def test_attention_with_capped_and_mixed_scores(monkeypatch, dtype, tensor_cores, nh, nkv, hd, vd, cap, window, chunked):
    """A prompt step (old keys in shuffled pages, new ones packed) and a decode step of unequal sequences; sinks, gates and the
    masks beside the mixture; one key far back stands out for one query's head, so that a mixture that lost it would show."""
    ops = ops_module()
    monkeypatch.setattr(ops, "USE_MIX_MMA", tensor_cores)
    gen = torch.Generator().manual_seed(nh * hd + window)
    talk = torch.eye(nh) + 0.5 * torch.randn(nh, nh, generator=gen)
    sinks = torch.randn(nh, generator=gen)
    scale = 1.3 * hd ** -0.5
    first = (lambda p: 0) if not window else (lambda p: p // window * window) if chunked else (lambda p: max(0, p - window + 1))
    tol = 3e-5 if dtype == torch.float32 else 1.5e-2
    form = ops.AttentionForm(value_dim=vd, sinks=sinks.cuda(), gated=True, chunked=chunked, softcap=cap, head_mix=talk.cuda())
    before, counts = [0, 130, 5, 64], [33, 1, 70, 100]
    total = [b + c for b, c in zip(before, counts)]
    ring = 4
    for decode in (False, True):
        if decode:
            before, counts = [t - 1 for t in (1, 129, 200, 64, 65)], [1] * 5
            total = [b + 1 for b in before]
        k = [torch.randn(t, nkv, hd, generator=gen).to(dtype) for t in total]
        v = [torch.randn(t, nkv, vd, generator=gen).to(dtype) for t in total]
        q = [torch.randn(c, nh, hd, generator=gen).to(dtype) for c in counts]
        far = 2 if decode else 3                                    # its last query and a key of 60 (or 40) positions earlier
        back = total[far] - 1 - (40 if window else 60)
        k[far][back, 0] = (3.0 * q[far][-1, 0].float()).to(dtype)
        gate = torch.rand(sum(counts), nh, generator=gen)
        kp, vp, table, slots = _paged(k, v, total if decode else before, ring, gen, dtype)
        sl, cu, _, lb, _ = layout(counts, before, slots)
        out = torch.empty(sum(counts), nh * vd, dtype=dtype, device="cuda")
        qd = torch.cat(q).cuda()
        if decode:
            for max_len in (max(total), 1024):
                plan = ops.attn_decode_plan(dtype, len(counts), nh, nkv, hd, max_len, form)
                scratch = torch.empty(max(1, plan.scratch_floats), device="cuda")
                counters = torch.zeros(plan.n_counters, dtype=torch.int32, device="cuda") if plan.n_counters else None
                for _ in range(2):
                    out.zero_()
                    ops.attn_decode(qd, kp, vp, table, ring, sl, lb, out, scratch, scale=scale, window=window, plan=plan, counters=counters,
                                    form=form, gate=gate.cuda())
        else:
            tq = ops.prefill_tile_queries(dtype, hd, form)
            tiles = [(b, q0) for b, c in enumerate(counts) for q0 in range(0, c, tq)]
            tiles = torch.tensor(tiles, dtype=torch.int32, device="cuda")
            k_new = torch.cat([x[b:] for x, b in zip(k, before)]).contiguous().cuda()
            v_new = torch.cat([x[b:] for x, b in zip(v, before)]).contiguous().cuda()
            ops.attn_prefill(qd, k_new, v_new, kp, vp, table, ring, tiles, cu, lb, sl, out, scale=scale, window=window, tile_queries=tq,
                             form=form, gate=gate.cuda())
        o = 0
        for b, c in enumerate(counts):
            want = _mixed_attention(q[b], k[b], v[b], scale, cap, talk, sinks, gate[o:o + c], first)
            near(out[o:o + c], want, tol, ("decode" if decode else "prompt", b))
            o += c


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_capped_or_mixed_scores_alone(dtype):
    """The cap without a mixture and the mixture without a cap, without sinks and gates."""
    ops = ops_module()
    gen = torch.Generator().manual_seed(3)
    nh, nkv, hd, vd, t = 4, 2, 32, 32, 90
    q, k, v = (torch.randn(t, h, d, generator=gen).to(dtype) for h, d in ((nh, hd), (nkv, hd), (nkv, vd)))
    talk = torch.eye(nh) + 0.5 * torch.randn(nh, nh, generator=gen)
    kp, vp, table, slots = _paged([k], [v], [0], 2, gen, dtype)
    sl, cu, _, lb, _ = layout([t], [0], slots)
    for cap, mix in ((2.0, None), (0.0, talk)):
        form = ops.AttentionForm(softcap=cap, head_mix=None if mix is None else mix.cuda())
        tq = ops.prefill_tile_queries(dtype, hd, form)
        tiles = torch.tensor([(0, q0) for q0 in range(0, t, tq)], dtype=torch.int32, device="cuda")
        out = torch.empty(t, nh * vd, dtype=dtype, device="cuda")
        ops.attn_prefill(q.cuda(), k.cuda(), v.cuda(), kp, vp, table, 2, tiles, cu, lb, sl, out, scale=0.4, window=0, tile_queries=tq, form=form)
        near(out, _mixed_attention(q, k, v, 0.4, cap, mix, None, torch.ones(t, nh), lambda p: 0), 3e-5 if dtype == torch.float32 else 1.5e-2, cap)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_preparations_leave_the_heads_gates(dtype):
    """``qk_prep`` (neighbours rotated over a part of the head, values of another size) and ``latent_prep`` with gates."""
    ops = ops_module()
    gen = torch.Generator().manual_seed(8)
    nh, nkv, hd, vd, n, rd = 6, 2, 24, 40, 11, 10
    width = (nh + nkv) * hd + nkv * vd + nh
    rows = torch.randn(3, n, width, generator=gen)
    x = rows.double().sum(0)
    pos = torch.tensor([0, 1, 2, 70, 71, 72, 73, 5, 6, 900, 901])
    rot = {"base": 90.0, "dims": rd}
    ang = torch.arange(1000, dtype=F64)[:, None] * (90.0 ** (-2.0 * torch.arange(rd // 2, dtype=F64) / rd))[None, :]
    q, gate = torch.empty(n, nh, hd, dtype=dtype, device="cuda"), torch.empty(n, nh, device="cuda")
    k, v = torch.empty(n, nkv, hd, dtype=dtype, device="cuda"), torch.empty(n, nkv, vd, dtype=dtype, device="cuda")
    ops.qk_prep(rows.cuda(), n_heads=nh, n_kv_heads=nkv, head_dim=hd, q_norm_w=None, k_norm_w=None, norm_eps=1e-6, bias=None,
                cos=torch.cos(ang).float().cuda(), sin=torch.sin(ang).float().cuda(), rotary_dim=rd, pairing=1,
                positions=pos.int().cuda(), q_out=q, k_new=k, v_new=v, value_dim=vd, gate_out=gate)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    near(q, MP.rotate_neighbours(x[:, :nh * hd].reshape(n, nh, hd), pos, rot), tol, "q")
    near(k, MP.rotate_neighbours(x[:, nh * hd:(nh + nkv) * hd].reshape(n, nkv, hd), pos, rot), tol, "k")
    near(v, x[:, (nh + nkv) * hd:-nh].reshape(n, nkv, vd), tol, "v")
    near(gate, torch.sigmoid(x[:, -nh:]), 1e-5, "gate")
    dim, rank = 16, 40
    rows = torch.randn(2, n, nh * dim + rank + nh + 2, generator=gen)
    x = rows.double().sum(0)
    qp, qo = torch.empty(n, nh, dim, dtype=dtype, device="cuda"), torch.empty(n, nh, rank, dtype=dtype, device="cuda")
    c, nw = torch.empty(n, 1, rank, dtype=dtype, device="cuda"), torch.randn(rank, generator=gen)
    ops.latent_prep(rows.cuda(), n_heads=nh, head_dim=dim, rot_dim=0, kv_rank=rank, c_norm_w=nw.cuda(), norm_eps=1e-5, cos=None, sin=None,
                    positions=pos.int().cuda(), q_plain_out=qp, q_out=qo, k_new=c, gate_col=nh * dim + rank + 1, gate_out=gate)
    near(qp, x[:, :nh * dim].reshape(n, nh, dim), tol, "q")
    near(c[:, 0], MP.unit_rms(x[:, nh * dim:nh * dim + rank], 1e-5) * nw.double(), tol, "latent")
    near(gate, torch.sigmoid(x[:, nh * dim + rank + 1:-1]), 1e-5, "gate")


# ---- whole models ------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", list(MM.CONFIGS))
def test_whole_prompt_and_first_tokens(engines, models, name, dtype):
    eng = engines(name, dtype)
    for n in (1, 2, 3, 190):
        toks, ref = sequence(models, name, dtype, n, n)
        slot = eng.open()
        lg = eng.step([(slot, toks)], [list(range(n))])
        close(lg, ref, dtype, (name, "whole", n))
        eng.close(slot)
    eng.cache.audit()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_residual_after_every_layer(llogos, models, dtype):
    """The residual after each layer that runs (a looped layer counts each time), read from the engine by models whose run
    order is cut short, is what the plain model's trace holds."""
    import os
    name = "mixed"
    d, cfg, w = models[name, dtype]
    toks, _ = sequence(models, name, dtype, 50, 4)
    trace = []
    MP.forward(w, cfg, toks, trace)
    order = MP.run_order(cfg)
    assert len(trace) == len(order) == 11
    start, stop = cfg["loop"]["start"], cfg["loop"]["stop"]
    for depth in range(1, len(order) + 1):
        if depth <= stop:                              # the loop's first round: the layers by themselves
            cut = {k: v for k, v in cfg.items() if k != "loop"}
            cut["layers"] = cfg["layers"][:depth]
        elif depth == len(order):
            cut = cfg
        elif (depth - start) % (stop - start) == 0:    # whole rounds
            cut = dict(cfg, layers=cfg["layers"][:stop], loop=dict(cfg["loop"], times=(depth - start) // (stop - start)))
        else:
            continue
        keep = {k: v for k, v in w.items() if not (k.startswith("l") and k[1].isdigit() and int(k[1:k.index(".")]) >= len(cut["layers"]))}
        sub = os.path.join(d, f"cut{depth}")
        MM.write_model(llogos, sub, cut, 0, weights={k: v.to(torch.bfloat16) for k, v in keep.items()})
        model = llogos.weights.load_model(sub, dtype=dtype, device="cuda:0")
        eng = llogos.engine.Engine(model, max_tokens=256)
        slot = eng.open()
        lg = eng.step([(slot, toks)], [list(range(len(toks)))])
        close(lg, MP.linear(MP.layer_norm(trace[depth - 1], w["final.norm"], cfg["norm"]["eps"]), w["embed"]), dtype, ("after", depth))
        eng.close(slot)


@pytest.mark.parametrize("graphs", [True, False], ids=["graph", "eager"])
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", list(MM.CONFIGS))
def test_prompt_then_token_by_token(engines, models, name, dtype, graphs):
    """The decoded positions pass page borders (128, 192) and the border of the memory's pieces; the first token alone too."""
    eng = engines(name, dtype, graphs)
    toks, ref = sequence(models, name, dtype, 215, 7)
    for cut in (1, 120):
        slot = eng.open()
        lg = eng.step([(slot, toks[:cut])])
        close(lg, ref[cut - 1:cut], dtype, (name, "prompt end", cut))
        got = [eng.step([(slot, [toks[p]])]).clone() for p in range(cut, len(toks) if cut > 1 else 40)]
        close(torch.cat(got), ref[cut:cut + len(got)], dtype, (name, "decoded from", cut))
        eng.close(slot)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", list(MM.CONFIGS))
def test_portions_of_several_sizes(engines, models, name, dtype):
    eng = engines(name, dtype)
    toks, ref = sequence(models, name, dtype, 300, 9)
    for sizes in ([2] * 20 + [3, 64, 65, 1, 1, 2, 124], [63, 1, 64, 2, 170], [129, 171]):
        assert sum(sizes) == len(toks)
        slot = eng.open()
        at, got = 0, []
        for s in sizes:
            got.append(eng.step([(slot, toks[at:at + s])], [list(range(s))]).clone())
            at += s
        close(torch.cat(got), ref, dtype, (name, "portions", sizes[:4]))
        eng.close(slot)
    eng.cache.audit()


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", list(MM.CONFIGS))
def test_unequal_batches_with_slots_pages_and_states_used_again(engines, models, name, dtype):
    eng = engines(name, dtype)
    pairs = [sequence(models, name, dtype, n, 20 + n) for n in (1, 66, 140, 259, 33)]
    seqs, refs = [p[0] for p in pairs], [p[1] for p in pairs]
    for order in ([0, 1, 2, 3], [4, 3, 0], [2, 1, 4, 3, 0]):
        slots = {i: eng.open() for i in order}
        cut = {i: max(1, len(seqs[i]) - 4 - 9 * j) for j, i in enumerate(order)}
        lg = eng.step([(slots[i], seqs[i][:cut[i]]) for i in order])
        for j, i in enumerate(order):
            close(lg[j], refs[i][cut[i] - 1], dtype, (name, "batched prompt", i))
        live = [i for i in order if cut[i] < len(seqs[i])]
        for i in set(order) - set(live):
            eng.close(slots[i])
        while live:
            lg = eng.step([(slots[i], [seqs[i][cut[i]]]) for i in live])
            for j, i in enumerate(live):
                close(lg[j], refs[i][cut[i]], dtype, (name, "batched decode", i, cut[i]))
                cut[i] += 1
            for i in [i for i in live if cut[i] == len(seqs[i])]:
                eng.close(slots[i])
            live = [i for i in live if cut[i] < len(seqs[i])]
        eng.cache.audit()
    assert eng.cache.slots.free_count == eng.cache.slots.n_slots


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_long_decoding(engines, models, dtype):
    """420 decoded tokens after a prompt of 30: the memories are carried through every step, the keys grow over seven pages."""
    name = "mixed"
    eng = engines(name, dtype)
    toks, ref = sequence(models, name, dtype, 450, 5)
    slot = eng.open()
    eng.step([(slot, toks[:30])], [[]])
    got = [eng.step([(slot, [toks[p]])]).clone() for p in range(30, len(toks))]
    close(torch.cat(got), ref[30:], dtype, ("long decoding",))
    eng.close(slot)


def _random_config(seed):
    """A configuration drawn from the seed: two to five layers of the three kinds in any order; sizes, caps, rotations, limits and
    the loop, all drawn."""
    g = torch.Generator().manual_seed(4000 + seed)
    pick = lambda xs: xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    width = pick([48, 64, 72, 96, 120])
    layers = []
    for _ in range(pick([2, 3, 4, 5])):
        mlp = None
        if pick([0, 1, 1, 1]):
            n_exp = pick([1, 2, 3, 6, 9])
            mlp = MM.moe(n_exp, pick(list(range(1, n_exp + 1))), pick([8, 24, 40]), pick([0.5, 1.0, 7.0]),
                         shared=pick([None, (16, 0.6), (56, 3.0)]))
        kind = pick([0, 1, 2])
        if kind == 0:
            mix = MM.mlstm(pick([1, 2, 3, 5]), pick([4, 10, 16, 40, 64]), pick([4, 12, 24, 48, 80]), pick([2.0, 15.0]))
        elif kind == 1:
            mix = MM.latent(pick([1, 2, 4, 5]), pick([8, 12, 32]), pick([8, 20, 32]), pick([16, 24, 48, 96, 160]), scale=pick([0.1, 0.3]))
        else:
            kv, dim = pick([1, 2, 3]), pick([8, 16, 24, 40, 64])
            mix = MM.attention(kv * pick([1, 2, 4]), kv, dim, pick([8, 16, 24, dim]), pick([None, 2, 4, dim]), base=pick([50.0, 10000.0, 3e6]),
                               scale=pick([0.05, 0.2, 0.5]), cap=pick([0.0, 1.0, 30.0]))
        layers.append(MM.layer(mix, mlp))
    n = len(layers)
    start = pick(list(range(n)))
    return MM.config(layers, vocab=pick([61, 128, 257]), width=width, eps=pick([1e-6, 1e-5, 1e-3]),
                     loop=pick([None, (start, pick(list(range(start + 1, n + 1))), pick([1, 2, 3]))]))


@pytest.mark.parametrize("seed", range(14))
def test_configurations_drawn_at_random(llogos, tmp_path, seed):
    """float32: a prompt whole, a batch of two unequal prompts decoded together for a dozen steps, against the plain model."""
    cfg = _random_config(seed)
    d = str(tmp_path / "m")
    w = {k: v.float() for k, v in MM.write_model(llogos, d, cfg, seed=seed).items()}
    model = llogos.weights.load_model(d, dtype=torch.float32, device="cuda:0")
    eng = llogos.engine.Engine(model, max_tokens=64 * 12)
    g = torch.Generator().manual_seed(seed)
    seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (171, 40)]
    refs = [MP.forward(w, cfg, s) for s in seqs]
    slot = eng.open()
    close(eng.step([(slot, seqs[0])], [list(range(len(seqs[0])))]), refs[0], torch.float32, ("random", seed, "whole"))
    eng.close(slot)
    slots = [eng.open(), eng.open()]
    cut = [len(s) - 12 for s in seqs]
    lg = eng.step([(sl, s[:c]) for sl, s, c in zip(slots, seqs, cut)])
    for i in range(2):
        close(lg[i], refs[i][cut[i] - 1], torch.float32, ("random", seed, "prompt", i))
    for k in range(12):
        lg = eng.step([(sl, [s[c + k]]) for sl, s, c in zip(slots, seqs, cut)])
        for i in range(2):
            close(lg[i], refs[i][cut[i] + k], torch.float32, ("random", seed, "decode", i, k))
    for sl in slots:
        eng.close(sl)
    eng.cache.audit()


def _random_tensor_config(seed):
    """As ``_random_config``, of sizes that the tensor-core kernels take."""
    g = torch.Generator().manual_seed(5000 + seed)
    pick = lambda xs: xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    layers = []
    for kind in torch.randperm(3, generator=g).tolist():
        n_exp = pick([2, 4, 8])
        mlp = MM.moe(n_exp, pick([1, 2]), pick([32, 72, 136]), pick([0.8, 3.0]), shared=pick([None, (64, 0.9)]))
        if kind == 0:
            mix = MM.mlstm(pick([2, 4, 6]), pick([32, 48, 96]), pick([32, 80, 128]), pick([6.0, 15.0]))
        elif kind == 1:
            mix = MM.latent(pick([2, 4, 6, 9]), pick([16, 32, 48]), pick([16, 32, 64]), pick([32, 64, 96, 128, 192]))
        else:
            kv, dim = pick([1, 2, 4, 5]), pick([16, 48, 80, 112, 128])
            mix = MM.attention(kv * pick([1, 2, 3, 4, 5]), kv, dim, pick([16, 32, 96, 128]), pick([None, 8, dim]), base=pick([500.0, 1e6]),
                               cap=pick([0.0, 15.0, 50.0]))
        layers.append(MM.layer(mix, mlp))
    return MM.config(layers, vocab=pick([160, 257]), width=pick([64, 128, 200]), loop=pick([None, (0, 2, 2), (1, 3, 2)]))


@pytest.mark.parametrize("seed", range(8))
def test_tensor_core_configurations_drawn_at_random(llogos, tmp_path, seed):
    """bfloat16: a prompt whole, and a batch of two unequal prompts decoded together, against the plain model."""
    cfg = _random_tensor_config(seed)
    d = str(tmp_path / "m")
    w = {k: v.float() for k, v in MM.write_model(llogos, d, cfg, seed=seed, steady_routing=True).items()}
    model = llogos.weights.load_model(d, dtype=torch.bfloat16, device="cuda:0")
    eng = llogos.engine.Engine(model, max_tokens=64 * 12)
    key = {("random", torch.bfloat16): (d, cfg, w)}
    for store in (_tokens, _refs, _pools):
        for k in [k for k in store if k[0] == "random"]:
            del store[k]
    pairs = [sequence(key, "random", torch.bfloat16, n, n) for n in (230, 45)]
    (a, ra), (b, rb) = pairs
    slot = eng.open()
    close(eng.step([(slot, a)], [list(range(len(a)))]), ra, torch.bfloat16, ("random", seed, "whole"))
    eng.close(slot)
    slots = [eng.open(), eng.open()]
    cut = [len(a) - 14, len(b) - 14]
    lg = eng.step([(slots[0], a[:cut[0]]), (slots[1], b[:cut[1]])])
    close(lg[0], ra[cut[0] - 1], torch.bfloat16, ("random", seed, "prompt"))
    got = [eng.step([(slots[0], [a[cut[0] + k]]), (slots[1], [b[cut[1] + k]])]).clone() for k in range(14)]
    close(torch.stack([g[0] for g in got]), ra[cut[0]:], torch.bfloat16, ("random", seed, "decoded, long"))
    close(torch.stack([g[1] for g in got]), rb[cut[1]:], torch.bfloat16, ("random", seed, "decoded, short"))


# ---- faults that random weights would hide ---------------------------------------------------------

A_TOK, B_TOK = 11, 12


def _far_model(llogos, folder, kind):
    """One layer without a feed-forward, made so that only token a writes under a direction z that token b asks with (every
    other token's normed embedding is orthogonal to z).  "latent": a key among hundreds in the latent's head 0.  "attention":
    head 0 finds a, and head 3 (whose own query and key are silent) gets that score through the mixture alone; heads 0 to 2
    write nothing to the output.  "mlstm": head 0's memory, whose gates do not forget, holds a's value under z."""
    d = 48
    mixer = {"latent": MM.latent(2, 32, 24, 40, scale=0.5), "attention": MM.attention(4, 2, 32, 24, 4, scale=0.5, cap=30.0),
             "mlstm": MM.mlstm(2, 32, 24, cap=15.0)}[kind]
    cfg = MM.config([MM.layer(mixer, None)], vocab=50, width=d)
    w = MM.random_weights(cfg, 77)
    gen = torch.Generator().manual_seed(1)

    def centred(t):
        return t - t.mean()
    z = centred(torch.randn(d, generator=gen))
    z = z / z.norm()
    emb = w["embed"].float()
    emb -= emb.mean(-1, keepdim=True)
    emb -= (emb @ z)[:, None] * z[None, :]
    r = [centred(torch.randn(d, generator=gen)) for _ in range(2)]
    r = [x - (x @ z) * z for x in r]
    for tok, x in zip((A_TOK, B_TOK), r):
        emb[tok] = 5.0 * z + 5.0 * x / x.norm()
    w["embed"] = emb.to(torch.bfloat16)
    w["l0.norm1"][:] = 1.0
    w["l0.ls1"][:] = 4.0                                                   # what the layer finds weighs on the logits
    e = torch.zeros(32)
    e[4:] = 28 ** -0.5                                                     # outside the rotated elements
    p = "l0.mix."
    row = (1.3 * e[:, None] * z[None, :]).to(torch.bfloat16)
    if kind == "latent":
        w[p + "q"][:32] = row
        w[p + "dkv"][0] = (1.5 * z).to(torch.bfloat16)                     # the latent's first element says "a (or b)"
        w[p + "dkv.norm"][:] = 1.0
        w[p + "uk"][:32] = 0.0
        w[p + "uk"][:32, 0] = (1.3 * e).to(torch.bfloat16)
        w[p + "g"][:] = 0.0
    elif kind == "attention":
        w[p + "q"][:] = 0.0
        w[p + "k"][:] = 0.0
        w[p + "q"][:32] = row
        w[p + "k"][:32] = row
        w[p + "talk"] = torch.zeros(4, 4, dtype=torch.bfloat16)
        w[p + "talk"][3, 0] = 1.0
        w[p + "sink"][:] = 0.0
        w[p + "o"][:, :72] = 0.0
        w[p + "g"][:] = 0.0
    else:
        w[p + "q"][:32] = row
        w[p + "k"][:32] = row
        w[p + "i"][:] = 0.0
        w[p + "f"][:] = 0.0
        w[p + "i.b"][:] = 0.0
        w[p + "f.b"][:] = 12.0
        w[p + "v"][24:] = 0.0                                              # the second head stays silent
    MM.write_model(llogos, folder, cfg, 0, weights=w)
    return cfg, {k: v.float() for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("kind", ["latent", "attention", "mlstm"])
def test_what_token_a_left_330_positions_back(llogos, tmp_path, dtype, kind):
    """Token a stands at position 2, token b 330 positions (five pages, three pieces of the memory's walk) later.  b's logits
    with a there and with another token in a's place are far apart, in a prompt, in portions, decoded, and beside another
    request."""
    d = str(tmp_path / kind)
    cfg, wf = _far_model(llogos, d, kind)
    model = llogos.weights.load_model(d, dtype=dtype, device="cuda:0")
    eng = llogos.engine.Engine(model, max_tokens=64 * 16)
    gen = torch.Generator().manual_seed(3)
    toks = torch.randint(13, 50, (336,), generator=gen).tolist()
    b_at = 332
    toks[b_at] = B_TOK
    with_a, without_a = list(toks), list(toks)
    with_a[2] = A_TOK
    refs = [MP.forward(wf, cfg, t) for t in (with_a, without_a)]
    assert float((refs[0][b_at] - refs[1][b_at]).abs().max()) > 0.05 * float(refs[0][b_at].abs().max())
    for t, ref in zip((with_a, without_a), refs):
        for cut in (len(t), b_at, 3):
            slot = eng.open()
            lg = eng.step([(slot, t[:cut])], [[b_at] if b_at < cut else []])
            for p in range(cut, b_at + 1):
                lg = eng.step([(slot, [t[p]])])
            close(lg, ref[b_at:b_at + 1], dtype, (kind, "a far back", cut), tol=TIGHT)
            eng.close(slot)
        slot = eng.open()
        for lo, hi in ((0, 2), (2, 4), (4, 70), (70, 199), (199, 330)):
            eng.step([(slot, t[lo:hi])], [[]])
        close(eng.step([(slot, t[330:])], [[b_at - 330]]), ref[b_at:b_at + 1], dtype, (kind, "a far back, portions"), tol=TIGHT)
        eng.close(slot)
    slots = [eng.open(), eng.open()]
    eng.step([(slots[0], with_a[:200]), (slots[1], without_a[:90])], [[], []])
    eng.step([(slots[1], without_a[90:200])], [[]])
    for p in range(200, b_at):
        eng.step([(slots[0], [with_a[p]]), (slots[1], [without_a[p]])], [[], []])
    lg = eng.step([(slots[0], [with_a[b_at]]), (slots[1], [without_a[b_at]])])
    close(lg[0], refs[0][b_at], dtype, (kind, "batched, with a"), tol=TIGHT)
    close(lg[1], refs[1][b_at], dtype, (kind, "batched, without a"), tol=TIGHT)


# ---- the library's entry points ----------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_greedy_generation_through_the_entry_point(models, dtype):
    """``LlogosModel.generate`` (scheduler, sampler, run-ahead decoding) makes the plain model's best tokens."""
    import llogos_b200 as L
    name = "mixed"
    d, cfg, w = models[name, dtype]
    model = L.LlogosModel.load(d, dtype=dtype, max_context=256, max_batch=3)
    prompts = [sequence(models, name, dtype, n, 60 + n)[0] for n in (5, 70, 23, 1)]
    out = model.generate(prompts, L.GenerationParams.greedy_params(12, stop_tokens=()))
    for p, made in zip(prompts, out.tokens):
        assert len(made) == 12
        toks = list(p)
        for tok in made:
            lg = MP.forward(w, cfg, toks)[-1]
            slack = 1e-4 if dtype == torch.float32 else 0.05
            assert float(lg[tok]) >= float(lg.max()) - slack * float(lg.abs().max()), (len(toks), tok)
            toks.append(tok)


def test_command_line_and_trace_replay_take_the_design(models, tmp_path):
    """``python -m llogos_b200`` generates with a Memilorn folder, and ``bin/trace_run`` replays steps on it (two requests
    started together, decoded together, the shorter one ending first, a third in portions), as they do for every model."""
    import json
    import os
    import subprocess
    import sys
    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    d, cfg, w = models["tensor", torch.float32]
    env = dict(os.environ, PYTHONPATH=root)
    base = [sys.executable, "-m", "llogos_b200", "--model", d, "--dtype", "float32"]
    p = subprocess.run(base + ["--prompt-ids", "5,17,3", "-n", "6", "-t", "0", "--repeat-penalty", "1.0", "--max-context", "128"],
                       capture_output=True, text=True, env=env, cwd=root)
    assert p.returncode == 0, p.stderr
    made = [int(x) for x in p.stdout.split()]
    toks = [5, 17, 3]
    for tok in made:
        lg = MP.forward(w, cfg, toks)[-1]
        assert float(lg[tok]) >= float(lg.max()) - 1e-4 * float(lg.abs().max())
        toks.append(tok)
    d, cfg, w = models["tensor", torch.bfloat16]
    (a, ra), (b, rb) = sequence(models, "tensor", torch.bfloat16, 100, 1), sequence(models, "tensor", torch.bfloat16, 31, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:98], "want": [0, 69, 97]}, {"id": "b", "tokens": b[:30], "want": [29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[98:99], "want": [0]}, {"id": "b", "tokens": b[30:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[99:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b[:7], "want": []}], "end": []},
             {"step": 4, "entries": [{"id": "c", "tokens": b[7:30], "want": [22]}], "end": ["c"]}]
    out = tmp_path / "logits"
    p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "bfloat16", "--out", str(out), "--max-tokens", "200"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, env=env, cwd=root)
    assert p.returncode == 0, p.stderr
    assert [l for l in p.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(5)]
    want = {0: torch.stack([ra[0], ra[69], ra[97], rb[29]]), 1: torch.stack([ra[98], rb[30]]), 2: ra[99:100], 4: rb[29:30]}
    assert not (out / "3.f32").exists()
    for i, ref in want.items():
        got = torch.from_numpy(np.fromfile(str(out / f"{i}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]))
        close(got, ref, torch.bfloat16, ("replayed step", i))
