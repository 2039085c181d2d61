"""The Penasun decoder on the GPU against the plain implementation in penasun_plain.py, in float32 and bfloat16: every
mechanism's kernel alone; whole prompts; prompts against token-by-token decoding; prompts in portions down to two tokens;
batches of unequal requests against each alone, with slots, pages and state rows used again; a far key that only one map
of a head finds; what a state took up long ago; the first tokens; long decoding; sizes that differ from layer to layer;
greedy generation through the library's entry point."""

import pytest
import torch

import penasun_models as PM
import penasun_plain as PP

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
MARGIN = 0.01          # bfloat16: no router of a compared sequence decides by less than this (in choice scores)


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
    for i, (name, cfg) in enumerate(PM.CONFIGS.items()):
        for dtype in DTYPES:
            d = str(tmp_path_factory.mktemp(f"penasun_{name}_{IDS[DTYPES.index(dtype)]}"))
            w = PM.write_model(llogos, d, cfg, seed=470 + i, steady_routing=dtype == torch.bfloat16)
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
        ref = PP.forward(w, cfg, toks, margins=margins)
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


def part_context(ops, dtype):
    """What a feed-forward part needs of a step's context."""
    from importlib import import_module
    ws = import_module("daisi-llogos_b200.engine.context").Workspace(torch.device("cuda"))

    class Ctx:
        pass
    ctx = Ctx()
    ctx.ops, ctx.dtype = ops, dtype
    ctx.buffer = lambda name, shape, dt=None, zero=False: ws.get(name, tuple(shape), dt or dtype, zero)
    return ctx


# ---- mechanisms alone --------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("n", [9, 70])
@pytest.mark.parametrize("hidden", [50, 72, 1024, 4096])
def test_norm_adds_a_branch_with_a_bias(dtype, n, hidden):
    """Every form of the kernel: scalar, rows in registers, slices of a row as blocks of their own (the division left out)."""
    ops = ops_module()
    g = torch.Generator().manual_seed(hidden + n)
    res, branch = torch.randn(n, hidden, generator=g), torch.randn(3, n, hidden, generator=g)
    bias, w = torch.randn(hidden, generator=g), torch.randn(hidden, generator=g)
    want = res.double() + branch.double().sum(0) + bias.double()
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    for rows in (None, [7, 0, 3]):
        idx = slice(None) if rows is None else rows
        m = n if rows is None else len(rows)
        dev_rows = None if rows is None else torch.tensor(rows, dtype=torch.int32, device="cuda")
        dev, out = res.clone().cuda(), torch.empty(m, hidden, dtype=dtype, device="cuda")
        ops.add_rmsnorm(dev, branch.cuda(), w.cuda(), 1e-5, out, dev_rows, branch_bias=bias.cuda())
        near(dev[idx], want[idx], 1e-5, "sum")
        near(out, PP.rms_norm(want[idx], w, 1e-5), tol, "norm")
        dev, ss = res.clone().cuda(), torch.empty(m, ops.norm_ss_parts(m, hidden), device="cuda")
        ops.add_rmsnorm(dev, branch.cuda(), w.cuda(), 1e-5, out, dev_rows, ss_out=ss, branch_bias=bias.cuda())
        near(out, want[idx] * w.double(), tol, "unscaled")
        near(ss.sum(1), (want[idx] ** 2).sum(-1), 1e-5, "sums of squares")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("nh,nkv,hd,vd", [(4, 2, 64, 64), (3, 1, 128, 128), (4, 4, 24, 20), (2, 1, 10, 6), (3, 3, 128, 64)])
def test_preparation_with_query_factors_and_split_maps(dtype, nh, nkv, hd, vd):
    ops = ops_module()
    g = torch.Generator().manual_seed(nh * hd)
    counts, before, slots = (5, 1, 70), (0, 130, 60), (2, 0, 1)
    n = sum(counts)
    sl, cu, seq, lb, pos = layout(counts, before, slots)
    width = (nh + nkv) * hd + nkv * vd
    rows, bias = torch.randn(2, n, width, generator=g), torch.randn(width, generator=g)
    factor = 1.0 + torch.rand(200, generator=g)
    x = rows.double().sum(0) + bias.double()
    q = x[:, :nh * hd].view(n, nh, hd) * factor.double()[pos.cpu().long()][:, None, None]
    k, v = x[:, nh * hd:(nh + nkv) * hd].view(n, nkv, hd), x[:, (nh + nkv) * hd:].view(n, nkv, vd)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    ring = 4
    table = torch.randperm(3 * ring, generator=g).to(torch.int32).view(3, ring).cuda()
    for maps in (0, 2):
        q_out = torch.empty(n, nh * (maps or 1), hd, dtype=dtype, device="cuda")
        kn, vn = torch.empty(n, nkv, hd, dtype=dtype, device="cuda"), torch.empty(n, nkv, vd, dtype=dtype, device="cuda")
        kp, vp = torch.zeros(12, nkv, 64, hd, dtype=dtype, device="cuda"), torch.zeros(12, nkv, 64, vd, dtype=dtype, device="cuda")
        ops.qk_prep(rows.cuda(), n_heads=nh, n_kv_heads=nkv, head_dim=hd, q_norm_w=None, k_norm_w=None, norm_eps=1e-6, bias=bias.cuda(),
                    cos=None, sin=None, rotary_dim=0, pairing=0, positions=pos, q_out=q_out, k_new=kn, v_new=vn, k_pages=kp, v_pages=vp,
                    page_table=table, ring_pages=ring, seq_of_token=seq, slots=sl, value_dim=vd, q_scale=factor.cuda(), q_maps=maps)
        if maps:
            want = torch.zeros(n, nh, 2, hd, dtype=F64)
            want[:, :, 0, :hd // 2], want[:, :, 1, hd // 2:] = q[..., :hd // 2], q[..., hd // 2:]
            near(q_out, want.view(n, nh * 2, hd), tol, "queries, a map each")
        else:
            near(q_out, q, tol, "queries")
        near(kn, k, tol, "keys")
        near(vn, v, tol, "values")
        for t in (0, 5, n - 1):
            page = int(table[slots[int(seq[t])], int(pos[t]) // 64])
            near(kp[page, :, int(pos[t]) % 64], k[t], tol, ("page", t))
            near(vp[page, :, int(pos[t]) % 64], v[t], tol, ("value page", t))


@pytest.mark.parametrize("nh,nkv,hd", [(4, 2, 64), (2, 1, 128)])
def test_projection_with_the_preparation_as_its_epilogue(nh, nkv, hd):
    """Biases and query factors in the fused q/k/v product of a large prompt step."""
    ops = ops_module()
    g = torch.Generator().manual_seed(hd)
    n, k = 400, 96
    x, w = torch.randn(n, k, generator=g).to(torch.bfloat16), (torch.randn((nh + 2 * nkv) * hd, k, generator=g) * k ** -0.5).to(torch.bfloat16)
    bias, factor = torch.randn((nh + 2 * nkv) * hd, generator=g).to(torch.bfloat16), 1.0 + torch.rand(500, generator=g)
    pos = torch.arange(37, 37 + n, dtype=torch.int32, device="cuda")
    out = [torch.empty(n, h, hd, dtype=torch.bfloat16, device="cuda") for h in (nh, nkv, nkv)]
    assert ops.gemm_tc_qkv_supported(x.cuda(), w.cuda(), hd, 0, 0)
    ops.gemm_tc_qkv(x.cuda(), w.cuda(), n_heads=nh, n_kv_heads=nkv, head_dim=hd, q_norm_w=None, k_norm_w=None, norm_eps=1e-6, bias=bias.cuda(),
                    cos=None, sin=None, rotary_dim=0, pairing=0, positions=pos, q_out=out[0], k_new=out[1], v_new=out[2], q_scale=factor.cuda())
    y = PP.linear(x, w, bias).view(n, nh + 2 * nkv, hd)
    near(out[0], y[:, :nh] * factor.double()[pos.cpu().long()][:, None, None], 1e-2, "queries")
    near(out[1], y[:, nh:nh + nkv], 1e-2, "keys")
    near(out[2], y[:, nh + nkv:], 1e-2, "values")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("nh,vd", [(3, 64), (1, 7), (5, 96), (2, 300), (1, 515)])
def test_difference_of_two_maps(dtype, nh, vd):
    ops = ops_module()
    g = torch.Generator().manual_seed(vd)
    n = 13
    raw = torch.randn(n, nh, 2, vd, generator=g)
    raw[3] *= 1e-3                                                         # eps inside the root shows
    out = torch.empty(n, nh * vd, dtype=dtype, device="cuda")
    ops.map_difference(raw.cuda(), out, ops.MapDifference(0.83, 1e-4, 0.4))
    want = PP.unit_rms(raw[:, :, 0].double() - 0.83 * raw[:, :, 1].double(), 1e-4) * 0.4
    near(out, want.reshape(n, nh * vd), 1e-5 if dtype == torch.float32 else 1e-2)


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


# (query heads, key/value heads, elements of both maps, elements of a value): the tcgen05 / TMA kernels (64 and 128, up to eight
# maps a key head), more maps than the TMA kernel takes, the mma.sync kernels, the CUDA-core kernels
MAP_SIZES = [(4, 2, 64, 64), (4, 1, 128, 128), (3, 3, 128, 128), (6, 1, 64, 64), (6, 2, 48, 48), (2, 1, 96, 96), (5, 5, 16, 16),
             (4, 2, 24, 20), (2, 1, 10, 33), (2, 2, 128, 64)]


@pytest.mark.parametrize("dtype,tcgen05", [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)], ids=["f32", "bf16", "bf16-mma"])
@pytest.mark.parametrize("nh,nkv,hd,vd", MAP_SIZES)
def test_attention_of_two_maps(monkeypatch, dtype, tcgen05, nh, nkv, hd, vd):
    """A prompt step (old keys in shuffled pages, new ones packed) and a decode step of unequal sequences.  One key far back
    stands out for the first map of head 0 alone and another one for the second map alone, so that maps taken for one another, or
    one softmax over both, would show."""
    ops = ops_module()
    if dtype == torch.bfloat16 and not tcgen05 and hd not in (64, 128):
        pytest.skip("the same kernel either way")
    monkeypatch.setattr(ops, "USE_TC_PROMPT_ATTENTION", tcgen05)
    monkeypatch.setattr(ops, "USE_TMA_DECODE_ATTENTION", tcgen05)
    gen = torch.Generator().manual_seed(nh * hd + vd)
    maps = ops.MapDifference(0.7, 1e-5, 0.45)
    form = ops.AttentionForm(value_dim=vd, maps=maps)
    scale, half = 1.3 * (hd // 2) ** -0.5, hd // 2
    tol = 3e-5 if dtype == torch.float32 else 2e-2
    for decode in (False, True):
        before, counts = ([t - 1 for t in (1, 129, 200, 64, 65)], [1] * 5) if decode else ([0, 130, 5, 64, 0], [33, 1, 70, 100, 200])
        total = [b + c for b, c in zip(before, counts)]
        q, k, v, want = [], [], [], []
        for b, c, t in zip(before, counts, total):
            qs, ks = torch.randn(c, nh, hd, generator=gen), torch.randn(t, nkv, hd, generator=gen)
            if t > 60:
                qs[-1, 0] = 0.0
                qs[-1, 0, 0], qs[-1, 0, half] = 4.0, 4.0
                ks[2, 0, 0] = 6.0 / scale
                ks[t - 59, 0, half] = 6.0 / scale
            q.append(qs.to(dtype).float())
            k.append(ks.to(dtype).float())
            v.append(torch.randn(t, nkv, vd, generator=gen).to(dtype).float())
            full = torch.zeros(t, nh, 2, half, dtype=F64)
            full[b:] = q[-1].double().view(c, nh, 2, half)
            a1, a2 = PP.two_maps(full, k[-1].double().view(t, nkv, 2, half), v[-1].double(), scale)
            want.append((PP.unit_rms(a1 - 0.7 * a2, 1e-5) * 0.45)[b:].reshape(c, nh * vd))
        kp, vp, table, slots = _paged(k, v, total if decode else before, 4, gen, dtype)
        sl, cu, seq, lb, pos = layout(counts, before, slots)
        qd = torch.cat(q).to(dtype).cuda()
        n = qd.shape[0]
        split = decode or not ops.maps_in_kernel(dtype, hd, form)
        if split:
            parts = torch.zeros(n, nh, 2, hd, dtype=dtype, device="cuda")
            parts[:, :, 0, :half], parts[:, :, 1, half:] = qd[..., :half], qd[..., half:]
            qd = parts.view(n, 2 * nh, hd)
        else:
            assert dtype == torch.bfloat16 and tcgen05 and hd == vd and hd in (64, 128)
        out = torch.empty(n, nh * vd, dtype=dtype, device="cuda")
        raw = torch.empty(n, 2 * nh * vd, device="cuda") if split else out
        if decode:
            plan = ops.attn_decode_plan(dtype, n, 2 * nh, nkv, hd, max(total), form)
            scratch = torch.empty(max(1, plan.scratch_floats), device="cuda")
            counters = torch.zeros(max(1, plan.n_counters), dtype=torch.int32, device="cuda")
            ops.attn_decode(qd, kp, vp, table, 4, sl, lb, raw, scratch, scale=scale, window=0, plan=plan, counters=counters, form=form)
        else:
            tq = ops.prefill_tile_queries(dtype, hd, form)
            tiles = torch.tensor([(b, o) for b, c in enumerate(counts) for o in range(0, c, tq)], dtype=torch.int32, device="cuda")
            kn = torch.cat([x[b:] for x, b in zip(k, before)]).to(dtype).cuda()
            vn = torch.cat([x[b:] for x, b in zip(v, before)]).to(dtype).cuda()
            ops.attn_prefill(qd, kn, vn, kp, vp, table, 4, tiles, cu, lb, sl, raw, scale=scale, window=0, tile_queries=tq, form=form)
        if split:
            ops.map_difference(raw.view(n, nh, 2, vd), out, maps)
        near(out, torch.cat(want), tol, ("decode" if decode else "prompt", ))
    if dtype == torch.bfloat16 and tcgen05 and hd in (64, 128):
        assert ops.attn_tc_status() == 0


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_convolution_with_an_activation_and_one_output(taps):
    """silu on what is written, the state without it; output in the compute type alone; steps shorter than the taps and long ones."""
    ops = ops_module()
    g = torch.Generator().manual_seed(taps)
    c, col0, width = 36, 5, 50
    w, bias = torch.randn(c, taps, generator=g), torch.randn(c, generator=g)
    state = torch.zeros(3, max(1, taps - 1), c, device="cuda")
    done = {0: torch.zeros(0, c, dtype=F64), 2: torch.zeros(0, c, dtype=F64)}
    for counts in ((2, 1), (1, 1), (3, 40), (1, 2)):
        n = sum(counts)
        rows = torch.randn(2, n, width, generator=g)
        before = [len(done[0]), len(done[2])]
        sl, cu, seq, lb, pos = layout(counts, before, (0, 2))
        out = torch.empty(n, c, dtype=torch.bfloat16, device="cuda")
        ops.causal_conv(rows.cuda(), col0, w.cuda(), state if taps > 1 else None, sl, cu, seq, lb, None, bias=bias.cuda(), out2=out, act="silu")
        x, o = rows.double().sum(0)[:, col0:col0 + c], 0
        for s, cnt in zip((0, 2), counts):
            done[s] = torch.cat([done[s], x[o:o + cnt]])
            near(out[o:o + cnt], PP.silu(PP.causal_conv(done[s], w, bias))[-cnt:], 1e-2, (counts, s))
            o += cnt


# (heads, vdim, state, groups, tokens of each sequence)
SPACE_SIZES = [(4, 32, 64, 2, (5, 1, 9)), (2, 64, 128, 1, (300, 1, 130)), (6, 16, 16, 3, (64, 65, 63)), (3, 8, 48, 1, (17, 200)),
               (1, 96, 256, 1, (70, 2)), (5, 7, 10, 5, (33, 128)), (2, 300, 20, 1, (18, 3)), (3, 1, 1, 3, (40, 1)), (2, 24, 33, 2, (129, 16)),
               (8, 64, 16, 4, (257,)), (1, 40, 700, 1, (20, 1))]


@pytest.mark.parametrize("dtype,chunks", [(torch.float32, False), (torch.bfloat16, True), (torch.bfloat16, False)], ids=["f32", "bf16", "bf16-walk"])
@pytest.mark.parametrize("gated", [True, False], ids=["gate", "plain"])
@pytest.mark.parametrize("nh,vdim,n_state,groups,counts", SPACE_SIZES)
def test_state_space_walk_and_chunks(monkeypatch, dtype, chunks, gated, nh, vdim, n_state, groups, counts):
    """Both forms from states that earlier tokens left, with heads that hardly forget, heads that forget at once, and steps from
    near nothing to large; the state of a slot that is not in the step stays as it was.  B, C and x are what the compute type
    holds; everything else keeps float32's digits."""
    ops = ops_module()
    monkeypatch.setattr(ops, "USE_STATE_SPACE_MMA", chunks)
    g = torch.Generator().manual_seed(nh * vdim + n_state)
    n, inner, lead = sum(counts), nh * vdim, 3
    width = lead + inner + nh
    rows = torch.randn(2, n, width, generator=g)
    rows[:, :, lead + inner:] *= 3.0
    mixed = torch.randn(n, inner + 2 * groups * n_state, generator=g).to(dtype)
    dt_bias, d_skip = torch.randn(nh, generator=g) - 2.0, torch.randn(nh, generator=g)
    a_log = torch.linspace(-7.0, 3.0, nh) if nh > 1 else torch.tensor([-3.0])
    s0 = torch.randn(len(counts) + 1, nh, n_state, vdim, generator=g)
    slots = list(range(len(counts) - 1, -1, -1))
    sl, cu, _, _, _ = layout(counts, [0] * len(counts), slots)
    state, out = s0.clone().cuda(), torch.empty(n, inner, device="cuda")
    ops.state_space(mixed.cuda(), rows.cuda(), z_col=lead if gated else -1, dt_col=lead + inner, dt_bias=dt_bias.cuda(), a_log=a_log.cuda(),
                    d_skip=d_skip.cuda(), n_heads=nh, groups=groups, n_state=n_state, vdim=vdim, state=state, slots=sl, cu_tokens=cu, out=out,
                    max_count=max(counts))
    r, m = rows.double().sum(0), mixed.double()
    dt = torch.nn.functional.softplus(r[:, lead + inner:] + dt_bias.double(), threshold=1e9)
    x = m[:, :inner].reshape(n, nh, vdim)
    b, c = (m[:, inner + i * groups * n_state:inner + (i + 1) * groups * n_state].reshape(n, groups, n_state) for i in range(2))
    o = 0
    for i, cnt in enumerate(counts):
        y, last = PP.state_space(x[o:o + cnt], b[o:o + cnt], c[o:o + cnt], dt[o:o + cnt], a_log, d_skip, s0[slots[i]])
        y = y.reshape(cnt, inner)
        if gated:
            y = y * PP.silu(r[o:o + cnt, lead:lead + inner])
        near(out[o:o + cnt], y, 1e-4, ("read-out", i))
        near(state[slots[i]], last, 1e-4, ("state", i))
        o += cnt
    assert torch.equal(state[len(counts)].cpu(), s0[len(counts)])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("n,width,parts", [(3, 60, 4), (1, 7, 7), (70, 512, 2), (5, 8192, 1), (100, 96, 3), (2, 20000, 1), (66, 4096, 8), (4, 50, 1)])
def test_norm_in_equal_parts(dtype, n, width, parts):
    ops = ops_module()
    g = torch.Generator().manual_seed(width)
    x, w = torch.randn(n, width, generator=g), torch.randn(width, generator=g)
    x[0] *= 1e-3
    out = torch.empty(n, width, dtype=dtype, device="cuda")
    ops.part_rmsnorm(x.cuda(), w.cuda(), parts, 1e-5, out)
    want = PP.unit_rms(x.view(n, parts, -1), 1e-5).reshape(n, width) * w.double()
    near(out, want, 2e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("experts,identity,top,groups", [(7, 3, 3, (5, 3)), (8, 0, 2, None), (3, 5, 2, (2, 1)), (4, 4, 8, (4, 4)), (1, 1, 1, (2, 1)),
                                                         (60, 4, 6, (16, 5)), (300, 40, 9, (4, 2))])
def test_routing_by_corrected_scores_in_groups(experts, identity, top, groups):
    """Corrections that make most choice scores negative, and change choices; both ways to the logits."""
    ops = ops_module()
    g = torch.Generator().manual_seed(experts)
    n, hidden, routed = 60, 40, experts + identity
    h, wr = torch.randn(n, hidden, generator=g), torch.randn(routed, hidden, generator=g) * 0.4
    corr = 0.2 * torch.randn(routed, generator=g) - 0.3
    rt = {"top": top, "scale": 1.9, "groups": dict(zip(("count", "keep"), groups)) if groups else None}
    idx, wt, margin = PP.route(h, wr, corr, rt)
    plain = PP.route(h, wr, torch.zeros(routed), rt)[0]
    sure = margin > 1e-6
    assert int(sure.sum()) > n // 2 and (top == routed or routed == 2 or not torch.equal(idx, plain))
    rule = ops.RouterRule("softmax_all", groups=groups[0] if groups else 0, keep_groups=groups[1] if groups else 0, group_score_top=1,
                          weight_scale=1.9, normalize=False, correction=corr.cuda())
    for way in ("route", "topk"):
        choice = torch.empty(n, top, dtype=torch.int32, device="cuda")
        weight = torch.empty(n, top, device="cuda")
        if way == "route":
            ops.moe_route(h.cuda(), wr.cuda(), None, choice, weight, rule)
        else:
            z = h @ wr.t()
            ops.moe_topk(torch.stack([0.3 * z, 0.7 * z]).contiguous().cuda(), None, choice, weight, rule)
        for t in torch.nonzero(sure).flatten().tolist():
            assert sorted(choice[t].tolist()) == sorted(idx[t].tolist()), (way, t)
            order = {e: float(x) for e, x in zip(idx[t].tolist(), wt[t])}
            assert all(abs(float(x) - order[e]) < 1e-5 for e, x in zip(choice[t].tolist(), weight[t])), (way, t)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("n,experts,identity,top,hidden,inner", [(1, 4, 2, 2, 64, 32), (40, 5, 1, 3, 72, 48), (37, 3, 3, 6, 50, 10),
                                                                 (600, 2, 2, 2, 128, 192), (5, 1, 7, 1, 64, 16)])
def test_mixture_with_identity_experts(dtype, n, experts, identity, top, hidden, inner):
    """The feed-forward part alone: tiles of 32 rows and of 128, no pair at all for an expert, tokens that only pass themselves on."""
    from importlib import import_module
    base = import_module("daisi-llogos_b200.parts.base")
    moe = import_module("daisi-llogos_b200.parts.moe")
    ops = ops_module()
    g = torch.Generator().manual_seed(n + experts)
    routed = experts + identity
    env = base.BuildEnv(dtype=dtype, device=torch.device("cuda"), ops=ops, encodings={})
    part = moe.MoeFeedForward({"hidden_size": hidden, "num_experts": experts, "identity": identity, "top": top, "expert_size": inner,
                               "score": "softmax_all", "normalize": False, "correction": True, "weight_scale": 2.3, "activation": "clamped",
                               "gate_alpha": 1.702, "up_offset": 1.0, "limit": 0.7}, "", env)
    w = {}
    for name, d in part.tensors().items():
        w[name] = (1.5 * d.shape[-1] ** -0.5 * torch.randn(d.shape, generator=g)).to(dtype)
    # no close calls: every token's logits are whole halves in an order of its own, and the corrections all one number
    w["router.weight"] = torch.zeros(routed, hidden, dtype=dtype)
    w["router.weight"][:, :routed] = torch.eye(routed)
    w["correction"][:] = -0.75
    part.bind({k: v.cuda() for k, v in w.items()})
    x = torch.randn(n, hidden, generator=g)
    x[:, :routed] = torch.stack([torch.randperm(routed, generator=g) for _ in range(n)]).float() * 0.5 - 1.0
    x = x.to(dtype)
    got = part.forward(x.cuda(), part_context(ops, dtype)).data.sum(0)
    names = {"router": w["router.weight"], "correction": w["correction"]}
    for i in range(experts):
        for what in ("gate", "up", "down"):
            names[f"e{i}.{what}"] = w[f"experts.{i}.{what}_proj.weight"]
    ml = {"router": {"experts": experts, "identity": identity, "top": top, "scale": 2.3}, "expert": {"ff": inner, "limit": 0.7}}
    near(got, PP.mixture(x.double(), names, "", ml), 3e-5 if dtype == torch.float32 else 2e-2)


# ---- whole models ------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", list(PM.CONFIGS))
def test_whole_prompts_and_first_tokens(engines, models, name, dtype):
    eng = engines(name, dtype)
    for n in (1, 2, 3, 5, 64, 65, 330, 700):
        toks, ref = sequence(models, name, dtype, n, n)
        slot = eng.open()
        close(eng.step([(slot, toks)], [list(range(n))]), ref, dtype, (name, "whole", n))
        eng.close(slot)


@pytest.mark.parametrize("name", list(PM.CONFIGS))
def test_residual_after_every_layer(llogos, models, name):
    """float32: the residual after each layer, read from the engine by models that are cut short, is the plain model's."""
    import os
    d, cfg, w = models[name, torch.float32]
    toks, _ = sequence(models, name, torch.float32, 50, 4)
    trace = []
    PP.forward(w, cfg, toks, trace)
    for depth in range(1, len(cfg["layers"]) + 1):
        cut = dict(cfg, layers=cfg["layers"][:depth])
        keep = {k: v for k, v in w.items() if not (k[0] == "l" and k[1].isdigit() and int(k[1:k.index(".")]) >= depth)}
        sub = os.path.join(d, f"cut{depth}")
        PM.write_model(llogos, sub, cut, 0, weights={k: v.to(torch.bfloat16) for k, v in keep.items()})
        eng = llogos.engine.Engine(llogos.weights.load_model(sub, dtype=torch.float32, device="cuda:0"), max_tokens=256)
        slot = eng.open()
        lg = eng.step([(slot, toks)], [list(range(len(toks)))])
        close(lg, PP.linear(PP.rms_norm(trace[depth - 1], w["final.norm"], cfg["norm"]["eps"]), w["embed"]), torch.float32, ("after", depth))
        eng.close(slot)


@pytest.mark.parametrize("graphs", [True, False], ids=["graph", "eager"])
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", list(PM.CONFIGS))
def test_prompt_then_token_by_token(engines, models, name, dtype, graphs):
    """The decoded positions pass page borders (128, 192) and borders of the query factors' steps; the first token alone too."""
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
@pytest.mark.parametrize("name", list(PM.CONFIGS))
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
@pytest.mark.parametrize("name", list(PM.CONFIGS))
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
def test_one_token_beside_a_prompt(engines, models, dtype):
    """A request that goes on by one token in the same step in which another brings hundreds."""
    name = "tensor"
    eng = engines(name, dtype)
    (a, ra), (b, rb) = sequence(models, name, dtype, 90, 31), sequence(models, name, dtype, 230, 32)
    sa, sb = eng.open(), eng.open()
    eng.step([(sa, a[:88])], [[]])
    lg = eng.step([(sa, a[88:89]), (sb, b[:200])], [[0], [0, 199]])
    close(lg, torch.stack([ra[88], rb[0], rb[199]]), dtype, ("one token beside a prompt",))
    lg = eng.step([(sb, b[200:]), (sa, a[89:])], [[29], [0]])
    close(lg, torch.stack([rb[229], ra[89]]), dtype, ("the rest",))
    eng.close(sa)
    eng.close(sb)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_long_decoding(engines, models, dtype):
    """420 decoded tokens after a prompt of 30: the states are carried through every step, the keys grow over seven pages."""
    name = "mixed"
    eng = engines(name, dtype)
    toks, ref = sequence(models, name, dtype, 450, 5)
    slot = eng.open()
    eng.step([(slot, toks[:30])], [[]])
    got = [eng.step([(slot, [toks[p]])]).clone() for p in range(30, len(toks))]
    close(torch.cat(got), ref[30:], dtype, ("long decoding",))
    eng.close(slot)


def _random_config(seed, tensor_cores=False):
    """A configuration drawn from the seed: two to five layers of both kinds in any order, and every size, limit, factor and group
    drawn; with ``tensor_cores`` of sizes that those kernels take."""
    g = torch.Generator().manual_seed(4000 + seed + 500 * tensor_cores)
    pick = lambda xs: xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    layers = []
    for _ in range(pick([2, 3, 4, 5])):
        mlp = None
        if pick([0, 1, 1, 1]):
            experts, identity = pick([1, 2, 3, 6, 9]), pick([0, 1, 3, 6])
            routed = experts + identity
            counts = [c for c in range(2, routed + 1) if routed % c == 0]
            groups = None
            if counts and pick([0, 1, 1]):
                count = pick(counts)
                groups = (count, pick(list(range(1, count + 1))))
            most = routed if groups is None else groups[1] * (routed // groups[0])
            mlp = PM.moe(experts, pick(list(range(1, most + 1))), pick([32, 72] if tensor_cores else [8, 24, 7]), pick([0.5, 1.0, 7.0]), identity,
                         groups, pick([0.6, 1.0, 2.5]))
        if pick([0, 1]):
            groups = pick([1, 2, 3])
            heads, vdim = groups * pick([1, 2, 3]), pick([16, 32, 48, 64] if tensor_cores else [3, 8, 20, 40])
            mix = PM.mamba(heads, vdim, pick([16, 32, 80, 128] if tensor_cores else [1, 6, 20, 33]), groups, pick([1, 2, 4, 5]),
                           pick([p for p in range(1, heads * vdim + 1) if heads * vdim % p == 0][:6]))
        else:
            kv, dim = pick([1, 2, 3]), pick([8, 16, 24, 32, 40, 64] if tensor_cores else [3, 8, 12, 20])
            mix = PM.attention(kv * pick([1, 2, 4]), kv, dim, 2 * dim if tensor_cores else pick([5, 8, 24]), scale=pick([0.1, 0.3]),
                               diff=pick([0.0, 0.35, 0.8]), temp=pick([None, (0.2, 40), (0.5, 7)]))
        layers.append(PM.layer(mix, mlp))
    return PM.config(layers, vocab=pick([61, 128, 257]), width=pick([64, 128, 200] if tensor_cores else [48, 64, 72, 90]), eps=pick([1e-6, 1e-5, 1e-3]))


@pytest.mark.parametrize("seed", range(14))
def test_configurations_drawn_at_random(llogos, tmp_path, seed):
    """float32: a prompt whole, a batch of two unequal prompts decoded together for a dozen steps, against the plain model."""
    cfg = _random_config(seed)
    d = str(tmp_path / "m")
    w = {k: v.float() for k, v in PM.write_model(llogos, d, cfg, seed=seed).items()}
    eng = llogos.engine.Engine(llogos.weights.load_model(d, dtype=torch.float32, device="cuda:0"), max_tokens=64 * 12)
    g = torch.Generator().manual_seed(seed)
    seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (171, 40)]
    refs = [PP.forward(w, cfg, s) for s in seqs]
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


@pytest.mark.parametrize("seed", range(8))
def test_tensor_core_configurations_drawn_at_random(llogos, tmp_path, seed):
    """bfloat16: a prompt whole, and a batch of two unequal prompts decoded together, against the plain model."""
    cfg = _random_config(seed, tensor_cores=True)
    d = str(tmp_path / "m")
    w = {k: v.float() for k, v in PM.write_model(llogos, d, cfg, seed=seed, steady_routing=True).items()}
    eng = llogos.engine.Engine(llogos.weights.load_model(d, dtype=torch.bfloat16, device="cuda:0"), max_tokens=64 * 12)
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
    close(torch.stack([x[0] for x in got]), ra[cut[0]:], torch.bfloat16, ("random", seed, "decoded, long"))
    close(torch.stack([x[1] for x in got]), rb[cut[1]:], torch.bfloat16, ("random", seed, "decoded, short"))


# ---- faults that random weights would hide ---------------------------------------------------------

A_TOK, B_TOK = 11, 12


def _far_model(llogos, folder, kind):
    """One layer without a feed-forward, made so that only token a answers what token b asks along a direction z (every other
    token's normed embedding is orthogonal to z).  "map1", "map2": that map of head 0 finds a among hundreds of keys, and no other
    query or key of the layer says anything; at b the queries' factor is large.  "state": every token but a and b takes a step of
    almost nothing, head 0 hardly forgets and holds a's x under z."""
    d = 48
    mixer = PM.mamba(2, 24, 16, 1, 4, 1) if kind == "state" else PM.attention(4, 2, 16, 24, scale=0.5, diff=0.3, temp=(0.5, 100))
    cfg = PM.config([PM.layer(mixer, None)], vocab=50, width=d)
    w = PM.random_weights(cfg, 77)
    gen = torch.Generator().manual_seed(1)
    z = torch.randn(d, generator=gen)
    z = z / z.norm()
    emb = w["embed"].float()
    emb -= (emb @ z)[:, None] * z[None, :]
    r = [torch.randn(d, generator=gen) for _ in range(2)]
    r = [x - (x @ z) * z for x in r]
    for tok, x in zip((A_TOK, B_TOK), r):
        emb[tok] = 5.0 * z + 5.0 * x / x.norm()
    w["embed"] = emb.to(torch.bfloat16)
    w["l0.norm1"][:] = 1.0
    p = "l0.mix."
    w[p + "o"] = (4.0 * w[p + "o"].float()).to(torch.bfloat16)             # what the layer finds weighs on the logits
    e = torch.ones(16) / 4.0
    row = (1.8 * e[:, None] * z[None, :]).to(torch.bfloat16)
    if kind == "state":
        inner, n = 48, 16
        w_in = w[p + "in"]
        w_in[2 * inner:2 * inner + n], w_in[2 * inner + n:2 * inner + 2 * n] = row, row             # B and C
        w_in[2 * inner + 2 * n:] = (1.5 * z).to(torch.bfloat16)
        conv = torch.zeros(inner + 2 * n, 4)
        conv[:, 3] = 1.0
        w[p + "conv"] = conv.to(torch.bfloat16)
        w[p + "conv.b"][:] = 0.0
        w[p + "dt_bias"][:] = -9.0
        w[p + "A_log"][:] = torch.tensor([-8.0, 6.0]).to(torch.bfloat16)                           # the second head forgets at once
    else:
        m = int(kind[-1]) - 1
        for n in ("q", "k"):
            w[p + n][:] = 0.0
            w[p + n + ".b"][:] = 0.0
            w[p + n][16 * m:16 * m + 16] = row
    PM.write_model(llogos, folder, cfg, 0, weights=w)
    return cfg, {k: v.float() for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("kind", ["map1", "map2", "state"])
def test_what_token_a_left_330_positions_back(llogos, tmp_path, dtype, kind):
    """Token a stands at position 2, token b 330 positions (five pages, five chunks of the state's walk) later.  b's logits
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
    refs = [PP.forward(wf, cfg, t) for t in (with_a, without_a)]
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
            margins = []
            lg = PP.forward(w, cfg, toks, margins=margins)[-1]
            if dtype == torch.bfloat16 and margins and float(torch.stack(margins).min()) <= MARGIN:
                break                              # made tokens may bring a router a close call: what follows hangs on rounding
            slack = 1e-4 if dtype == torch.float32 else 0.05
            assert float(lg[tok]) >= float(lg.max()) - slack * float(lg.abs().max()), (len(toks), tok)
            toks.append(tok)


def test_command_line_and_trace_replay_take_the_design(models, tmp_path):
    """``python -m llogos_b200`` generates with a Penasun folder, and ``bin/trace_run`` replays steps on it (two requests
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
        lg = PP.forward(w, cfg, toks)[-1]
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
