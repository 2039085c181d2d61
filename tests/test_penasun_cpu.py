"""The Penasun decoder without a GPU: its configuration reader and spec, the plain implementation's mechanisms against
closed forms, and the engine's host logic (packing, cache units that keep several things, state slots used again) over the
CPU stand-ins of the kernels against the plain implementation."""
import copy
import importlib
import math

import pytest
import torch

import cpu_ops
import penasun_models as PM
import penasun_plain as PP

F64 = torch.float64


def test_reader_takes_every_size_from_the_file_and_names_the_key_of_an_error(llogos):
    raw = PM.CONFIGS["mixed"]
    cfg = llogos.config.registry.architecture_of(raw).read_config(raw)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, len(cfg.layers)) == (179, 88, 1e-5, 5)
    s, a = cfg.layers[0].mixer, cfg.layers[1].mixer
    assert (s.heads, s.vdim, s.state, s.groups, s.conv, s.norm_groups) == (6, 10, 12, 3, 4, 4)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.diff, a.q_temp.coef, a.q_temp.every) == (4, 2, 12, 20, 0.4, 0.3, 0.25, 37)
    m = cfg.layers[0].mlp
    assert (m.experts, m.identity, m.top, m.scale, m.groups, m.keep_groups, m.expert.ff, m.expert.limit) == (7, 3, 3, 1.7, 5, 3, 24, 1.2)
    assert cfg.layers[2].mlp is None and cfg.layers[4].mlp.groups == 0
    odd = llogos.config.registry.architecture_of(PM.CONFIGS["odd"]).read_config(PM.CONFIGS["odd"])
    assert odd.layers[1].mixer.q_temp is None and odd.layers[1].mixer.diff == 0.0 and odd.layers[2].mlp.identity == 0
    bare = copy.deepcopy(raw)
    for key in ("identity", "groups", "scale"):
        del bare["layers"][0]["mlp"]["router"][key]
    m = llogos.config.registry.architecture_of(bare).read_config(bare).layers[0].mlp
    assert (m.identity, m.groups, m.scale) == (0, 0, 1.0)
    ConfigError = llogos.config.ConfigError
    for path, value, word in ((("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"), (("layers", 0, "mlp", "router", "top"), 11, "top"),
                              (("layers", 0, "mlp", "router", "top"), 7, "top"), (("layers", 0, "type"), "conv", "type"),
                              (("layers", 0, "mixer", "groups"), 4, "groups"), (("layers", 0, "mixer", "norm_groups"), 7, "norm_groups"),
                              (("layers", 0, "mixer", "state"), None, "state"), (("layers", 0, "mixer", "conv"), 0, "conv"),
                              (("layers", 1, "mlp", "kind"), "dense", "kind"), (("layers", 1, "mixer", "q_temp", "every"), 0, "every"),
                              (("layers", 1, "mixer", "diff"), None, "diff"), (("layers", 1, "mixer", "scale"), 0.0, "scale"),
                              (("layers", 1, "mixer"), None, "mixer"), (("layers", 0, "mlp", "router", "groups", "count"), 4, "groups"),
                              (("layers", 0, "mlp", "router", "groups", "keep"), 6, "groups"), (("layers", 0, "mlp", "router", "identity"), -1, "identity"),
                              (("layers", 0, "mlp", "expert", "limit"), -1.0, "limit"), (("norm", "eps"), 0.0, "eps")):
        bad = copy.deepcopy(raw)
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            llogos.config.registry.architecture_of(bad).read_config(bad)


def test_spec_names_parts_tensors_and_cache_units(llogos):
    for name, cfg in PM.CONFIGS.items():
        model = llogos.weights.build_model(cfg, dtype=torch.float32, device="cpu", ops=cpu_ops)
        assert {n: tuple(d.shape) for n, d in model.tensor_decls().items()} == {n: tuple(t.shape) for n, t in PM.random_weights(cfg, 0).items()}
    model = llogos.weights.build_model(PM.CONFIGS["mixed"], dtype=torch.float32, device="cpu", ops=cpu_ops)
    base = llogos.parts.base
    needs = model.cache_needs()
    assert needs[1] == base.KvNeed(2, 24, 0, 20) and needs[3] == base.KvNeed(3, 16, 0, 0)      # two maps are one key row
    assert dict(needs[0].needs) == {"state": base.StateNeed((6, 12, 10), torch.float32), "conv": base.StateNeed((3, 132), torch.float32)}
    assert len(needs) == 5 and len(model.spec.encodings) == 2
    odd = llogos.weights.build_model(PM.CONFIGS["odd"], dtype=torch.float32, device="cpu", ops=cpu_ops)
    assert odd.cache_needs()[0] == base.StateNeed((1, 10, 7), torch.float32)                   # one tap: nothing of the convolution is kept


def test_parts_refuse_what_does_not_go_together(llogos):
    base = importlib.import_module("daisi-llogos_b200.parts.base")
    att = importlib.import_module("daisi-llogos_b200.parts.attention")
    moe = importlib.import_module("daisi-llogos_b200.parts.moe")
    norm = importlib.import_module("daisi-llogos_b200.parts.norm")
    env = base.BuildEnv(dtype=torch.float32, device=torch.device("cpu"), ops=cpu_ops, encodings={})
    plain = {"hidden_size": 8, "num_heads": 2, "num_kv_heads": 1, "head_dim": 4, "maps": 2, "diff": 0.5, "diff_eps": 1e-5}
    att.Attention(dict(plain), "", env)
    for extra in ({"sink": "learned"}, {"softcap": 3.0}, {"head_gate": True}, {"own_kv": False}, {"conv_taps": 2}, {"maps": 3}):
        with pytest.raises(ValueError):
            att.Attention(dict(plain, **extra), "", env)
    mix = {"hidden_size": 8, "num_experts": 3, "top": 2, "expert_size": 4, "identity": 2, "score": "softmax_all", "correction": True}
    moe.MoeFeedForward(dict(mix), "", env)
    for extra in ({"score": "softmax"}, {"weight_on": "input"}, {"top": 6}, {"groups": 2, "keep_groups": 1}, {"identity": -1}):
        with pytest.raises(ValueError):
            moe.MoeFeedForward(dict(mix, **extra), "", env)

    class Ctx:
        ops, dtype = cpu_ops, torch.float32
        buffer = staticmethod(lambda name, shape, dtype=None, zero=False: torch.zeros(shape))
    biased = base.Branch(torch.ones(1, 2, 4), bias=torch.full((4,), 2.0))
    rms = norm.RmsNorm({"size": 4, "eps": 1e-5}, "", env)
    rms.bind({"weight": torch.ones(4)})
    res = torch.zeros(2, 4)
    rms.forward(res, biased, Ctx)
    assert torch.equal(res, torch.full((2, 4), 3.0))
    ln = norm.LayerNorm({"size": 4, "eps": 1e-5, "bias": False}, "", env)
    ln.bind({"weight": torch.ones(4)})
    with pytest.raises(ValueError, match="bias"):
        ln.forward(torch.zeros(2, 4), biased, Ctx)
    with pytest.raises(ValueError, match="bias"):
        biased.as_terms()


def test_query_factors_are_tabled_as_far_as_the_cache_reaches():
    base = importlib.import_module("daisi-llogos_b200.parts.base")
    pos = importlib.import_module("daisi-llogos_b200.parts.position")
    env = base.BuildEnv(dtype=torch.float32, device=torch.device("cpu"), ops=cpu_ops, encodings={})
    q = pos.QueryTemperature({"coef": 0.5, "every": 3}, "", env)
    assert q.limit() is None and q.rotation() is None
    q.prepare(7)
    want = [1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3), 1 + 0.5 * math.log(3)]
    assert torch.allclose(q.query_scale(), torch.tensor(want)) and q.limit() == 7
    q.prepare(4)
    assert q.limit() == 7
    q.prepare(9)
    assert q.limit() == 9 and torch.allclose(q.query_scale().double(), PP.query_temperature(torch.arange(9), {"coef": 0.5, "every": 3}), atol=1e-7)


def test_plain_mechanisms_against_closed_forms():
    # convolution: the last column weighs the current token, the first the oldest; zeros before the start
    y = PP.causal_conv(torch.tensor([[1.0], [10.0], [100.0]]), torch.tensor([[2.0, 3.0]]), torch.tensor([0.5]))
    assert y.flatten().tolist() == [3.5, 32.5, 320.5]
    # the state with a decay of one half and a step of one: S = 1, 1/2 + 10, (1/2 + 10) / 2 + 100, y = S C + D x
    one = torch.ones(3, 1, 1, dtype=F64)
    x = torch.tensor([1.0, 10.0, 100.0], dtype=F64).view(3, 1, 1)
    y, s = PP.state_space(x, one, 2 * one, torch.ones(3, 1, dtype=F64), torch.tensor([math.log(math.log(2.0))]), torch.tensor([0.1]))
    assert torch.allclose(y.flatten(), torch.tensor([2.1, 22.0, 220.5], dtype=F64), atol=1e-5) and abs(float(s) - 105.25) < 1e-5
    # groups: heads 0, 1 read group 0, heads 2, 3 group 1
    b = torch.tensor([[[1.0], [5.0]]], dtype=F64)
    y, _ = PP.state_space(torch.ones(1, 4, 1, dtype=F64), b, torch.ones(1, 2, 1, dtype=F64), torch.ones(1, 4, dtype=F64), torch.zeros(4), torch.zeros(4))
    assert y.flatten().tolist() == [1.0, 1.0, 5.0, 5.0]
    # the gate comes before the norm, every part by its own root mean square
    y = PP.gated_group_norm(torch.tensor([[3.0, 3.0, -0.5, 0.5]]), torch.full((1, 4), 40.0), torch.tensor([1.0, 2.0, 1.0, 1.0]), 2, 0.0)
    assert torch.allclose(y, torch.tensor([[1.0, 2.0, -1.0, 1.0]], dtype=F64))
    # query factors: the first `every - 1` positions are as they are
    f = PP.query_temperature(torch.tensor([0, 98, 99, 298, 299]), {"coef": 2.0, "every": 100})
    assert torch.allclose(f, torch.tensor([1.0, 1.0, 1 + 2 * math.log(2), 1 + 2 * math.log(3), 1 + 2 * math.log(4)], dtype=F64))
    # two maps over the same values: map 1 weighs both keys alike, map 2 (score log 3 against 0) weighs them 3 : 1
    q = torch.zeros(2, 1, 2, 1, dtype=F64)
    q[1, 0, 1, 0] = 1.0
    k = torch.zeros(2, 1, 2, 1, dtype=F64)
    k[0, 0, 1, 0] = math.log(3.0)
    a1, a2 = PP.two_maps(q, k, torch.tensor([4.0, 8.0], dtype=F64).view(2, 1, 1), 1.0)
    assert torch.allclose(a1.flatten(), torch.tensor([4.0, 6.0], dtype=F64)) and torch.allclose(a2.flatten(), torch.tensor([4.0, 5.0], dtype=F64))
    lam = PP.difference_factor(torch.tensor([1.0, 0.0]), torch.tensor([math.log(2.0), 7.0]), torch.zeros(2), torch.ones(2), 0.25)
    assert abs(lam - 1.25) < 1e-6
    # routing: scores are a softmax over all; the correction chooses, the plain score weighs; of two groups {0, 1} and {2, 3} the
    # one of the largest corrected score stays, and a negative choice score inside it is still taken before the other group
    z = torch.tensor([[math.log(4.0), math.log(3.0), math.log(2.0), 0.0]])
    c, wt, margin = PP.route(z, torch.eye(4), torch.tensor([0.0, -0.9, 0.1, 0.0]), {"top": 2, "scale": 10.0, "groups": {"count": 2, "keep": 1}})
    assert c.tolist() == [[0, 1]] and torch.allclose(wt, torch.tensor([[4.0, 3.0]], dtype=F64)) and abs(float(margin) - 0.1) < 1e-6
    # identity experts return their input times their weight
    w = {"router": torch.tensor([[0.0], [0.0]]), "correction": torch.tensor([0.0, 1.0])}
    got = PP.mixture(torch.tensor([[6.0]]), w, "", {"router": {"experts": 1, "top": 1, "identity": 1, "scale": 3.0}, "expert": {"ff": 1, "limit": 1.0}})
    assert abs(float(got) - 9.0) < 1e-12
    w.update({"e0.gate": torch.ones(1, 1), "e0.up": torch.ones(1, 1), "e0.down": torch.ones(1, 1), "correction": torch.tensor([1.0, 0.0])})
    got = PP.mixture(torch.tensor([[6.0]]), w, "", {"router": {"experts": 1, "top": 1, "identity": 1, "scale": 1.0}, "expert": {"ff": 1, "limit": 2.0}})
    assert abs(float(got) - 0.5 * 2.0 / (1 + math.exp(-3.404)) * 3.0) < 1e-12


@pytest.mark.parametrize("name", list(PM.CONFIGS))
def test_engine_host_logic_on_stand_ins(llogos, tmp_path, name):
    """Whole prompts, portions down to two tokens, a token decoded alone, unequal batches and slots used again give the plain
    model's logits when the kernels are the CPU stand-ins."""
    cfg = PM.CONFIGS[name]
    w = PM.write_model(llogos, str(tmp_path), cfg, seed=5)
    wf = {k: v.float() for k, v in w.items()}
    model = llogos.weights.load_model(str(tmp_path), dtype=torch.float32, device="cpu", ops=cpu_ops)
    eng = llogos.engine.Engine(model, max_tokens=64 * 12, n_slots=3, use_graphs=False)
    g = torch.Generator().manual_seed(3)
    seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (1, 25, 68, 9)]
    refs = [PP.forward(wf, cfg, s) for s in seqs]

    def close(got, ref, what):
        err = float((got.double() - ref).abs().max() / ref.abs().max())
        assert err < 2e-4, (name, what, err)

    slot = eng.open()
    at, got = 0, []
    for s in (2, 2, 3, 1, 1, 27, 2, 30):
        got.append(eng.step([(slot, seqs[2][at:at + s])], [list(range(s))]).clone())
        at += s
    close(torch.cat(got), refs[2], "portions")
    eng.close(slot)
    for rounds in range(2):                      # the second round finds slots, pages and state rows used before
        slots = [eng.open() for _ in range(3)]
        order = [1, 0, 3] if rounds else [3, 1, 0]
        cut = {i: max(1, len(seqs[i]) - 4) for i in order}
        lg = eng.step([(slots[j], seqs[i][:cut[i]]) for j, i in enumerate(order)])
        for j, i in enumerate(order):
            close(lg[j], refs[i][cut[i] - 1], ("batched prompt", i))
        live = [(j, i) for j, i in enumerate(order) if cut[i] < len(seqs[i])]
        while live:
            lg = eng.step([(slots[j], [seqs[i][cut[i]]]) for j, i in live])
            for r, (j, i) in enumerate(live):
                close(lg[r], refs[i][cut[i]], ("batched decode", i, cut[i]))
                cut[i] += 1
            live = [(j, i) for j, i in live if cut[i] < len(seqs[i])]
        for s in slots:
            eng.close(s)
        eng.cache.audit()
    assert eng.cache.slots.free_count == eng.cache.slots.n_slots


def test_cost_model_counts_both_maps_the_chosen_experts_and_no_pairs_for_a_state(llogos):
    measure = importlib.import_module("daisi-llogos_b200.measure")
    cfg = PM.CONFIGS["mixed"]
    model = llogos.weights.build_model(cfg, dtype=torch.bfloat16, device="cpu", ops=cpu_ops)
    costs = measure.model_costs(model)
    d, pairs, stored, active = cfg["width"], 0, 0, 0
    for lay in cfg["layers"]:
        m = lay["mixer"]
        inner = m["heads"] * m["vdim"]
        if lay["type"] == "mamba2":
            n = d * (2 * inner + 2 * m["groups"] * m["state"] + m["heads"]) + d * inner
        else:
            n = d * (2 * m["dim"] * (m["heads"] + m["kv_heads"]) + m["kv_heads"] * m["vdim"]) + d * inner
            pairs += 2 * m["heads"] * 2 * (m["dim"] + m["vdim"])
        ml = lay["mlp"]
        r = ml["router"] if ml else None
        e = 0 if not ml else d * (r["experts"] + r["identity"])
        x = 0 if not ml else 3 * d * ml["expert"]["ff"]
        stored += n + e + (0 if not ml else r["experts"] * x)
        active += n + e + (0 if not ml else r["top"] * x)
    assert (costs.matrix_params, costs.active_params, costs.attn_flops_per_pair) == (stored, active, pairs)
    assert [u for u in costs.kv_units] == [(2 * (24 + 20) * 2, 0), (3 * (16 + 16) * 2, 0)]


def test_a_norm_ahead_of_no_feed_forward_is_skipped_with_a_warning(llogos, tmp_path):
    cfg = PM.CONFIGS["odd"]
    w = PM.random_weights(cfg, 3)
    w["l3.norm2"] = torch.ones(cfg["width"], dtype=torch.bfloat16)
    PM.write_model(llogos, str(tmp_path), cfg, 0, weights=w)
    model = llogos.weights.load_model(str(tmp_path), dtype=torch.float32, device="cpu", ops=cpu_ops)
    assert any("l3.norm2" in x for x in model.load_warnings)


def test_fixed_size_state_refuses_a_rollback(llogos, tmp_path):
    cfg = PM.CONFIGS["odd"]
    PM.write_model(llogos, str(tmp_path), cfg, seed=1)
    model = llogos.weights.load_model(str(tmp_path), dtype=torch.float32, device="cpu", ops=cpu_ops)
    eng = llogos.engine.Engine(model, max_tokens=128, n_slots=2, use_graphs=False)
    slot = eng.open()
    eng.step([(slot, [1, 2, 3])])
    with pytest.raises(llogos.engine.StepError, match="rolled back"):
        eng.truncate(slot, 1)
