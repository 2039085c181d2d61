"""The Memilorn decoder without a GPU: its configuration reader and spec, the plain implementation's mechanisms against
closed forms, and the engine's host logic (packing, cache units that keep several things, a loop whose later rounds add the
embedding again, state slots used again) over the CPU stand-ins of the kernels against the plain implementation."""
import copy
import math

import pytest
import torch

import cpu_ops
import memilorn_models as MM
import memilorn_plain as MP

F64 = torch.float64


def test_reader_takes_every_size_from_the_file_and_names_the_key_of_an_error(llogos):
    raw = MM.CONFIGS["mixed"]
    cfg = llogos.config.registry.architecture_of(raw).read_config(raw)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, len(cfg.layers), cfg.loop) == (179, 88, 1e-5, 5, (1, 4, 3))
    a, s, l = (cfg.layers[i].mixer for i in range(3))
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.rot.dims, a.rot.base) == (4, 2, 16, 24, 0.3, 5.0, 8, 500.0)
    assert (s.heads, s.dim, s.vdim, s.gate_cap) == (3, 16, 40, 8.0) and (l.heads, l.dim, l.vdim, l.kv_rank, l.scale) == (5, 24, 16, 32, 0.25)
    m = cfg.layers[0].mlp
    assert (m.experts, m.top, m.expert.ff, m.expert.limit, m.shared.ff, m.shared.limit) == (6, 2, 24, 1.2, 40, 0.8)
    assert cfg.layers[2].mlp is None and cfg.layers[3].mlp.shared is None
    assert cfg.run_order() == ((0, False), (1, False), (2, False), (3, False), (1, True), (2, False), (3, False), (1, True), (2, False),
                               (3, False), (4, False))
    assert list(cfg.run_order()) == MP.run_order(raw)
    odd = llogos.config.registry.architecture_of(MM.CONFIGS["odd"]).read_config(MM.CONFIGS["odd"])
    assert odd.loop is None and odd.layers[1].mixer.softcap == 0.0 and odd.layers[3].mixer.rot is None
    ConfigError = llogos.config.ConfigError
    for path, value, word in ((("layers", 0, "mixer", "kv_heads"), 3, "kv_heads"), (("layers", 0, "mlp", "router", "top"), 7, "top"),
                              (("layers", 0, "type"), "conv", "type"), (("layers", 1, "mixer", "gate_cap"), 0, "gate_cap"),
                              (("layers", 1, "mlp", "kind"), "dense", "kind"), (("layers", 0, "mixer", "rot", "dims"), 7, "rot.dims"),
                              (("layers", 2, "mixer", "kv_rank"), None, "kv_rank"), (("layers", 1, "mixer"), None, "mixer"),
                              (("layers", 0, "mlp", "shared", "limit"), -1.0, "shared.limit"), (("loop", "stop"), 9, "loop"),
                              (("layers", 0, "mixer", "softcap"), -2.0, "softcap"), (("norm", "eps"), 0.0, "eps")):
        bad = copy.deepcopy(raw)
        node = bad
        for k in path[:-1]:
            node = node[k]
        node[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            llogos.config.registry.architecture_of(bad).read_config(bad)


def test_spec_names_parts_tensors_and_cache_units(llogos):
    for name, cfg in MM.CONFIGS.items():
        model = llogos.weights.build_model(cfg, dtype=torch.float32, device="cpu", ops=cpu_ops)
        assert {n: tuple(d.shape) for n, d in model.tensor_decls().items()} == {n: tuple(t.shape) for n, t in MM.random_weights(cfg, 0).items()}
    cfg = MM.CONFIGS["mixed"]
    model = llogos.weights.build_model(cfg, dtype=torch.float32, device="cpu", ops=cpu_ops)
    base = llogos.parts.base
    needs = model.cache_needs()
    assert [e.layer for e in model.spec.schedule] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4] and len(needs) == 11
    assert [i for i, e in enumerate(model.spec.schedule) if e.add_embedding] == [4, 7]
    assert needs[0] == base.KvNeed(2, 16, 0, 24) and needs[10] == base.KvNeed(3, 8, 0, 0)
    assert needs[2] == base.KvNeed(1, 32, 0, values_in_keys=True) == needs[5] == needs[8]
    assert dict(needs[1].needs) == {"memory": base.StateNeed((3, 16, 40), torch.float32), "normaliser": base.StateNeed((3, 16), torch.float32),
                                    "maximum": base.StateNeed((3,), torch.float32)} == dict(needs[7].needs)
    assert [type(b).__name__ for b in model.blocks] == ["PreNormBlock"] * 5 and len(model.spec.encodings) == 2
    with pytest.raises(ValueError, match="add_embedding"):
        spec = llogos.parts.spec if hasattr(llogos.parts, "spec") else __import__("importlib").import_module("daisi-llogos_b200.parts.spec")
        bad = spec.ModelSpec(**{**model.spec.__dict__, "schedule": (spec.ScheduleEntry(0, add_embedding=True),)})
        bad.validate()


def test_norms_refuse_what_they_cannot_add(llogos):
    import importlib
    base = importlib.import_module("daisi-llogos_b200.parts.base")
    norm = importlib.import_module("daisi-llogos_b200.parts.norm")
    env = base.BuildEnv(dtype=torch.float32, device=torch.device("cpu"), ops=cpu_ops, encodings={})
    b = base.Branch(torch.zeros(1, 2, 4)).with_gain(torch.ones(4))
    rms = norm.RmsNorm({"size": 4, "eps": 1e-5}, "", env)
    rms.bind({"weight": torch.ones(4)})

    class Ctx:
        ops = cpu_ops
        buffer = staticmethod(lambda name, shape, dtype=None, zero=False: torch.zeros(shape))
    with pytest.raises(ValueError, match="gain"):
        rms.forward(torch.zeros(2, 4), b, Ctx)
    with pytest.raises(ValueError, match="gain already"):
        b.with_gain(torch.ones(4))
    ln = norm.LayerNorm({"size": 4, "eps": 1e-5, "bias": False}, "", env)
    ln.bind({"weight": torch.ones(4)})
    with pytest.raises(ValueError, match="one factor"):
        ln.forward(torch.zeros(2, 4), base.Branch.of_terms([base.Term(torch.zeros(1, 2, 4), scale=1.0), base.Term(torch.zeros(1, 2, 4), scale=2.0)]), Ctx)


def test_plain_mechanisms_against_closed_forms():
    # layer norm: mean off, unit variance, weight
    y = MP.layer_norm(torch.tensor([[1.0, 3.0]]), torch.tensor([2.0, 5.0]), 0.0)
    assert torch.allclose(y, torch.tensor([[-2.0, 5.0]], dtype=F64))
    # rotation of neighbours: a quarter turn of the pair (0, 1) at position 1 with base 1; elements behind `dims` stay
    x = torch.tensor([[[1.0, 5.0, 2.0, 3.0, 9.0]]])
    y = MP.rotate_neighbours(x, torch.tensor([math.pi / 2], dtype=F64), {"base": 1.0, "dims": 4})
    assert torch.allclose(y, torch.tensor([[[-5.0, 1.0, -3.0, 2.0, 9.0]]], dtype=F64), atol=1e-12)
    # scores: the cap first, then the heads' mixture
    s = torch.tensor([[[3.0]], [[-100.0]]], dtype=F64)
    talk = torch.tensor([[0.0, 2.0], [1.0, 1.0]])
    m = MP.mixed_scores(s, 4.0, talk)
    c = [4 * math.tanh(0.75), -4.0]
    assert torch.allclose(m.flatten(), torch.tensor([2 * c[1], c[0] + c[1]], dtype=F64), atol=1e-9)
    # the sink: two equal scores of log 3 and a sink of log 2 leave 3/8 each
    p = MP.sink_softmax(torch.full((1, 1, 2), math.log(3.0), dtype=F64), torch.zeros(1, 2, dtype=torch.bool), torch.tensor([math.log(2.0)], dtype=F64))
    assert torch.allclose(p.flatten(), torch.tensor([0.375, 0.375], dtype=F64))
    # the memory with both gates at zero (i = f = 0): S is the sum, n the sum of keys, m stays 0
    q = torch.ones(3, 1, 1, dtype=F64)
    k = torch.tensor([0.5, 1.0, 2.0], dtype=F64).view(3, 1, 1)
    v = torch.tensor([1.0, 10.0, 100.0], dtype=F64).view(3, 1, 1)
    o, (S, n, mm) = MP.matrix_memory(q, k, v, torch.zeros(3, 1, dtype=F64), torch.zeros(3, 1, dtype=F64))
    assert torch.allclose(o.flatten(), torch.tensor([0.5 / (1 + 1e-6), 10.5 / (1.5 + 1e-6), 210.5 / (3.5 + 1e-6)], dtype=F64))
    assert float(S) == 210.5 and float(n) == 3.5 and float(mm) == 0.0
    # the maximum: an input gate of log 8 after a start at m = 0 sets m = log 8, and the stored S is the true one over 8
    o, (S, n, mm) = MP.matrix_memory(q[:1], k[:1], v[:1], torch.full((1, 1), math.log(8.0), dtype=F64), torch.zeros(1, 1, dtype=F64))
    assert abs(float(mm) - math.log(8.0)) < 1e-12 and abs(float(S) - 0.5) < 1e-12 and abs(float(o) - 0.5 / (0.5 + 1e-6)) < 1e-12
    # the maximum starts at 0, not at minus infinity: a closed input gate leaves m' = f + m
    _, (_, _, mm) = MP.matrix_memory(q[:1], k[:1], v[:1], torch.full((1, 1), -9.0, dtype=F64), torch.full((1, 1), -2.0, dtype=F64))
    assert float(mm) == -2.0
    # router: the largest sigmoids as they are; the weight is on the expert's input
    c, sc = MP.route(torch.tensor([[0.0, 2.0, 1.0]]), torch.eye(3), 2)
    assert c.tolist() == [[1, 2]] and torch.allclose(sc[0], torch.sigmoid(torch.tensor([2.0, 1.0], dtype=F64)))
    w = {"router": torch.eye(1), "e0.gate": torch.ones(1, 1), "e0.up": torch.ones(1, 1), "e0.down": torch.ones(1, 1)}
    got = MP.mixture(torch.tensor([[6.0]]), w, "", {"router": {"experts": 1, "top": 1}, "expert": {"ff": 1, "limit": 2.0}})
    assert abs(float(got) - 2.0 / (1 + math.exp(-3.404)) * 3.0) < 1e-12            # both clamped at 2
    got = MP.mixture(torch.tensor([[-6.0]]), w, "", {"router": {"experts": 1, "top": 1}, "expert": {"ff": 1, "limit": 2.0}})
    z = -6.0 / (1 + math.exp(6.0))                                                 # sigmoid(-6) * -6: nothing is clamped
    assert abs(float(got) - z / (1 + math.exp(-1.702 * z)) * (z + 1)) < 1e-12
    # the run order of a loop
    assert MP.run_order({"layers": [0] * 3, "loop": {"start": 1, "stop": 2, "times": 3}}) == [(0, False), (1, False), (1, True), (1, True), (2, False)]


@pytest.mark.parametrize("name", list(MM.CONFIGS))
def test_engine_host_logic_on_stand_ins(llogos, tmp_path, name):
    """Whole prompts, portions down to two tokens, a token decoded alone, unequal batches and slots used again give the plain
    model's logits when the kernels are the CPU stand-ins."""
    cfg = MM.CONFIGS[name]
    w = MM.write_model(llogos, str(tmp_path), cfg, seed=5)
    wf = {k: v.float() for k, v in w.items()}
    model = llogos.weights.load_model(str(tmp_path), dtype=torch.float32, device="cpu", ops=cpu_ops)
    eng = llogos.engine.Engine(model, max_tokens=64 * 12, n_slots=3, use_graphs=False)
    g = torch.Generator().manual_seed(3)
    seqs = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (1, 25, 68, 9)]
    refs = [MP.forward(wf, cfg, s) for s in seqs]

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


def test_cost_model_counts_the_loop_the_chosen_experts_and_no_pairs_for_a_memory(llogos):
    import importlib
    measure = importlib.import_module("daisi-llogos_b200.measure")
    cfg = MM.CONFIGS["mixed"]
    model = llogos.weights.build_model(cfg, dtype=torch.bfloat16, device="cpu", ops=cpu_ops)
    costs = measure.model_costs(model)
    d, pairs, stored, active = cfg["width"], 0, 0, 0
    for i, _ in MP.run_order(cfg):
        lay = cfg["layers"][i]
        m = lay["mixer"]
        h, dq, dv = m["heads"], m["dim"], m["vdim"]
        if lay["type"] == "mlstm":
            n = d * h * (2 * dq + 2 * dv + 2) + d * h * dv
        elif lay["type"] == "latent_attention":
            r = m["kv_rank"]
            n = d * h * dq + d * r + r * h * (dq + dv) + d * h + d * h * dv
            pairs += 2 * h * 2 * r
        else:
            n = d * h * dq + d * m["kv_heads"] * (dq + dv) + d * h + d * h * dv
            pairs += 2 * h * (dq + dv)
        ml = lay["mlp"]
        e = 0 if not ml else d * ml["router"]["experts"] + 3 * d * ((ml.get("shared") or {}).get("ff", 0))
        x = 0 if not ml else 3 * d * ml["expert"]["ff"]
        stored += n + e + (0 if not ml else ml["router"]["experts"] * x)
        active += n + e + (0 if not ml else ml["router"]["top"] * x)
    assert (costs.matrix_params, costs.active_params) == (stored, active)
    assert len(costs.kv_units) == 5 and costs.kv_units[0] == (2 * (16 + 24) * 2, 0) and costs.kv_units[1] == (32 * 2, 0)
    lat_vd = sum(1 for i, _ in MP.run_order(cfg) if cfg["layers"][i]["type"] == "latent_attention")
    assert lat_vd == 3 and costs.attn_flops_per_pair == pairs


def test_fixed_size_state_refuses_a_rollback(llogos, tmp_path):
    cfg = MM.CONFIGS["odd"]
    MM.write_model(llogos, str(tmp_path), cfg, seed=1)
    model = llogos.weights.load_model(str(tmp_path), dtype=torch.float32, device="cpu", ops=cpu_ops)
    eng = llogos.engine.Engine(model, max_tokens=128, n_slots=2, use_graphs=False)
    slot = eng.open()
    eng.step([(slot, [1, 2, 3])])
    with pytest.raises(llogos.engine.StepError, match="rolled back"):
        eng.truncate(slot, 1)
