"""Parunex without a GPU: its configuration, what it declares, the plain implementation's own consistency, and the host-side logic
(parts, block, values handed along the depth, states and pages side by side, step function) on the CPU with plain PyTorch functions
standing in for the kernels, in every cutting, against the plain implementation."""

from __future__ import annotations

import copy
import math
import random

import pytest
import torch

import helpers
import parunex_helpers as ph
import plain_ops
import plain_parunex as plain

F64 = torch.float64


def test_configuration_reads_every_size_and_round_trips():
    import miniserve_b200  # noqa: F401
    from miniserve_b200.config import ParunexConfig, resolve_architecture
    from miniserve_b200.parts import DecoderModel, PagedKVNeed, StateNeed

    for name, raw in ph.CONFIGS.items():
        architecture = resolve_architecture(raw)
        config = architecture.config_class.from_dict(raw)
        assert isinstance(config, ParunexConfig) and config.to_dict() == raw
        spec = architecture.build_spec(config)
        assert spec.output_name == "head" and spec.embedding_scale == raw["embedding"]["scale"]
        model = DecoderModel(spec, torch.float32, "cpu")
        names = {s.name: s for s in model.param_specs()}
        width, kept = raw["width"], False
        for index, (entry, plan) in enumerate(zip(raw["layers"], model.run_caches)):
            p, m = f"l{index}.", entry["mixer"]
            need = model.cache_groups[plan.group].need
            assert names[p + "norm1.alpha"].shape == () and names[p + "norm1.b"].shape == names[p + "norm1"].shape == (width,)
            if entry["type"] == "attention":
                assert need == PagedKVNeed(m["kv_heads"], m["dim"], None, None if m["vdim"] == m["dim"] else m["vdim"])
                assert names[p + "mix.q.b"].shape == (m["heads"] * m["dim"],) and names[p + "mix.v.b"].shape == (m["kv_heads"] * m["vdim"],)
                assert names[p + "mix.g"].shape == (m["heads"], width) and names[p + "mix.sink"].shape == (m["heads"],)
                assert p + "mix.o.b" not in names
                # the first layer that mixes gives its values and has no share of its own
                assert (p + "mix.vmix" in names) == (m["v_mix"] and kept) and (p + "mix.vmix" in spec.optional_names) == (p + "mix.vmix" not in names)
                kept = kept or m["v_mix"]
            else:
                assert need == StateNeed((m["heads"] * m["dim"] * m["vdim"],), torch.float32)
                assert names[p + "mix.a1"].shape == (m["rank"], width) and names[p + "mix.a2"].shape == (m["heads"] * m["dim"], m["rank"])
                assert names[p + "mix.a1"].kind == "matrix_f32" and names[p + "mix.norm"].shape == (m["vdim"],)
            assert (p + "norm2.alpha" in names) == (entry["mlp"] is not None)
            if entry["mlp"] and entry["mlp"]["kind"] == "moe":
                assert names[p + "mlp.router"].kind == "matrix_f32" and p + "mlp.router.b" not in names
    bare = copy.deepcopy(ph.PARUNEX_A)
    del bare["layers"][0]["mlp"]["router"]["groups"], bare["layers"][0]["mixer"]["softcap"], bare["layers"][0]["mixer"]["v_mix"]
    config = ParunexConfig.from_dict(bare)
    assert (config.layers[0].mlp.group_count, config.layers[0].mixer.softcap, config.layers[0].mixer.v_mix) == (1, None, False)
    bare["layers"][0]["mixer"].update(rot=None, v_mix=None, softcap=None)
    bare["layers"][0]["mlp"]["router"]["groups"] = None
    config = ParunexConfig.from_dict(bare)
    assert (config.layers[0].mixer.rot.dims, config.layers[0].mixer.v_mix, config.layers[0].mlp.group_keep) == (0, False, 1)


def test_the_decays_inner_size_comes_from_the_checkpoint(tmp_path):
    import miniserve_b200  # noqa: F401
    from miniserve_b200.config import load_model_config

    folder = ph.make_folder(tmp_path, "a", seed=1)
    architecture, config = load_model_config(folder)
    assert [layer.mixer.rank for layer in config.layers if layer.type == "gla"] == [5, 9]
    unknown = copy.deepcopy(ph.PARUNEX_A)
    for entry in unknown["layers"]:
        entry["mixer"].pop("rank", None)
    with pytest.raises(ValueError, match="inner size"):
        architecture.build_spec(architecture.config_class.from_dict(unknown))


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][1].__setitem__("type", "hyena"), "not implemented"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("heads", 7), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 18), "exceeds the head size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 5), "odd"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].__setitem__("factor", 0), "factor"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].__delitem__("low"), "low"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("softcap", -1.0), "softcap"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("vdim", 10), "cannot be mixed"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("tau", 0), "tau"),
    (lambda c: c["layers"][1]["mlp"].__setitem__("kind", "sparse"), "not implemented"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 5), "kept groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("count", 4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].__delitem__("scale"), "scale"),
    (lambda c: c["embedding"].__delitem__("scale"), "scale"),
    (lambda c: c["norm"].__setitem__("eps", 0.0), "positive"),
])
def test_configuration_refuses_what_it_cannot_run(change, message):
    import miniserve_b200  # noqa: F401
    from miniserve_b200.config import resolve_architecture

    raw = copy.deepcopy(ph.PARUNEX_A)
    change(raw)
    with pytest.raises(ValueError, match=message):
        resolve_architecture(raw).config_class.from_dict(raw)


def test_parts_refuse_what_they_do_not_implement():
    import miniserve_b200  # noqa: F401
    from miniserve_b200.parts import BLOCKS, FEED_FORWARDS, MIXERS, POSITIONS, PartSpec

    base = dict(hidden_size=32, num_heads=2, num_kv_heads=1, head_dim=8, qk_norm=False, eps=1e-6, position=PartSpec("none"), prefix="")
    for args in (dict(value_mix="borrow"), dict(value_mix="mix", conv_taps=3), dict(value_mix="keep", own_kv=False), dict(bias="k")):
        with pytest.raises(ValueError):
            MIXERS.build(PartSpec("attention", dict(base, **args)))
    with pytest.raises(ValueError, match="bias of the scores"):
        MIXERS.build(PartSpec("attention", dict(base, sink=True, score_bias_slopes=[0.1, 0.2])))
    with pytest.raises(ValueError, match="scaling"):
        POSITIONS.build(PartSpec("rope", dict(head_dim=8, theta=100.0, scaling=dict(factor=2.0, low=1.0))))
    with pytest.raises(ValueError, match="tau"):
        MIXERS.build(PartSpec("gated_linear_attention", dict(prefix="", hidden_size=8, heads=1, head_dim=4, value_dim=4, rank=2, tau=0.0, eps=1e-6)))
    experts = dict(prefix="", hidden_size=8, experts=4, top=2, expert_size=4, router_bias=False, activation="silu_glu")
    for args in (dict(scoring="sigmoid", group_score="median"), dict(normalize=0.0), dict(weight_scale=2.0)):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build(PartSpec("routed_experts", dict(experts, **args)))
    with pytest.raises(ValueError, match="biases"):
        FEED_FORWARDS.build(PartSpec("gated_mlp", dict(prefix="", hidden_size=8, intermediate_size=8, activation="gelu_tanh", bias=True)))
    with pytest.raises(ValueError, match="neither"):
        BLOCKS.build(PartSpec("pre_norm"), mixer=object(), feed_forward=None, mixer_norm=object(), feed_forward_norm=object())


def test_plain_mechanisms_one_by_one():
    """The oracle on hand-made numbers: the norm, the three kinds of wavelengths, the rotation's pairs, the cap, a sink's share, mixed
    values, the decay's power, the recurrence against its unrolled sum, the ranking of groups, the weights' sum."""
    torch.manual_seed(0)
    x = torch.tensor([[0.5, -2.0]], dtype=F64)
    y = plain.dynamic_tanh(x, 0.7, torch.tensor([1.5, -1.0], dtype=F64), torch.tensor([0.1, 0.2], dtype=F64))
    assert y[0].tolist() == pytest.approx([1.5 * math.tanh(0.35) + 0.1, -math.tanh(-1.4) + 0.2])
    plain_f = plain.frequencies(dict(base=10000.0, dims=8))
    assert plain_f == pytest.approx([1.0, 0.1, 0.01, 0.001])
    scaled = plain.frequencies(dict(base=10000.0, dims=8, scaling=dict(factor=4.0, low=1.0, high=4.0, original=200)))
    # wavelengths 6.3, 62.8, 628.3, 6283.2 against original / high = 50 and original / low = 200
    s = (200 / (2 * math.pi / 0.1) - 1.0) / 3.0
    assert scaled == pytest.approx([1.0, (1 - s) * 0.1 / 4 + s * 0.1, 0.01 / 4, 0.001 / 4])
    v = torch.randn(5, 2, 8, dtype=F64)
    turned = plain.rotate_halves(v, dict(base=50.0, dims=4))
    assert torch.allclose(turned[..., 4:], v[..., 4:]) and torch.allclose(turned[0], v[0])
    a = 3 * 50.0 ** (-2.0 / 4)
    assert torch.allclose(turned[3, :, 1], v[3, :, 1] * math.cos(a) - v[3, :, 3] * math.sin(a))
    assert torch.allclose(turned[3, :, 3], v[3, :, 3] * math.cos(a) + v[3, :, 1] * math.sin(a))
    assert plain.capped(torch.tensor([7.0], dtype=F64), 5.0).item() == pytest.approx(5 * math.tanh(1.4)) and plain.capped(3.0, None) == 3.0
    p = plain.softmax_rows(torch.tensor([0.3, -1.0], dtype=F64), 1.2)
    assert float(p.sum()) == pytest.approx(1 - math.exp(1.2) / (math.exp(0.3) + math.exp(-1.0) + math.exp(1.2)))
    assert plain.mixed_values(1.0, None, 0.3) == 1.0 and plain.mixed_values(1.0, 2.0, 0.25) == 1.25
    z = torch.tensor([1.3], dtype=F64)
    w = {"x.a1": torch.eye(1, dtype=F64), "x.a2": torch.eye(1, dtype=F64), "x.a2.b": torch.tensor([0.4], dtype=F64)}
    decay = plain.key_decays(z[None], w, "x.", dict(tau=4.0, heads=1, dim=1))
    assert decay.item() == pytest.approx((1 / (1 + math.exp(-1.7))) ** 0.25)
    # the recurrence is sum_j (q_t prod_(i = j + 1 .. t) a_i) . k_j v_j
    T, width, m = 7, 6, ph.gla(2, 3, 4, 2.0, 5)["mixer"]
    h = torch.randn(T, width, dtype=F64)
    shapes = {"q": (6, width), "k": (6, width), "v": (8, width), "g": (8, width), "o": (8, 8), "norm": (4,), "a1": (5, width), "a2": (6, 5), "a2.b": (6,)}
    w = {"x." + k: torch.randn(s, dtype=F64) for k, s in shapes.items()}
    w["x.o"] = torch.eye(8, dtype=F64)
    got = plain.gated_linear_attention(h, w, "x.", m, 1e-6).view(T, 2, 4)
    decay = plain.key_decays(h, w, "x.", m)
    q, k, v = ((h @ w["x." + n].T).view(T, 2, -1) for n in "qkv")
    t = 5
    o = sum(((q[t] * 3 ** -0.5 * decay[j + 1:t + 1].prod(dim=0) * k[j]).sum(-1, keepdim=True) * v[j]) for j in range(t + 1))
    gate = (h @ w["x.g"].T).view(T, 2, 4)[t]
    assert torch.allclose(got[t], plain.rms_norm(o, w["x.norm"], 1e-6) * gate * torch.sigmoid(gate))
    # experts 0 .. 5 in groups of two: the group with the single best score (0) loses against two good ones
    scores = torch.tensor([0.9, 0.1, 0.6, 0.55, 0.58, 0.5], dtype=F64)
    assert plain.chosen_experts(scores, dict(experts=6, top=2, groups=dict(count=3, keep=1))) == [2, 3]
    assert plain.chosen_experts(scores, dict(experts=6, top=3, groups=dict(count=3, keep=2))) == [2, 4, 3]
    assert plain.chosen_experts(scores, dict(experts=6, top=2, groups=None)) == [0, 2]
    assert plain.chosen_experts(scores, dict(experts=6, top=2, groups=dict(count=6, keep=3))) == [0, 2]      # (groups of one)
    eye = torch.eye(2, dtype=F64)
    w = {"m.router": torch.tensor([[2.0, 0.0], [0.0, 1.0], [-5.0, -5.0]], dtype=F64)}
    for e in range(3):
        w.update({f"m.e{e}.gate": (e + 1) * eye, f"m.e{e}.up": eye, f"m.e{e}.down": eye})
    h = torch.tensor([[0.5, 0.8]], dtype=F64)
    out = plain.mixture(h, w, "m.", dict(router=dict(experts=3, top=2, scale=2.0, groups=None)))
    s0, s1 = 1 / (1 + math.exp(-1.0)), 1 / (1 + math.exp(-0.8))
    want = sum(2.0 * s / (s0 + s1) * plain.silu((e + 1) * h[0]) * h[0] for e, s in ((0, s0), (1, s1)))
    assert torch.allclose(out[0], want)


def test_attention_depends_on_every_earlier_token_and_on_the_first_layers_values():
    torch.manual_seed(1)
    T, width = 12, 10
    m = ph.attention(4, 2, 6, 4, 0.4, ph.rot(100.0, 4), 3.0)["mixer"]
    shapes = {"q": (24, width), "k": (12, width), "v": (8, width), "g": (4, width), "o": (width, 16), "sink": (4,), "q.b": (24,), "k.b": (12,), "v.b": (8,)}
    w = {"x." + k: 0.5 * torch.randn(s, dtype=F64) for k, s in shapes.items()}
    w["x.vmix"] = torch.tensor(0.3, dtype=F64)
    h = torch.randn(T, width, dtype=F64)
    shared: dict = {}
    whole = plain.attention(h, w, "x.", m, 1e-6, shared)
    changed = h.clone()
    changed[4] += 1.0
    after = plain.attention(changed, w, "x.", m, 1e-6, {})
    assert torch.allclose(after[:4], whole[:4]) and all(not torch.allclose(after[t], whole[t], atol=1e-9) for t in range(4, T))
    given = torch.randn(T, 8, dtype=F64)
    mixed = plain.attention(h, w, "x.", m, 1e-6, dict(first_values=given))
    assert not torch.allclose(mixed, whole, atol=1e-3)
    # an output is linear in the values: the mix of the two outputs
    alone = plain.attention(h, dict(w, **{"x.vmix": torch.tensor(1.0, dtype=F64)}), "x.", m, 1e-6, dict(first_values=given))
    assert torch.allclose(mixed, 0.7 * whole + 0.3 * alone)


def test_frequencies_of_the_position_part():
    import miniserve_b200  # noqa: F401
    from miniserve_b200.parts.position import RotaryPosition

    for scaling in (None, (4.0, 1.0, 4.0, 64), (2.0, 2.0, 5.0, 40), (8.0, 1.0, 2.0, 1000)):
        rot = ph.rot(500.0, 12, scaling)
        part = RotaryPosition(head_dim=16, theta=500.0, rotary_dim=12, scaling=rot.get("scaling"), frequencies="float64")
        want = torch.tensor(plain.frequencies(rot), dtype=F64)
        assert torch.equal(part.inv_freq("cpu"), want.to(torch.float32)) and part.magnitude == 1.0


@pytest.fixture
def cpu_runtime(monkeypatch, tmp_path):
    import miniserve_b200  # noqa: F401
    from miniserve_b200.config import EngineConfig
    from miniserve_b200.engine import runtime as runtime_module

    plain_ops.install(monkeypatch)
    monkeypatch.setattr(runtime_module, "require_device", lambda device: torch.device("cpu"))
    monkeypatch.setattr(runtime_module.kernels, "library", lambda: None)
    monkeypatch.setattr(torch.cuda, "set_device", lambda device: None)

    def build(name, num_pages, page_size, max_seqs=4, config=None):
        folder = ph.make_folder(tmp_path, name, seed=2, config=config)
        runtime = runtime_module.build_runtime(folder, EngineConfig(
            dtype="float32", kv_block_size=page_size, num_kv_blocks=num_pages, max_num_seqs=max_seqs,
            enable_prefix_cache=False, device="cpu", decode_execution="eager"))
        return folder, runtime
    return build


def run_and_compare(cpu_runtime, name, page_size, cutting, config=None):
    from miniserve_b200.trace import TraceSession

    vocab = (config or ph.CONFIGS[name])["vocab"]
    requests = {f"r{i}": helpers.random_tokens(vocab, n, seed=20 + i) for i, n in enumerate((1, 6, 17, 30, 41))}
    steps = {"whole": helpers.cut_whole, "tail": lambda r: helpers.cut_decode_tail(r, 9),
             "portions": helpers.cut_portions, "mixed": helpers.cut_mixed}[cutting](requests)
    pages = (helpers.max_live_tokens(steps, granule=page_size * 2) + page_size - 1) // page_size
    folder, runtime = cpu_runtime(name, pages, page_size, config=config)
    session, outputs = TraceSession(runtime), {}
    for record in steps:
        outputs[record["step"]] = session.run(record).double()
        runtime.manager.check_invariants()
    got = helpers.collect(steps, outputs)
    config, weights = ph.load_folder(folder)
    for rid, tokens in requests.items():
        expected = plain.forward(tokens, weights, config)
        assert sorted(got[rid]) == list(range(len(tokens)))
        bound = 2e-5 * max(1.0, float(expected.abs().max()))
        for position, row in got[rid].items():
            assert float((row - expected[position]).abs().max()) <= bound, (rid, position)
    assert not runtime.manager.requests
    assert all(a.free_count == a.num_pages for a in runtime.manager.allocators)


@pytest.mark.parametrize("name,page_size", [("a", 8), ("b", 4), ("d", 16), ("e", 8)])
@pytest.mark.parametrize("cutting", ["whole", "tail", "portions", "mixed"])
def test_cuttings_match_plain_on_cpu(cpu_runtime, name, page_size, cutting):
    run_and_compare(cpu_runtime, name, page_size, cutting)


@pytest.mark.parametrize("seed", range(8))
def test_random_configurations_on_cpu(cpu_runtime, seed):
    rng = random.Random(seed)
    config = ph.random_config(rng)
    run_and_compare(cpu_runtime, f"random{seed}", rng.choice([4, 8, 16]), rng.choice(["tail", "portions", "mixed"]), config)


def test_every_tensor_moves_the_logits(tmp_path):
    """The shaped weights of the test configurations leave no tensor without effect (else a fault in it would not show): changing one
    alone changes the plain implementation's logits."""
    folder = ph.make_folder(tmp_path, "a", seed=3)
    config, weights = ph.load_folder(folder)
    tokens = helpers.random_tokens(config["vocab"], 24, seed=1)
    base = plain.forward(tokens, weights, config)
    for name, value in weights.items():
        if ".mlp.e" in name:
            continue                    # (an expert that no token of these chose has none)
        moved = plain.forward(tokens, dict(weights, **{name: value * 1.2 + 0.05}), config)
        assert float((moved - base).abs().max()) > 1e-3 * float(base.abs().max()), name
    for change in (lambda c: c["layers"][0]["mixer"].__setitem__("softcap", 10.0),
                   lambda c: c["layers"][2]["mixer"].__setitem__("v_mix", False),
                   lambda c: c["layers"][0]["mixer"]["rot"].pop("scaling"),
                   lambda c: c["layers"][1]["mixer"].__setitem__("tau", 8.0),
                   lambda c: c["layers"][3]["mlp"]["router"].__setitem__("scale", 1.0),
                   lambda c: c["layers"][3]["mlp"]["router"].__setitem__("groups", dict(count=1, keep=1))):
        other = copy.deepcopy(config)
        change(other)
        assert float((plain.forward(tokens, weights, other) - base).abs().max()) > 1e-3 * float(base.abs().max())


def test_a_checkpoint_may_carry_tensors_that_nothing_reads(cpu_runtime):
    """Norms of a feed-forward that a layer does not have and the share of the layer that gives its values are accepted and not
    loaded; any other unknown name is refused."""
    from miniserve_b200.weights.loader import WeightLoadError
    from safetensors.torch import load_file, save_file

    folder, _ = cpu_runtime("d", 8, 8)
    tensors = load_file(str(folder / "model.safetensors"))
    extra = {"l2.norm2": torch.ones(44), "l2.norm2.b": torch.ones(44), "l2.norm2.alpha": torch.tensor(1.0), "l0.mix.vmix": torch.tensor(0.5)}
    save_file({**tensors, **extra}, str(folder / "model.safetensors"))
    cpu_runtime("d", 8, 8)
    for unknown in ({"l0.mix.o.b": torch.ones(44)}, {"l0.mlp.gate.b": torch.ones(30)}):
        save_file({**tensors, **unknown}, str(folder / "model.safetensors"))
        with pytest.raises(WeightLoadError, match="unexpected"):
            cpu_runtime("d", 8, 8)
