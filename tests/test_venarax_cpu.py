"""Venarax without a GPU: its configuration, what it declares, the plain implementation's own consistency, and the host-side logic
(parts, block, transition, windowed and full caches side by side, a cache per pass, step function) on the CPU with plain PyTorch
functions standing in for the kernels, in every cutting, against the plain implementation."""

from __future__ import annotations

import copy
import math
import random

import pytest
import torch

import helpers
import plain_ops
import plain_venarax as plain
import venarax_helpers as vh


def test_configuration_reads_every_size_and_round_trips():
    import miniserve_b200  # noqa: F401
    from miniserve_b200.config import VenaraxConfig, resolve_architecture
    from miniserve_b200.parts import DecoderModel, PagedKVNeed, PagedLatentNeed

    for name, raw in vh.CONFIGS.items():
        architecture = resolve_architecture(raw)
        config = architecture.config_class.from_dict(raw)
        assert isinstance(config, VenaraxConfig) and config.to_dict() == raw
        spec = architecture.build_spec(config)
        assert spec.output_name == "head" and spec.embedding_scale == 1.0
        assert [(run.layer, None if run.enters is None else run.enters[1]) for run in spec.order] == plain.layer_order(raw)
        model = DecoderModel(spec, torch.float32, "cpu")
        names = {s.name: s for s in model.param_specs()}
        width = raw["width"]
        caches = set()
        for run, plan in zip(spec.order, model.run_caches):
            entry, p = raw["layers"][run.layer], f"l{run.layer}.mix."
            m = entry["mixer"]
            need = model.cache_groups[plan.group].need
            if entry["type"] == "latent_attention":
                assert need == PagedLatentNeed(m["kv_rank"], m["rot_dim"], m["mask"]["size"])
                assert names[p + "g"].shape == (m["heads"] * m["vdim"], width) and names[p + "dkv"].shape == (m["kv_rank"] + m["rot_dim"], width)
                assert names[p + "uk"].shape == (m["heads"] * m["dim"], m["kv_rank"]) and names[p + "dkv.norm"].shape == (m["kv_rank"],)
            else:
                assert need == PagedKVNeed(m["kv_heads"], m["dim"], None, None if m["vdim"] == m["dim"] else m["vdim"])
                assert names[p + "sink"].shape == (m["heads"],) and names[p + "q.norm"].shape == (m["heads"] * m["dim"],)
                assert names[p + "k.norm"].shape == (m["kv_heads"] * m["dim"],)
            caches.add((plan.group, plan.slot))
            assert (f"l{run.layer}.norm2.b" in names) == (entry["mlp"] is not None)
        assert len(caches) == len(spec.order)             # every run of a layer, repeated or not, keeps a cache of its own
        if raw["loop"]:
            assert names["loop.in"].shape == (width, 2 * width) and names["loop.step"].shape == (raw["loop"]["times"], width)
        else:
            assert "loop.in" not in names


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][1].__setitem__("type", "hyena"), "not implemented"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("heads", 7), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 6), "exceeds the rotated part"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 3), "odd"),
    (lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0), "positive"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].__setitem__("every", 0), "every"),
    (lambda c: c["layers"][2]["mlp"].__setitem__("kind", "sparse"), "not implemented"),
    (lambda c: c["layers"][2]["mlp"].__delitem__("limit"), "limit"),
    (lambda c: c["loop"].__setitem__("stop", 9), "loop"),
    (lambda c: c["loop"].__setitem__("times", 0), "times"),
    (lambda c: c["norm"].__setitem__("eps", 0.0), "positive"),
])
def test_configuration_refuses_what_it_cannot_run(change, message):
    import miniserve_b200  # noqa: F401
    from miniserve_b200.config import resolve_architecture

    raw = copy.deepcopy(vh.VENARAX_A)
    change(raw)
    with pytest.raises(ValueError, match=message):
        resolve_architecture(raw).config_class.from_dict(raw)


def test_plain_mechanisms_one_by_one():
    """The oracle on hand-made numbers: norms, the rotation's pairs, the window's edge, the temperature's steps, a sink's share,
    the activation's clamps, the order of passes."""
    torch.manual_seed(0)
    x = torch.randn(5, 8, dtype=plain.F64)
    one, zero = torch.ones(8, dtype=plain.F64), torch.zeros(8, dtype=plain.F64)
    y = plain.layer_norm(x, one, zero, 1e-9)
    assert torch.allclose(y.mean(-1), torch.zeros(5, dtype=plain.F64), atol=1e-12) and torch.allclose(y.pow(2).mean(-1), torch.ones(5, dtype=plain.F64), atol=1e-6)
    assert torch.allclose(plain.layer_norm(x + 3.0, one, zero, 1e-9), y)              # (an RMS norm would change)
    assert torch.allclose(plain.layer_norm(x, 2 * one, 5 + zero, 1e-9), 2 * y + 5)
    v = torch.randn(7, 2, 8, dtype=plain.F64)
    turned = plain.rotate_pairs(v, dict(base=50.0, dims=4))
    assert torch.allclose(turned[..., 4:], v[..., 4:]) and torch.allclose(turned[0], v[0])
    a = 3 * 50.0 ** (-2.0 / 4)
    assert torch.allclose(turned[3, :, 2], v[3, :, 2] * math.cos(a) - v[3, :, 3] * math.sin(a))
    assert torch.allclose(turned[3, :, 3], v[3, :, 3] * math.cos(a) + v[3, :, 2] * math.sin(a))
    temp = dict(coef=0.5, every=4)
    assert [plain.query_temperature(p, temp) for p in (0, 2)] == [1.0, 1.0]           # floor((p + 1) / 4) is 0 up to p = 2
    assert plain.query_temperature(3, temp) == pytest.approx(1 + 0.5 * math.log(2)) == plain.query_temperature(6, temp)
    assert plain.query_temperature(7, temp) == pytest.approx(1 + 0.5 * math.log(3))
    p = plain.softmax_rows(torch.tensor([0.3, -1.0], dtype=plain.F64), 1.2)
    assert float(p.sum()) == pytest.approx(1 - math.exp(1.2) / (math.exp(0.3) + math.exp(-1.0) + math.exp(1.2)))
    w = {"m.gate": torch.eye(2, dtype=plain.F64), "m.up": torch.eye(2, dtype=plain.F64), "m.down": torch.eye(2, dtype=plain.F64)}
    g, u = 0.5, -0.5
    out = plain.feed_forward(torch.tensor([[9.0, -9.0]], dtype=plain.F64), w, "m.", dict(limit=0.5))
    assert float(out[0, 0]) == pytest.approx(g / (1 + math.exp(-1.702 * g)) * 1.5)
    assert float(out[0, 1]) == pytest.approx(-9.0 / (1 + math.exp(1.702 * 9)) * (u + 1))       # the gate has no lower clamp
    # a token's output depends on the window's first token and not on the one before it; the sink attention on every token
    width, T = 12, 20
    h = torch.randn(T, width, dtype=plain.F64)
    m = vh.latent(2, 4, 2, 3, 5, 0.5, 100.0, 6)["mixer"]
    shapes = {"q": (12, width), "dkv": (7, width), "dkv.norm": (5,), "uk": (8, 5), "uv": (6, 5), "g": (6, width), "o": (width, 6)}
    wl = {"x." + k: 0.4 * torch.randn(s, dtype=plain.F64) for k, s in shapes.items()}
    whole = plain.latent_attention(h, wl, "x.", m, 1e-6)
    changed = h.clone()
    changed[8] += 1.0
    after = plain.latent_attention(changed, wl, "x.", m, 1e-6)
    assert torch.allclose(after[:8], whole[:8]) and torch.allclose(after[14:], whole[14:])
    assert all(not torch.allclose(after[t], whole[t], atol=1e-7) for t in range(8, 14))
    m = vh.sink(2, 1, 4, 3, 0.5, 0.3, 5)["mixer"]
    shapes = {"q": (8, width), "k": (4, width), "v": (3, width), "q.norm": (8,), "k.norm": (4,), "sink": (2,), "o": (width, 6)}
    wa = {"x." + k: 0.4 * torch.randn(s, dtype=plain.F64) for k, s in shapes.items()}
    whole, after = plain.sink_attention(h, wa, "x.", m, 1e-6), plain.sink_attention(changed, wa, "x.", m, 1e-6)
    assert torch.allclose(after[:8], whole[:8]) and all(not torch.allclose(after[t], whole[t], atol=1e-9) for t in range(8, T))
    assert plain.layer_order(dict(layers=[0] * 5, loop=dict(start=1, stop=3, times=2))) == [
        (0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None), (4, None)]


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
        folder = vh.make_folder(tmp_path, name, seed=2, config=config)
        runtime = runtime_module.build_runtime(folder, EngineConfig(
            dtype="float32", kv_block_size=page_size, num_kv_blocks=num_pages, max_num_seqs=max_seqs,
            enable_prefix_cache=False, device="cpu", decode_execution="eager"))
        return folder, runtime
    return build


def run_and_compare(cpu_runtime, name, page_size, cutting, config=None):
    from miniserve_b200.trace import TraceSession

    vocab = (config or vh.CONFIGS[name])["vocab"]
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
    config, weights = vh.load_folder(folder)
    for rid, tokens in requests.items():
        expected = plain.forward(tokens, weights, config)
        assert sorted(got[rid]) == list(range(len(tokens)))
        bound = 2e-5 * float(expected.abs().max())
        for position, row in got[rid].items():
            assert float((row - expected[position]).abs().max()) <= bound, (rid, position)
    assert not runtime.manager.requests
    assert all(a.free_count == a.num_pages for a in runtime.manager.allocators)


@pytest.mark.parametrize("name,page_size", [("a", 8), ("b", 4), ("d", 16)])
@pytest.mark.parametrize("cutting", ["whole", "tail", "portions", "mixed"])
def test_cuttings_match_plain_on_cpu(cpu_runtime, name, page_size, cutting):
    run_and_compare(cpu_runtime, name, page_size, cutting)


@pytest.mark.parametrize("seed", range(8))
def test_random_configurations_on_cpu(cpu_runtime, seed):
    rng = random.Random(seed)
    config = vh.random_config(rng)
    run_and_compare(cpu_runtime, f"random{seed}", rng.choice([4, 8, 16]), rng.choice(["tail", "portions", "mixed"]), config)


def test_a_checkpoint_may_carry_norms_and_passes_that_nothing_reads(cpu_runtime, tmp_path):
    """Norms of a feed-forward that a layer does not have and the tensors of a loop that a model does not run are accepted and
    not loaded; any other unknown name is refused."""
    from miniserve_b200.weights.loader import WeightLoadError
    from safetensors.torch import load_file, save_file

    config = copy.deepcopy(vh.VENARAX_D)
    config["layers"][0]["mlp"] = None
    folder, _ = cpu_runtime("unused", 8, 8, config=config)
    tensors = load_file(str(folder / "model.safetensors"))
    extra = {"l0.norm2": torch.ones(44), "l0.norm2.b": torch.ones(44), "loop.in": torch.ones(44, 88), "loop.step": torch.ones(2, 44)}
    save_file({**tensors, **extra}, str(folder / "model.safetensors"))
    cpu_runtime("unused", 8, 8, config=config)
    save_file({**tensors, "l0.mix.sink": torch.ones(3)}, str(folder / "model.safetensors"))
    with pytest.raises(WeightLoadError, match="unexpected"):
        cpu_runtime("unused", 8, 8, config=config)
