"""Parunex on the GPU against the plain implementation (``plain_parunex``) and the plain statements of the kernels (``plain_ops``):
every new or changed kernel alone, both mixers and the feed-forwards alone (fed in portions down to one and two tokens and token by
token through the cache, with keys and writes that stand out far back, pages and slots that are used again), and the whole model
through the engine's own session, scheduler and command line, in float32 and bfloat16, at sizes of its own."""

from __future__ import annotations

import json
import random
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import helpers
import parunex_helpers as ph
import plain_ops
import plain_parunex as plain
from test_parts_gpu import Harness, rand, tol

pytestmark = pytest.mark.gpu
REPO = Path(__file__).resolve().parent.parent
DTYPES = [torch.float32, torch.bfloat16]
F64 = torch.float64


def bound_of(dtype, expected):
    return (1e-5 if dtype in ("float32", torch.float32) else 1.5e-2) * max(1.0, float(expected.abs().max()))


def cpu(tensor):
    return None if tensor is None else tensor.detach().cpu().clone()


def ints(values):
    return torch.tensor(values, dtype=torch.int32).cuda()


def close(got, expected, dtype=torch.float32, scale=None):
    expected = expected.double().cpu()
    return torch.allclose(got.double().cpu(), expected, **tol(dtype, float(expected.abs().max()) if scale is None else scale))


# --------------------------------------------------------------------------- kernels alone


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [1, 44, 96, 1000, 2048, 8200])
@pytest.mark.parametrize("rows", [1, 5, 700])
@pytest.mark.parametrize("pending", ["nothing", "one", "two"])
def test_add_dynamic_tanh_kernel(dtype, hidden, rows, pending):
    """Every kind of pending addition, rows picked out (the stream stays), entries deep in both tails of the tanh and near zero."""
    from miniserve_b200 import kernels

    residual = rand((rows, hidden), torch.float32, 1, 3.0)
    residual[0, 0], residual[-1, -1] = 60.0, -1e-4
    delta = rand((rows, hidden), dtype, 2) if pending != "nothing" else None
    delta2 = rand((rows, hidden), dtype, 3) if pending == "two" else None
    weight, bias = 1 + rand((hidden,), torch.float32, 4, 0.3), rand((hidden,), torch.float32, 5, 0.3)
    for picked in (None, ints([rows - 1, 0])):
        stream, want_stream = residual.clone(), cpu(residual).double()
        n = rows if picked is None else 2
        out, want = torch.empty((n, hidden), dtype=dtype, device="cuda"), torch.empty((n, hidden), dtype=F64)
        kernels.add_dynamic_tanh(stream, delta, -0.7, weight, bias, out, picked, delta2)
        plain_ops.add_dynamic_tanh(want_stream, cpu(delta), -0.7, cpu(weight), cpu(bias), want, cpu(picked), cpu(delta2))
        assert torch.allclose(cpu(stream).double(), want_stream, atol=1e-5) and close(out, want, dtype, 1.0)
        if picked is not None or pending == "nothing":
            assert torch.equal(stream, residual)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(3, 20, 12), (1, 10, 14), (5, 7, 9), (4, 64, 32), (2, 128, 64), (16, 128, 128), (2, 200, 40)])
def test_matrix_scan_with_channel_decays(dtype, heads, dim, vdim):
    """Unequal requests in slots out of order from states that are not zero, one that brings nothing, against the plain walk; the
    same tokens in portions of one and two leave the same rows and states to the bit.  Some channels keep everything for hundreds of
    tokens, some forget at once."""
    from miniserve_b200 import kernels

    lengths, slots, offset = [40, 0, 1, 150], [2, 1, 3, 0], 8
    n = sum(lengths)
    ld = heads * (2 * dim + vdim) + 3
    proj = rand((n, ld), dtype, 1, 0.7)
    cols = (0, heads * dim, 2 * heads * dim)
    decays = torch.sigmoid(rand((n, heads * dim), torch.float32, 2, 2.0) + 2.0)
    decays[:, ::5], decays[:, 3::7] = 1.0 - 1e-4, 1e-6
    states = rand((4, offset + heads * dim * vdim + 1), torch.float32, 3)
    start = states.clone()
    y = torch.zeros((n, heads, vdim), device="cuda")
    starts = torch.tensor([sum(lengths[:i]) for i in range(len(lengths) + 1)], dtype=torch.int32)
    want_states, want = cpu(states).double(), torch.zeros(y.shape, dtype=F64)
    args = dict(q_scale=dim ** -0.5)
    plain_ops.matrix_scan("channel_decay", cpu(proj), cols[0], cpu(proj), cols[1], cpu(proj), cols[2], None, want_states, offset, torch.tensor(slots),
                          starts, max(lengths), heads, heads, dim, vdim, want, channel_decay=cpu(decays), **args)

    def run(rows, spans, into, out):
        kernels.matrix_scan("channel_decay", rows, cols[0], rows, cols[1], rows, cols[2], None, into, offset, ints(slots), ints(spans),
                            max(b - a for a, b in zip(spans[:-1], spans[1:])), heads, heads, dim, vdim, out[0],
                            channel_decay=out[1], **args)

    run(proj, starts.tolist(), states, (y, decays))
    assert close(y, want) and torch.allclose(states.cpu().double(), want_states, atol=2e-5, rtol=2e-5)
    assert torch.equal(states[1], start[1])
    again, at, pieces = start.clone(), [0] * len(lengths), torch.zeros_like(y)
    for step in range(200):
        take = [min(length - a, 1 + (step + i) % 2 if step < 20 else 30) for i, (length, a) in enumerate(zip(lengths, at))]
        if not sum(take):
            break
        rows = torch.cat([torch.arange(int(starts[i]) + at[i], int(starts[i]) + at[i] + t) for i, t in enumerate(take)]).cuda()
        part = torch.zeros((rows.numel(), heads, vdim), device="cuda")
        run(proj[rows].contiguous(), [sum(take[:i]) for i in range(len(take) + 1)], again, (part, decays[rows].contiguous()))
        pieces[rows] = part
        at = [a + t for a, t in zip(at, take)]
    # (lanes a column depend on the launch's size: the order of a column's sum may differ, not what is summed)
    assert at == lengths and torch.allclose(pieces, y, atol=2e-5, rtol=2e-5) and torch.allclose(again, states, atol=2e-5, rtol=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(3, 20, 12), (5, 7, 9), (4, 64, 32), (16, 128, 128), (2, 200, 40)])
@pytest.mark.parametrize("lengths,chunk", [([40, 0, 1, 150], 16), ([33, 32, 31, 64, 65], 32), ([1, 1, 200, 1, 7], 48), ([130], 1), ([5, 2], 100)])
def test_matrix_scan_in_chunks(dtype, heads, dim, vdim, lengths, chunk):
    """Portions of one chunk, of several with a short last one and of exact multiples, beside single tokens and nothing at all, from
    states that are not zero, against the plain walk; what lies around the states' rows stays as it was."""
    from miniserve_b200 import kernels

    n, slots = sum(lengths), list(range(len(lengths)))[::-1]
    offset = 4
    proj = rand((n, heads * (2 * dim + vdim)), dtype, 1, 0.7)
    cols = (0, heads * dim, 2 * heads * dim)
    decays = torch.sigmoid(rand((n, heads * dim), torch.float32, 2, 2.0) + 2.0)
    decays[:, ::5], decays[:, 3::7] = 1.0 - 1e-4, 1e-6
    states = rand((len(lengths) + 1, offset + heads * dim * vdim + 3), torch.float32, 3)
    start = cpu(states)
    y, want = torch.zeros((n, heads, vdim), device="cuda"), torch.zeros((n, heads, vdim), dtype=F64)
    starts = torch.tensor([sum(lengths[:i]) for i in range(len(lengths) + 1)], dtype=torch.int32)
    want_states = cpu(states).double()
    plain_ops.matrix_scan("channel_decay", cpu(proj), cols[0], cpu(proj), cols[1], cpu(proj), cols[2], None, want_states, offset, torch.tensor(slots),
                          starts, max(lengths), heads, heads, dim, vdim, want, q_scale=dim ** -0.5, channel_decay=cpu(decays))
    kernels.matrix_scan("channel_decay", proj, cols[0], proj, cols[1], proj, cols[2], None, states, offset, ints(slots), starts.cuda(), max(lengths),
                        heads, heads, dim, vdim, y, q_scale=dim ** -0.5, channel_decay=decays, chunk=chunk)
    assert close(y, want) and torch.allclose(states.cpu().double(), want_states, atol=2e-5, rtol=2e-5)
    assert torch.equal(states.cpu()[:, :offset], start[:, :offset]) and torch.equal(states.cpu()[:, -3:], start[:, -3:])
    assert torch.equal(states.cpu()[-1], start[-1])


def test_long_portions_are_scanned_in_chunks():
    """What the library chooses: chunks for few long portions, none for many, for short ones and for keys of more than 256 entries."""
    from miniserve_b200 import kernels

    choose = kernels.library().ms_channel_scan_chunk
    assert 64 <= choose(1, 2048, 16, 128, 128) <= 512 and choose(1, 100, 16, 128, 128) == 0 and choose(64, 512, 16, 128, 128) == 0
    assert choose(1, 2048, 16, 300, 128) == 0
    n, heads, dim, vdim = 700, 2, 24, 40
    proj, decays = rand((n, heads * (2 * dim + vdim)), torch.bfloat16, 1), torch.sigmoid(rand((n, heads * dim), torch.float32, 2) + 3.0)
    results = []
    for chunk in (0, None):
        states, y = torch.zeros((1, heads * dim * vdim), device="cuda"), torch.empty((n, heads, vdim), device="cuda")
        kernels.matrix_scan("channel_decay", proj, 0, proj, heads * dim, proj, 2 * heads * dim, None, states, 0, ints([0]), ints([0, n]), n, heads,
                            heads, dim, vdim, y, channel_decay=decays, chunk=chunk)
        results.append((y, states))
    assert choose(1, n, heads, dim, vdim) > 0
    for a, b in zip(*results):
        assert torch.allclose(a, b, atol=1e-4, rtol=1e-5) and float(a.abs().max()) > 1.0


@pytest.mark.parametrize("rank,rows,tau,n", [(1, 12, 1.0, 1), (5, 60, 16.0, 9), (16, 300, 4.0, 70), (64, 2048, 16.0, 33)])
def test_decays_to_a_power(rank, rows, tau, n):
    from miniserve_b200 import kernels

    mid, weight, bias = rand((n, rank + 3), torch.float32, 1, 2.0), rand((rank, rows), torch.float32, 2), rand((rows,), torch.float32, 3, 4.0)
    bias[0], bias[-1] = -200.0, 200.0              # (sigmoids that vanish, or are one)
    out, want = torch.empty((n, rows), device="cuda"), torch.empty((n, rows), dtype=F64)
    kernels.low_rank_expand(mid, 2, weight, out, bias=bias, tau=tau)
    z = cpu(mid).double()[:, 2:2 + rank] @ cpu(weight).double() + cpu(bias).double()
    want = torch.exp(torch.nn.functional.logsigmoid(z) / tau)
    assert torch.allclose(out.cpu().double(), want, atol=1e-6, rtol=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,top,count,keep", [(8, 2, 2, 1), (6, 2, 3, 2), (16, 4, 4, 2), (9, 3, 3, 1), (6, 3, 6, 4), (5, 5, 1, 1), (60, 6, 5, 3), (64, 8, 8, 4)])
@pytest.mark.parametrize("rows", [1, 7, 300])
def test_router_with_groups_by_their_two_best(dtype, experts, top, count, keep, rows):
    """Choices, weights that add up to the scale, and that the other rank of groups would choose otherwise."""
    from miniserve_b200 import kernels

    width = 88
    x, weight = rand((rows, width), dtype, 1), rand((experts, width), torch.float32, 2, 0.3)
    ids, weights = torch.empty((rows, top), dtype=torch.int32, device="cuda"), torch.empty((rows, top), device="cuda")
    kernels.router_topk(x, weight, None, top, ids, weights, scoring="sigmoid", groups=(count, keep), group_score="two_largest",
                        normalize=1e-20, weight_scale=2.5)
    scores = torch.sigmoid(cpu(x).double() @ cpu(weight).double().T)
    router = dict(experts=experts, top=top, groups=dict(count=count, keep=keep))
    want = [plain.chosen_experts(row, router) for row in scores]
    same = [i for i in range(rows) if ids[i].tolist() == want[i]]
    assert len(same) >= rows - 1 - rows // 100                     # (a close call may go either way)
    assert torch.allclose(weights.sum(dim=1).cpu(), torch.full((rows,), 2.5), atol=1e-5)
    for i in same:
        s = scores[i, want[i]]
        assert torch.allclose(weights[i].cpu().double(), 2.5 * s / s.sum(), atol=1e-5)
    if rows == 300 and keep < count < experts:
        kernels.router_topk(x, weight, None, top, ids, weights, scoring="sigmoid", groups=(count, keep))
        assert sum(ids[i].tolist() != want[i] for i in range(rows)) > 5
        for i in range(rows):
            assert torch.allclose(weights[i].cpu().double(), scores[i, ids[i].tolist()], atol=1e-5)      # (neither normalized nor scaled)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 8, 40, 700])
@pytest.mark.parametrize("inner,width", [(64, 96), (512, 256), (30, 44)])
def test_gelu_gated_activation(dtype, rows, inner, width):
    """The fused products' choice for these sizes and every kernel that can carry the activation, called by name."""
    from miniserve_b200 import kernels

    x, gate, up = rand((rows, width), dtype, 1), rand((inner, width), dtype, 2, 0.3), rand((inner, width), dtype, 3, 0.15)
    g, u = cpu(x).double() @ cpu(gate).double().T, cpu(x).double() @ cpu(up).double().T
    want = plain.gelu_tanh(g) * u
    both = torch.cat([g, u], dim=1).to(dtype).cuda()
    out = torch.empty((rows, inner), dtype=dtype, device="cuda")
    kernels.silu_mul(both, out, activation="gelu_tanh")
    assert close(out, want, dtype)
    if inner % 8:
        return
    paired = kernels.interleave_gate_up(gate, up).contiguous()
    runs = [lambda: kernels.gated_up(x, paired, out, activation="gelu_tanh")]
    if dtype == torch.bfloat16:
        if rows <= 8:
            runs.append(lambda: kernels.linear_wide(x, paired, out, gated=True, activation="gelu_tanh"))
        runs += [lambda wide=wide: kernels.linear_pair(x, paired, out, gated=True, wide=wide, activation="gelu_tanh") for wide in (False, True)]
    for run in runs:
        out.zero_()
        run()
        assert close(out, want, dtype)
    kernels.check_device_errors(out.device)
    with pytest.raises(kernels.KernelError):
        kernels.silu_mul(both, out, activation="gelu_tanh", limit=1.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n_q,n_kv,d,dv,rotary", [(4, 2, 16, 24, 12), (3, 3, 7, 9, 4), (8, 2, 64, 64, 64), (2, 1, 128, 48, 32), (5, 5, 6, 10, 0)])
def test_prepare_keeps_and_mixes_values(dtype, n_q, n_kv, d, dv, rotary):
    from miniserve_b200 import kernels

    n, page, pages = 9, 4, 8
    ld = (n_q * d + n_kv * (d + dv) + n_q + 7) // 8 * 8
    proj, bias = rand((n, ld), dtype, 1), rand((ld,), torch.float32, 2)
    positions, slots = ints([0, 1, 2, 3, 5, 6, 200, 4094, 100001]), ints([5, 9, -1, 0, 31, 12, 13, 14, 2])
    table = None
    if rotary:
        table = torch.empty((n, rotary // 2, 2), device="cuda")
        kernels.rope_table(positions, torch.tensor([100.0 ** (-2 * i / rotary) for i in range(rotary // 2)], device="cuda"), table)
    cols = (0, n_q * d, (n_q + n_kv) * d)
    for share in (None, 0.3, -0.25, 1.0, 0.0):
        kept = rand((n, n_kv * dv), dtype, 3, 2.0)
        want_kept = cpu(kept).double()
        k_pool, v_pool = torch.zeros((pages, n_kv, page, d), dtype=dtype).cuda(), torch.zeros((pages, n_kv, page, dv), dtype=dtype).cuda()
        q = torch.empty((n, n_q, d), dtype=dtype).cuda()
        want = [torch.zeros(t.shape, dtype=F64) for t in (q, k_pool, v_pool)]
        kernels.qkv_prepare(proj, *cols, n_q, n_kv, d, dv, slots, None, None, 1e-5, table, rotary, k_pool, v_pool, q, bias=bias, kept_values=kept,
                            mix_share=share)
        plain_ops.qkv_prepare(cpu(proj), *cols, n_q, n_kv, d, dv, cpu(slots), None, None, 1e-5, cpu(table), rotary, want[1], want[2], want[0],
                              bias=cpu(bias), kept_values=want_kept, mix_share=share)
        for got, expected in zip((q, k_pool, v_pool, kept), want + [want_kept]):
            assert close(got, expected, dtype)


def attention_case(dtype, n_q, n_kv, d, dv, page, queries, contexts, seed=0, key_scale=1.0):
    """A batch over scrambled pages: (arguments of kernels.paged_attention up to the context length, the same on the CPU)."""
    requests = len(queries)
    width = (max(contexts) + page - 1) // page
    order = torch.randperm(requests * width + 3, generator=torch.Generator().manual_seed(seed))
    tables = order[:requests * width].view(requests, width).to(torch.int32)
    k_pool, v_pool = rand((requests * width + 3, n_kv, page, d), dtype, seed + 1, key_scale), rand((requests * width + 3, n_kv, page, dv), dtype, seed + 2)
    n = sum(queries)
    q = rand((n, n_q, d), dtype, seed + 3)
    request_of = torch.tensor([r for r, m in enumerate(queries) for _ in range(m)], dtype=torch.int32)
    positions = torch.tensor([contexts[r] - queries[r] + i for r in range(requests) for i in range(queries[r])], dtype=torch.int32)
    starts = [sum(queries[:i]) for i in range(requests + 1)]
    host = [q, k_pool, v_pool, tables, request_of, positions, torch.tensor(starts, dtype=torch.int32), torch.tensor(contexts, dtype=torch.int32)]
    return [t.cuda() for t in host], [t.cpu() for t in host], starts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n_q,n_kv,d,dv,page", [(6, 2, 48, 80, 16), (4, 4, 32, 64, 8), (4, 2, 96, 96, 16), (3, 1, 7, 9, 4), (8, 2, 64, 64, 16),
                                                (16, 4, 128, 128, 64), (4, 4, 32, 32, 16), (8, 1, 128, 48, 16)])
@pytest.mark.parametrize("queries,contexts", [([1, 1, 1], [1, 700, 33]), ([1, 150, 2], [300, 170, 2]), ([200], [200])])
@pytest.mark.parametrize("softcap", [2.0, 30.0])
def test_attention_kernels_with_a_soft_cap(dtype, n_q, n_kv, d, dv, page, queries, contexts, softcap):
    """Every attention kernel (general; tensor cores for any size, for unrolled sizes and, on prompts, tcgen05), single tokens with their
    keys split and prompt portions in one batch, scores from far inside the cap to far beyond it on both sides, beside a learned
    sink and a gate."""
    from miniserve_b200 import kernels

    scores = torch.tensor([[-40.0, 0.0, 1.5, -2.0, 4.0, 3.0][h % 6] for h in range(n_q)])
    scale = 3.0 * d ** -0.5
    args, host, starts = attention_case(dtype, n_q, n_kv, d, dv, page, queries, contexts)
    gate = rand((sum(queries), n_q + 8), dtype, 9)
    for extra, plain_extra in ((dict(), dict()), (dict(sink=scores.cuda(), gate=gate, gate_col=3), dict(sink=scores, gate=gate.cpu(), gate_col=3))):
        out = torch.empty((sum(queries), n_q, dv), dtype=dtype, device="cuda")
        want, other = torch.empty(out.shape, dtype=F64), torch.empty(out.shape, dtype=F64)
        kernels.paged_attention(*args, max(queries), max(contexts), scale, None, out, starts, softcap, **extra)
        plain_ops.paged_attention(*host, max(queries), max(contexts), scale, None, want, None, softcap, **plain_extra)
        kernels.check_device_errors(out.device)
        assert torch.isfinite(out).all() and close(out, want, dtype)
        plain_ops.paged_attention(*host, max(queries), max(contexts), scale, None, other, None, None, **plain_extra)
        if softcap == 2.0:
            assert float((other - want).abs().max()) > 0.1 * float(want.abs().max())        # the cap matters


@pytest.mark.parametrize("n_q,n_kv,d,dv,page", [(8, 2, 64, 64, 16), (8, 1, 128, 128, 16), (4, 2, 128, 48, 16), (4, 4, 32, 32, 16)])
def test_capped_scores_far_beyond_the_cap(n_q, n_kv, d, dv, page):
    """Scores hundreds of times the cap (the exponential inside overflows or vanishes): every key weighs e^cap or e^-cap."""
    from miniserve_b200 import kernels

    for queries, contexts in (([1, 1], [200, 65]), ([130], [130])):
        args, host, starts = attention_case(torch.bfloat16, n_q, n_kv, d, dv, page, queries, contexts, key_scale=300.0)
        out, want = torch.empty((sum(queries), n_q, dv), dtype=torch.bfloat16, device="cuda"), torch.empty((sum(queries), n_q, dv), dtype=F64)
        kernels.paged_attention(*args, max(queries), max(contexts), 1.0, None, out, starts, 1.5)
        plain_ops.paged_attention(*host, max(queries), max(contexts), 1.0, None, want, None, 1.5)
        kernels.check_device_errors(out.device)
        assert torch.isfinite(out).all() and close(out, want, torch.bfloat16)


def test_which_kernels_take_a_soft_cap(caplog):
    from miniserve_b200 import kernels

    assert kernels.attention_kernels(torch.bfloat16, 128, 8, 2, 16, False, 48, True)["prompt"] == "mma.sync (any size)"
    assert kernels.attention_kernels(torch.bfloat16, 128, 8, 2, 16, False, None, True)["prompt"] == "tcgen05"
    assert kernels.attention_kernels(torch.bfloat16, 128, 8, 2, 16, True, 48, True)["prompt"] == "general"


# --------------------------------------------------------------------------- parts alone


def layer_parts(entry, width, eps=1e-5, value_mix=None):
    """Mixer and feed-forward of one layer (tensor names under ``l0.``), built as the architecture builds them."""
    import miniserve_b200  # noqa: F401
    from miniserve_b200.architectures.parunex import build_parunex_spec
    from miniserve_b200.config import ParunexConfig
    from miniserve_b200.parts import FEED_FORWARDS, MIXERS, PartSpec

    layer = build_parunex_spec(ParunexConfig.from_dict(ph.model(50, width, 1.0, eps, [entry]))).layers[0]
    mixer = layer.mixer
    if entry["type"] == "attention":
        mixer = PartSpec(mixer.kind, dict(mixer.args, value_mix=value_mix))
    return (MIXERS.build(mixer, prefix="l0."),
            None if layer.feed_forward is None else FEED_FORWARDS.build(layer.feed_forward, prefix="l0."))


def part_weights(part, dtype, seed, std=0.15):
    w = {}
    for i, spec in enumerate(part.param_specs()):
        if spec.name.endswith("norm"):
            value = 1 + rand(spec.shape, torch.float32, seed + i, 0.2)
        elif spec.name.endswith("sink"):
            value = torch.linspace(-1.0, 2.0, spec.shape[0]).cuda()
        elif spec.name.endswith("vmix"):
            value = torch.tensor(0.4).cuda()
        elif spec.name.endswith("a2.b"):
            value = rand(spec.shape, torch.float32, seed + i, 1.0) + 1.5
        elif spec.name.endswith(".b"):
            value = rand(spec.shape, torch.float32, seed + i, 0.3)
        else:
            value = rand(spec.shape, torch.float32, seed + i, std)
        w[spec.name] = value.to(torch.float32 if spec.kind == "matrix_f32" else dtype)
    return w


def run_plain(entry, w, x, shared=None):
    return plain.MIXERS[entry["type"]](x, w, "l0.mix.", entry["mixer"], 1e-5, {} if shared is None else shared)


ALONE = [(96, ph.PARUNEX_A["layers"][0]), (96, ph.PARUNEX_A["layers"][1]), (96, ph.PARUNEX_A["layers"][2]), (96, ph.PARUNEX_A["layers"][3]),
         (72, ph.PARUNEX_B["layers"][0]), (72, ph.PARUNEX_B["layers"][1]), (128, ph.PARUNEX_C["layers"][0]), (128, ph.PARUNEX_C["layers"][1]),
         (128, ph.PARUNEX_C["layers"][2]), (128, ph.PARUNEX_C["layers"][3]), (44, ph.PARUNEX_D["layers"][0]), (44, ph.PARUNEX_D["layers"][1]),
         (64, ph.PARUNEX_E["layers"][1]), (64, ph.layer(ph.attention(16, 1, 32, 48, 0.2, ph.rot(300.0, 16), 3.0), None))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(ALONE)))
def test_mixers_in_portions_and_pages_and_slots_used_again(dtype, case):
    """A sequence in portions down to one and two tokens and then token by token, a second beside it in the same steps, and a third on
    the pages, or in the slot, that the first gave back.  Attention layers mix in values that the step was handed."""
    width, entry = ALONE[case]
    mixes = entry["type"] == "attention"
    if mixes:
        entry = dict(entry, mixer=dict(entry["mixer"], v_mix=True))
    part, _ = layer_parts(entry, width, value_mix="mix" if mixes else None)
    w = part_weights(part, dtype, 70)
    part.load(w)
    wd = {k: v.double().cpu() for k, v in w.items()}
    harness = Harness([part.cache_need()], dtype, page_size=8, num_pages=40, max_seqs=2, max_len=512)
    first, second, third = rand((170, width), dtype, 80), rand((131, width), dtype, 81), rand((90, width), dtype, 82)
    total = entry["mixer"]["kv_heads"] * entry["mixer"]["vdim"] if mixes else 0
    given = {n: rand((len(x), total), dtype, 90 + i) for i, (n, x) in enumerate((("a", first), ("b", second), ("c", third)))}

    def forward(portions, batch, spans):
        ctx = harness.context(portions)
        ctx.dtype = dtype
        if mixes:
            ctx.buffer("attention.kept_values", (batch.shape[0], total), dtype).copy_(torch.cat([given[n][lo:hi] for n, lo, hi in spans]))
        return part.forward(batch.contiguous(), ctx, harness.view(ctx, 0)).clone()

    def expected(name, x):
        return run_plain(entry, wd, x.double().cpu(), dict(first_values=given[name].double().cpu()) if mixes else None)

    cuts = [0, 1, 3, 5, 62, 64, 150] + list(range(151, len(first) + 1))
    got_first, got_second, at = [], [], 0
    for start, end in zip(cuts[:-1], cuts[1:]):
        portions = {"a": end - start}
        take = min(len(second) - at, 1 if end - start > 20 else 17)
        if take:
            portions["b"] = take
        out = forward(portions, torch.cat([first[start:end], second[at:at + take]]), [("a", start, end), ("b", at, at + take)])
        got_first.append(out[:end - start])
        got_second.append(out[end - start:])
        at += take
    for got, name, x in ((got_first, "a", first), (got_second, "b", second)):
        assert close(torch.cat(got), expected(name, x), dtype)
    harness.manager.release("a")
    assert close(forward({"c": len(third)}, third, [("c", 0, len(third))]), expected("c", third), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 16, 24), (8, 2, 64, 64), (3, 1, 48, 32), (2, 2, 128, 128), (4, 2, 128, 48)])
def test_a_far_key_the_cap_and_the_sink_decide(dtype, heads, kv_heads, dim, vdim):
    """Most scores far below the sink: a loud key near the start takes the weight of every later query, in a prompt portion and in
    tokens decoded 300 positions on; without the sink or with another cap the rows would be others."""
    width, total, decode_from = 64, 320, 300
    rotation = ph.rot(1000.0, 8, (4.0, 1.0, 4.0, 400))
    entry = ph.attention(heads, kv_heads, dim, vdim, 1.5 * dim ** -0.5, rotation, 6.0)
    part, _ = layer_parts(dict(entry, mlp=None), width)
    w = part_weights(part, dtype, 31, 0.05)
    x = rand((total, width), dtype, 51)
    for name, factor in (("l0.mix.q", 1.0), ("l0.mix.k", -1.0)):
        w[name].view(-1, dim, width)[:, -2:, 0] = 3.0 * factor
        w[name].view(-1, dim, width)[:, :2, 1:9] = 0.3 * factor
    x[:, 0] = 1.0
    x[2, 0] = -4.0
    part.load(w)
    harness = Harness([part.cache_need()], dtype, page_size=8, num_pages=64, max_seqs=2, max_len=512)
    cuts = [(0, 2), (2, 9), (9, decode_from)] + [(i, i + 1) for i in range(decode_from, total)]
    got = []
    for start, end in cuts:
        ctx = harness.context({"r": end - start})
        ctx.dtype = dtype
        got.append(part.forward(x[start:end].contiguous(), ctx, harness.view(ctx, 0)).clone())
    xd, wd = x.double().cpu(), {k: v.double().cpu() for k, v in w.items()}
    expected = run_plain(entry, wd, xd)
    scale = float(expected.abs().max())
    assert close(torch.cat(got), expected, dtype)
    quiet = xd.clone()
    quiet[2, 0] = 1.0
    assert float((run_plain(entry, wd, quiet)[decode_from:] - expected[decode_from:]).abs().max()) > 0.1 * scale
    no_sink = dict(wd, **{"l0.mix.sink": torch.full((heads,), -1e4, dtype=F64)})
    assert float((run_plain(entry, no_sink, quiet)[decode_from:] - run_plain(entry, wd, quiet)[decode_from:]).abs().max()) > 0.02 * scale
    wide = dict(entry, mixer=dict(entry["mixer"], softcap=12.0))
    assert float((run_plain(wide, wd, xd)[decode_from:] - expected[decode_from:]).abs().max()) > 0.01 * scale


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,tau", [(3, 20, 12, 16.0), (2, 64, 64, 4.0), (1, 5, 40, 1.0)])
def test_a_far_write_is_kept_and_read_back(dtype, heads, dim, vdim, tau):
    """Most tokens write next to nothing and every channel forgets slowly; one token near the start writes loudly: tokens hundreds of
    positions on read it back, in a portion and decoded alone; a state that was lost or mixed up between steps, or a decay to
    another power, would give other rows."""
    width, total, decode_from = 64, 320, 300
    entry = ph.gla(heads, dim, vdim, tau, 6)
    part, _ = layer_parts(dict(entry, mlp=None), width)
    w = part_weights(part, dtype, 41)
    w["l0.mix.a2.b"] = (rand((heads * dim,), torch.float32, 3, 0.3) + float(torch.logit(torch.tensor(0.995 ** tau)))).to(dtype)
    w["l0.mix.k"][:, 1:] *= 0.2
    w["l0.mix.k"][:, 0] = 0.5
    w["l0.mix.q"][:, 0] = 0.5
    x = rand((total, width), dtype, 52)
    x[:, 0] = 0.05
    x[3, 0] = 8.0
    part.load(w)
    harness = Harness([part.cache_need()], dtype, page_size=8, num_pages=64, max_seqs=2, max_len=512)
    cuts = [(0, 2), (2, 9), (9, decode_from)] + [(i, i + 1) for i in range(decode_from, total)]
    got = []
    for start, end in cuts:
        ctx = harness.context({"r": end - start, "other": 3} if start == 9 else {"r": end - start})
        ctx.dtype = dtype
        batch = x[start:end] if start != 9 else torch.cat([x[start:end], rand((3, width), dtype, 60)])
        got.append(part.forward(batch.contiguous(), ctx, harness.view(ctx, 0))[:end - start].clone())
    xd, wd = x.double().cpu(), {k: v.double().cpu() for k, v in w.items()}
    expected = run_plain(entry, wd, xd)
    scale = float(expected.abs().max())
    assert close(torch.cat(got), expected, dtype)
    quiet = xd.clone()
    quiet[3, 0] = 0.05
    assert float((run_plain(entry, wd, quiet)[decode_from:] - expected[decode_from:]).abs().max()) > 0.1 * scale
    other = dict(entry, mixer=dict(entry["mixer"], tau=1.5 * tau))
    assert float((run_plain(other, wd, xd)[decode_from:] - expected[decode_from:]).abs().max()) > 0.02 * scale
    assert float((run_plain(entry, wd, xd[200:])[decode_from - 200:] - expected[decode_from:]).abs().max()) > 0.1 * scale


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n", [1, 6, 9, 150])
@pytest.mark.parametrize("width,mlp", [(96, ph.dense(56)), (72, ph.dense(50)), (128, ph.dense(256)), (96, ph.moe(6, 2, 20, 1.7, 3, 2)),
                                       (64, ph.moe(8, 3, 26, 0.6, 2, 1)), (128, ph.moe(16, 4, 32, 2.5, 4, 2)), (44, ph.moe(5, 5, 18, 1.0))])
def test_feed_forwards(dtype, n, width, mlp):
    """Both kinds; rows whose choice is a close call at the compute type's rounding are left out."""
    from types import SimpleNamespace

    from miniserve_b200.parts.context import StepContext

    entry = dict(ph.gla(1, 4, 4, 1.0, 1), mlp=mlp)
    _, part = layer_parts(entry, width)
    w = part_weights(part, dtype, 7)
    part.load(w)
    wd = {k: v.double().cpu() for k, v in w.items()}
    x = rand((n, width), dtype, 8)
    ctx = SimpleNamespace(memo={}, device=torch.device("cuda"), dtype=dtype, n_tokens=n)
    ctx.buffer = lambda *args: StepContext.buffer(ctx, *args)
    out = part.forward(x, ctx).double().cpu()
    xd = x.double().cpu()
    expected = plain.feed_forward(xd, wd, "l0.mlp.", mlp)
    rows = list(range(n))
    if mlp["kind"] == "moe":
        scores = torch.sigmoid(xd @ wd["l0.mlp.router"].T)
        moved = [torch.sigmoid(xd @ wd["l0.mlp.router"].T + 1e-5 * torch.randn(scores.shape, generator=torch.Generator().manual_seed(s), dtype=F64))
                 for s in range(4)]
        rows = [t for t in rows if all(plain.chosen_experts(m[t], mlp["router"]) == plain.chosen_experts(scores[t], mlp["router"]) for m in moved)]
        assert len(rows) >= 0.9 * n
    assert torch.allclose(out[rows], expected[rows], **tol(dtype, float(expected.abs().max())))


# --------------------------------------------------------------------------- the whole model


def build(folder, dtype, num_pages, page_size, max_seqs=4, execution="eager"):
    import miniserve_b200  # noqa: F401
    from miniserve_b200.config import EngineConfig
    from miniserve_b200.engine.runtime import build_runtime

    return build_runtime(folder, EngineConfig(dtype=dtype, kv_block_size=page_size, num_kv_blocks=num_pages, max_num_seqs=max_seqs,
                                              enable_prefix_cache=False, decode_execution=execution))


def replay(runtime, steps):
    from miniserve_b200 import kernels
    from miniserve_b200.trace import TraceSession

    session, outputs = TraceSession(runtime), {}
    for record in steps:
        logits = session.run(record)
        if logits is not None:
            outputs[record["step"]] = logits.double().cpu()
    kernels.check_device_errors(runtime.step_function.device)
    runtime.manager.check_invariants()
    return outputs


_ORACLE: dict = {}


def oracle(folder, tokens):
    key = (Path(folder).name, tuple(tokens))      # (a folder's name says configuration, seed and stored type: the same weights)
    if key not in _ORACLE:
        config, weights = ph.load_folder(folder)
        _ORACLE[key] = plain.forward(tokens, weights, config)
    return _ORACLE[key]


def check(folder, dtype, requests, got, positions_of=None):
    worst = 0.0
    for rid, tokens in requests.items():
        expected = oracle(folder, tokens)
        bound = bound_of(dtype, expected)
        wanted = sorted(got[rid]) if positions_of is None else positions_of[rid]
        assert sorted(got[rid]) == list(wanted), rid
        for position, row in got[rid].items():
            ratio = float((row - expected[position]).abs().max()) / bound
            assert ratio <= 1.0, (rid, position, ratio)
            worst = max(worst, ratio)
    return worst


CUTTINGS = {
    "whole": helpers.cut_whole,
    "tail": lambda r: helpers.cut_decode_tail(r, 32),
    "portions": lambda r: helpers.cut_portions(r, seed=3),
    "mixed": lambda r: helpers.cut_mixed(r, seed=4),
}
# lengths at the borders of pages of 4, 8, 16 and 64 tokens, of key tiles of 32 and of the scan's chunks; a single token; a hundred
LENGTHS = (1, 2, 8, 9, 15, 16, 17, 32, 33, 64, 65, 130)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,page_size", [("a", 8), ("b", 16), ("c", 16), ("b", 4), ("c", 64), ("d", 8), ("e", 16)])
@pytest.mark.parametrize("cutting", list(CUTTINGS))
def test_cuttings_against_plain(tmp_path, request, dtype, name, page_size, cutting):
    """Whole prompts; last tokens decoded one by one; portions down to two tokens; unequal requests batched together in a pool so
    small that pages and slots are used again: always the logits of the plain whole-sequence computation."""
    folder = ph.make_folder(tmp_path, name, seed=11)
    vocab = ph.CONFIGS[name]["vocab"]
    requests = {f"r{i}": helpers.random_tokens(vocab, n, seed=400 + i) for i, n in enumerate(LENGTHS)}
    steps = CUTTINGS[cutting](requests)
    granule = max(64, page_size)
    runtime = build(folder, dtype, helpers.max_live_tokens(steps, granule=granule) // page_size, page_size)
    got = helpers.collect(steps, replay(runtime, steps))
    worst = check(folder, dtype, requests, got)
    helpers.note_ratio(request.node.name, worst)
    assert not runtime.manager.requests and all(a.free_count == a.num_pages for a in runtime.manager.allocators)


@pytest.mark.parametrize("seed", range(6))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_random_configurations(tmp_path, dtype, seed):
    rng = random.Random(100 + seed)
    config = ph.random_config(rng)
    folder = ph.make_folder(tmp_path, f"random{seed}", seed=3, config=config)
    requests = {f"r{i}": helpers.random_tokens(config["vocab"], n, seed=40 + i) for i, n in enumerate((1, 7, 18, 40, 90))}
    steps = CUTTINGS[rng.choice(["tail", "portions", "mixed"])](requests)
    page_size = rng.choice([4, 8, 16, 32])
    runtime = build(folder, dtype, helpers.max_live_tokens(steps, granule=64) // page_size, page_size)
    check(folder, dtype, requests, helpers.collect(steps, replay(runtime, steps)))


@pytest.mark.parametrize("name,page_size", [("a", 8), ("c", 16)])
def test_float32_logits_do_not_depend_on_cutting_or_batch(tmp_path, name, page_size):
    folder = ph.make_folder(tmp_path, name, seed=16)
    vocab = ph.CONFIGS[name]["vocab"]
    requests = {f"r{i}": helpers.random_tokens(vocab, n, seed=900 + i) for i, n in enumerate((1, 9, 33, 64, 65, 150))}
    results = {}
    for cutting in ("whole", "portions", "mixed"):
        steps = CUTTINGS[cutting](requests)
        runtime = build(folder, "float32", helpers.max_live_tokens(steps, granule=64) // page_size, page_size)
        results[cutting] = helpers.collect(steps, replay(runtime, steps))
    for rid, tokens in requests.items():
        for position in range(len(tokens)):
            alone = results["whole"][rid][position]
            scale = max(1.0, float(alone.abs().max()))
            for cutting in ("portions", "mixed"):
                assert float((results[cutting][rid][position] - alone).abs().max()) <= 4e-6 * scale, (rid, position, cutting)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_prefill_against_decoding_every_token(tmp_path, dtype, name):
    """The same sequence as one prompt and token by token from its first token on: a long decode over many pages."""
    folder = ph.make_folder(tmp_path, name, seed=12)
    tokens = helpers.random_tokens(ph.CONFIGS[name]["vocab"], 200, seed=500)
    runtime = build(folder, dtype, 64, 8)
    whole = replay(runtime, helpers.cut_whole({"w": tokens}))[0]
    steps = helpers.cut_decode_tail({"d": tokens}, tail=len(tokens))
    single = helpers.collect(steps, replay(runtime, steps))["d"]
    expected = oracle(folder, tokens)
    bound = bound_of(dtype, expected)
    for position in range(len(tokens)):
        for a, b in ((whole, expected), (single, expected), (single, whole)):
            assert float((a[position] - b[position]).abs().max()) <= bound, position


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("execution", ["eager", "cuda_graph"])
def test_many_live_requests_decoding(tmp_path, dtype, execution):
    """Seven requests live at once, decoded in steps of single tokens whose live set changes (captured graphs with padding rows when
    graphs are on)."""
    folder = ph.make_folder(tmp_path, "c", seed=13)
    vocab = ph.CONFIGS["c"]["vocab"]
    prompt_lens = {f"m{i}": n for i, n in enumerate((3, 1, 17, 40, 9, 64, 25))}
    requests = {rid: helpers.random_tokens(vocab, n + 11, seed=600 + i) for i, (rid, n) in enumerate(prompt_lens.items())}
    steps = helpers.cut_many_live(requests, prompt_lens, seed=2)
    runtime = build(folder, dtype, 7 * 6, 16, max_seqs=7, execution=execution)
    got = helpers.collect(steps, replay(runtime, steps))
    if execution == "cuda_graph":
        assert runtime.step_function.graph_replays > 0
    check(folder, dtype, requests, got, {rid: range(prompt_lens[rid] - 1, len(requests[rid])) for rid in requests})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,execution", [("a", "eager"), ("a", "cuda_graph"), ("e", "cuda_graph")])
def test_greedy_generation_through_the_scheduler(tmp_path, dtype, name, execution):
    """``LLM.generate``: the engine's own entry point, scheduler (chunked prompts, a token budget that forces portions, more prompts
    than state slots) and sampler; every generated token is the plain implementation's choice, or as good as it within rounding."""
    from miniserve_b200.engine.llm import LLM
    from miniserve_b200.sampling import SamplingParams

    folder = ph.make_folder(tmp_path, name, seed=14)
    config, weights = ph.load_folder(folder)
    prompts = [helpers.random_tokens(config["vocab"], n, seed=700 + n) for n in (1, 5, 30, 77)]
    llm = LLM(str(folder), dtype=dtype, kv_block_size=8, num_kv_blocks=48, max_num_seqs=3, max_num_batched_tokens=24,
              decode_execution=execution)
    results = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=24))
    for prompt, result in zip(prompts, results):
        assert len(result.token_ids) == 24
        sequence = list(prompt) + list(result.token_ids)
        logits = plain.forward(sequence, weights, config)
        for at, produced in enumerate(result.token_ids):
            row = logits[len(prompt) + at - 1]
            best = int(torch.argmax(row))
            assert produced == best or float(row[best] - row[produced]) <= 2 * bound_of(dtype, row), (produced, best)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program_and_command_line(tmp_path, dtype):
    """``bin/trace_run`` and ``python -m miniserve_b200.generate`` on a Parunex folder, as a user runs them."""
    folder = ph.make_folder(tmp_path, "d", seed=15)
    vocab = ph.CONFIGS["d"]["vocab"]
    requests = {f"q{i}": helpers.random_tokens(vocab, n, seed=800 + i) for i, n in enumerate((2, 19, 70, 45, 33))}
    steps = helpers.cut_mixed(requests, seed=6)
    out_dir = tmp_path / "out"
    process = subprocess.run([sys.executable, str(REPO / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out_dir),
                              "--max-tokens", str(helpers.max_live_tokens(steps, granule=64))],
                             input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert process.returncode == 0, process.stderr[-2000:]
    assert [line for line in process.stdout.splitlines() if line.startswith("done")] == [f"done {s['step']}" for s in steps]
    outputs = {s["step"]: torch.from_numpy(np.fromfile(out_dir / f"{s['step']}.f32", dtype="<f4").reshape(-1, vocab)).double()
               for s in steps if any(e["want"] for e in s["entries"])}
    check(folder, dtype, requests, helpers.collect(steps, outputs))
    generated = subprocess.run([sys.executable, "-m", "miniserve_b200.generate", "--model", str(folder), "--dtype", dtype,
                                "--prompt-ids", ",".join(map(str, requests["q1"])), "--max-new-tokens", "5", "--num-kv-blocks", "32",
                                "--kv-block-size", "8", "--json"], capture_output=True, text=True, timeout=600, cwd=str(REPO))
    assert generated.returncode == 0, generated.stderr[-2000:]
    produced = json.loads(generated.stdout.strip().splitlines()[-1])["token_ids"]
    assert len(produced) == 5
    tokens = list(requests["q1"])
    for token in produced:
        logits = oracle(folder, tokens)[-1]
        best = int(torch.argmax(logits))
        assert token == best or float(logits[best] - logits[token]) <= 2 * bound_of(dtype, logits)
        tokens.append(token)
