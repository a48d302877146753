"""Venarax on the GPU against the plain implementation (``plain_venarax``) and the plain statements of the kernels (``plain_ops``):
every new or changed kernel alone, both mixers, the transition and the block alone (fed in portions down to one and two tokens and
token by token through the cache, with keys that stand out just inside and just outside a window and far back, pages that are used
again), and the whole model through the engine's own session, scheduler and command line, in float32 and bfloat16, at sizes of its
own."""

from __future__ import annotations

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import helpers
import plain_ops
import plain_venarax as plain
import venarax_helpers as vh
from test_parts_gpu import Harness, rand, tol

pytestmark = pytest.mark.gpu
REPO = Path(__file__).resolve().parent.parent
DTYPES = [torch.float32, torch.bfloat16]


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
@pytest.mark.parametrize("hidden", [44, 96, 1000, 2048, 4104, 8200])
@pytest.mark.parametrize("pending", ["nothing", "one", "two", "vector"])
def test_add_layernorm_kernel(dtype, hidden, pending):
    """One and two outputs, every kind of pending addition, rows picked out; a stream whose mean is far larger than its
    deviations (a mean taken off too late, or a one-pass variance, would lose them)."""
    from miniserve_b200 import kernels

    rows = 5
    residual = rand((rows, hidden), torch.float32, 1) + 20.0 * torch.arange(rows, device="cuda")[:, None]
    delta = rand((rows, hidden), dtype, 2) if pending in ("one", "two") else None
    delta2 = rand((rows, hidden), dtype, 3) if pending == "two" else None
    vector = rand((hidden,), torch.float32, 4) if pending == "vector" else None
    weights = [(1 + rand((hidden,), torch.float32, 5 + i, 0.3)).to(dtype) if i % 2 == 0 else rand((hidden,), dtype, 5 + i) for i in range(4)]
    for two in (False, True):
        for picked in (None, ints([rows - 1, 0])):
            if two and picked is not None:
                continue
            stream, want_stream = residual.clone(), cpu(residual).double()
            n = rows if picked is None else 2
            out, out2 = (torch.empty((n, hidden), dtype=dtype, device="cuda") for _ in range(2))
            want, want2 = (torch.empty((n, hidden), dtype=torch.float64) for _ in range(2))
            extra = dict(weight2=weights[2], bias2=weights[3], out2=out2) if two else {}
            kernels.add_layernorm(stream, delta, weights[0], weights[1], 1e-5, out, picked, delta2, vector, **extra)
            extra = dict(weight2=cpu(weights[2]), bias2=cpu(weights[3]), out2=want2) if two else {}
            plain_ops.add_layernorm(want_stream, cpu(delta), cpu(weights[0]), cpu(weights[1]), 1e-5, want, cpu(picked), cpu(delta2), cpu(vector), **extra)
            # (a float32 stream around 80 is itself rounded to 4e-6)
            assert torch.allclose(cpu(stream).double(), want_stream, atol=2e-5)
            assert close(out, want, dtype, 12.0) and (not two or close(out2, want2, dtype, 12.0))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,ld,col", [(44, 100, 3), (96, 192, 0), (96, 192, 96), (64, 200, 8), (2048, 4096, 2048)])
def test_stream_to_columns_kernel(dtype, hidden, ld, col):
    from miniserve_b200 import kernels

    residual, delta, delta2 = rand((7, hidden), torch.float32, 1), rand((7, hidden), dtype, 2), rand((7, hidden), dtype, 3)
    before = cpu(residual)
    for a, b in ((None, None), (delta, None), (delta, delta2)):
        out = torch.full((7, ld), 9.0, dtype=dtype, device="cuda")
        kernels.stream_to_columns(residual, a, out, col, b)
        want = torch.full((7, ld), 9.0, dtype=torch.float64)
        plain_ops.stream_to_columns(before, cpu(a), want, col, cpu(b))
        assert close(out, want, dtype, 3.0)
        assert torch.equal(cpu(out)[:, :col], torch.full((7, col), 9.0, dtype=dtype)) and torch.equal(cpu(residual), before)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n_q,n_kv,d,dv,rotary,interleaved", [(4, 2, 16, 24, 0, False), (3, 3, 7, 9, 0, False), (8, 1, 64, 64, 0, False),
                                                              (6, 2, 20, 12, 8, True), (2, 1, 12, 8, 12, False), (32, 8, 128, 128, 0, False),
                                                              (64, 16, 64, 64, 0, False), (64, 16, 128, 64, 0, False), (128, 16, 128, 64, 0, False)])
@pytest.mark.parametrize("temperature", [None, (0.4, 3.0), (-0.2, 1.0)])
def test_prepare_with_norms_over_the_whole_row(dtype, n_q, n_kv, d, dv, rotary, interleaved, temperature):
    from miniserve_b200 import kernels

    n, page, pages = 9, 4, 8
    ld = (n_q * d + n_kv * (d + dv) + 7) // 8 * 8
    proj = rand((n, ld), dtype, 1, 2.0)
    qw, kw = 1 + rand((n_q * d,), torch.float32, 2, 0.3), 1 + rand((n_kv * d,), torch.float32, 3, 0.3)
    positions = ints([0, 1, 2, 3, 5, 6, 200, 4094, 100001])
    slots = ints([5, 9, -1, 0, 31, 12, 13, 14, 2])
    table = None
    if rotary:
        table = torch.empty((n, rotary // 2, 2), device="cuda")
        kernels.rope_table(positions, torch.tensor([100.0 ** (-2 * i / rotary) for i in range(rotary // 2)], device="cuda"), table)
    for weights in ((qw, kw), (None, None)):
        k_pool, v_pool = torch.zeros((pages, n_kv, page, d), dtype=dtype).cuda(), torch.zeros((pages, n_kv, page, dv), dtype=dtype).cuda()
        q = torch.empty((n, n_q, d), dtype=dtype).cuda()
        want = [torch.zeros(t.shape, dtype=torch.float64) for t in (q, k_pool, v_pool)]
        kernels.qkv_prepare_rows(proj, 0, n_q * d, (n_q + n_kv) * d, n_q, n_kv, d, dv, slots, *weights, 1e-5, table, rotary, k_pool, v_pool, q,
                                 interleaved=interleaved, positions=positions, temperature=temperature)
        plain_ops.qkv_prepare_rows(cpu(proj), 0, n_q * d, (n_q + n_kv) * d, n_q, n_kv, d, dv, cpu(slots), cpu(weights[0]), cpu(weights[1]), 1e-5,
                                   cpu(table), rotary, want[1], want[2], want[0], interleaved=interleaved, positions=cpu(positions),
                                   temperature=temperature)
        for got, expected in zip((q, k_pool, v_pool), want):
            assert close(got, expected, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_prepare_with_norms_over_the_whole_row_of_many_tokens(dtype):
    """More tokens than blocks: every block takes several, fetching the next row while it works on one."""
    from miniserve_b200 import kernels

    n, n_q, n_kv, d, dv, page = 2500, 4, 2, 16, 24, 16
    proj = rand((n, n_q * d + n_kv * (d + dv)), dtype, 1, 2.0)
    qw, kw = 1 + rand((n_q * d,), torch.float32, 2, 0.3), 1 + rand((n_kv * d,), torch.float32, 3, 0.3)
    slots = torch.randperm(n, generator=torch.Generator().manual_seed(4)).to(torch.int32)
    slots[::97] = -1
    k_pool, v_pool = torch.zeros((160, n_kv, page, d), dtype=dtype).cuda(), torch.zeros((160, n_kv, page, dv), dtype=dtype).cuda()
    q = torch.empty((n, n_q, d), dtype=dtype).cuda()
    want = [torch.zeros(t.shape, dtype=torch.float64) for t in (q, k_pool, v_pool)]
    positions = torch.arange(n, dtype=torch.int32)
    kernels.qkv_prepare_rows(proj, 0, 64, 96, n_q, n_kv, d, dv, slots.cuda(), qw, kw, 1e-5, None, 0, k_pool, v_pool, q,
                             positions=positions.cuda(), temperature=(0.3, 100.0))
    plain_ops.qkv_prepare_rows(cpu(proj), 0, 64, 96, n_q, n_kv, d, dv, slots, cpu(qw), cpu(kw), 1e-5, None, 0, want[1], want[2], want[0],
                               positions=positions, temperature=(0.3, 100.0))
    for got, expected in zip((q, k_pool, v_pool), want):
        assert close(got, expected, dtype)


def attention_case(dtype, n_q, n_kv, d, dv, page, queries, contexts, seed=0):
    """A batch over scrambled pages: (arguments of kernels.paged_attention up to the context length, the same on the CPU)."""
    requests = len(queries)
    width = (max(contexts) + page - 1) // page
    order = torch.randperm(requests * width + 3, generator=torch.Generator().manual_seed(seed))
    tables = order[:requests * width].view(requests, width).to(torch.int32)
    k_pool, v_pool = rand((requests * width + 3, n_kv, page, d), dtype, seed + 1), rand((requests * width + 3, n_kv, page, dv), dtype, seed + 2)
    n = sum(queries)
    q = rand((n, n_q, d), dtype, seed + 3)
    request_of = torch.tensor([r for r, m in enumerate(queries) for _ in range(m)], dtype=torch.int32)
    positions = torch.tensor([contexts[r] - queries[r] + i for r in range(requests) for i in range(queries[r])], dtype=torch.int32)
    starts = [sum(queries[:i]) for i in range(requests + 1)]
    host = [q, k_pool, v_pool, tables, request_of, positions, torch.tensor(starts, dtype=torch.int32), torch.tensor(contexts, dtype=torch.int32)]
    return [t.cuda() for t in host], [t.cpu() for t in host], starts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n_q,n_kv,d,dv,page", [(6, 2, 48, 80, 16), (4, 4, 32, 64, 8), (4, 2, 96, 96, 16), (3, 1, 7, 9, 4), (8, 2, 64, 64, 16),
                                                (16, 4, 128, 128, 64), (4, 4, 32, 32, 16)])
@pytest.mark.parametrize("queries,contexts", [([1, 1, 1], [1, 700, 33]), ([1, 150, 2], [300, 170, 2]), ([200], [200])])
def test_attention_kernels_with_a_learned_sink(dtype, n_q, n_kv, d, dv, page, queries, contexts):
    """Every attention kernel (general; tensor cores for any size, for unrolled sizes and, on prompts, tcgen05), single tokens with
    their keys split and prompt portions in one batch, with sinks from far below every score to far above them."""
    from miniserve_b200 import kernels

    scores = torch.tensor([[-40.0, 0.0, 1.5, -2.0, 4.0, 60.0][h % 6] for h in range(n_q)])
    args, host, starts = attention_case(dtype, n_q, n_kv, d, dv, page, queries, contexts)
    out = torch.empty((sum(queries), n_q, dv), dtype=dtype, device="cuda")
    want = torch.empty(out.shape, dtype=torch.float64)
    kernels.paged_attention(*args, max(queries), max(contexts), 1.5 * d ** -0.5, None, out, starts, sink=scores.cuda())
    plain_ops.paged_attention(*host, max(queries), max(contexts), 1.5 * d ** -0.5, None, want, sink=scores)
    kernels.check_device_errors(out.device)
    assert torch.isfinite(out).all() and close(out, want, dtype)
    other = torch.empty_like(want)
    plain_ops.paged_attention(*host, max(queries), max(contexts), 1.5 * d ** -0.5, None, other, sink=True)
    assert float((other - want).abs().max()) > 0.1 * float(want.abs().max())        # the scores matter


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 8, 40, 700])
@pytest.mark.parametrize("inner,width", [(64, 96), (512, 256), (30, 44)])
@pytest.mark.parametrize("limit", [0.4, 3.0])
def test_clamped_gated_activation(dtype, rows, inner, width, limit):
    """The fused products' choice for these sizes and every kernel that can carry the activation, called by name."""
    from miniserve_b200 import kernels

    x, gate, up = rand((rows, width), dtype, 1), rand((inner, width), dtype, 2, 0.15), rand((inner, width), dtype, 3, 0.15)
    g, u = cpu(x).double() @ cpu(gate).double().T, cpu(x).double() @ cpu(up).double().T
    want = plain_ops.clamped_glu_values(g, u, limit)
    both = torch.cat([g, u], dim=1).to(dtype).cuda()
    out = torch.empty((rows, inner), dtype=dtype, device="cuda")
    kernels.silu_mul(both, out, limit=limit)
    assert close(out, want, dtype)
    if inner % 8:
        return
    paired = kernels.interleave_gate_up(gate, up).contiguous()
    runs = [lambda: kernels.gated_up(x, paired, out, limit=limit)]
    if dtype == torch.bfloat16:
        if rows <= 8:
            runs.append(lambda: kernels.linear_wide(x, paired, out, gated=True, limit=limit))
        runs += [lambda wide=wide: kernels.linear_pair(x, paired, out, gated=True, wide=wide, limit=limit) for wide in (False, True)]
    for run in runs:
        out.zero_()
        run()
        assert close(out, want, dtype)
    kernels.check_device_errors(out.device)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,ld,col", [(5, 44, 100, 3), (130, 256, 512, 256), (3, 1000, 1000, 0), (9, 64, 80, 12)])
def test_gate_per_entry_kernel(dtype, rows, width, ld, col):
    from miniserve_b200 import kernels

    x, gate = rand((rows, width), dtype, 1, 2.0), rand((rows, ld), dtype, 2, 3.0)
    out, want = torch.empty_like(x), torch.empty((rows, width), dtype=torch.float64)
    kernels.sigmoid_gate_mul(x, gate, col, out)
    plain_ops.sigmoid_gate_mul(cpu(x), cpu(gate), col, want)
    assert close(out, want, dtype)
    kernels.sigmoid_gate_mul(x, gate, col, x)
    assert torch.equal(x, out)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rot,rot_dims,rank", [(5, 12, 4, 4, 24), (3, 7, 2, 2, 21), (8, 32, 16, 16, 64), (2, 16, 12, 6, 128)])
def test_latent_prepare_with_an_interleaved_rotation(dtype, heads, dim, rot, rot_dims, rank):
    from miniserve_b200 import kernels

    n, page = 6, 4
    ld = (heads * (dim + rot) + rank + rot + 7) // 8 * 8
    proj, weight = rand((n, ld), dtype, 1), 1 + rand((rank,), dtype, 2, 0.2)
    positions, slots = ints([0, 1, 9, 100, 4095, 100000]), ints([3, 0, -1, 7, 19, 11])
    table = torch.empty((n, rot_dims // 2, 2), device="cuda")
    kernels.rope_table(positions, torch.tensor([100.0 ** (-2 * i / rot_dims) for i in range(rot_dims // 2)], device="cuda"), table)
    for interleaved in (True, False):
        cache, q_full = torch.zeros((5, page, rank + rot), dtype=dtype).cuda(), torch.zeros((n, heads, rank + rot), dtype=dtype).cuda()
        want_cache, want_q = torch.zeros(cache.shape, dtype=torch.float64), torch.zeros(q_full.shape, dtype=torch.float64)
        kernels.latent_prepare(proj, 0, heads * (dim + rot), heads, dim, rot, rank, slots, weight, 1e-5, table, rot_dims, cache, q_full,
                               interleaved=interleaved)
        plain_ops.latent_prepare(cpu(proj), 0, heads * (dim + rot), heads, dim, rot, rank, cpu(slots), cpu(weight), 1e-5, cpu(table), rot_dims,
                                 want_cache, want_q, interleaved=interleaved)
        assert close(cache, want_cache, dtype) and close(q_full, want_q, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank,rot,page", [(8, 64, 16, 16), (3, 24, 4, 8), (20, 128, 32, 16), (16, 512, 64, 64), (2, 256, 16, 4)])
@pytest.mark.parametrize("window", [1, 31, 32, 33, 100])
def test_latent_attention_kernels_behind_a_window(dtype, heads, rank, rot, page, window):
    """Single tokens whose windows start at every place of a key tile (their keys split into few or many ranges, some empty) and
    prompt portions, with pages before the window gone from the table (their entries point at a page of huge numbers)."""
    from miniserve_b200 import kernels

    for queries, contexts in (([1] * 6, [1, 32, 33, 64, 700, 701]), ([70, 3, 1], [70, 300, 129])):
        requests, width = len(queries), (max(contexts) + page - 1) // page
        tables = torch.randperm(requests * width, generator=torch.Generator().manual_seed(3)).view(requests, width).to(torch.int32)
        cache = rand((requests * width + 1, page, rank + rot), dtype, 4)
        cache[-1] = 1e4
        for r in range(requests):
            first_page = max(0, contexts[r] - queries[r] - window + 1) // page
            tables[r, :first_page] = requests * width
        n = sum(queries)
        q = rand((n, heads, rank + rot), dtype, 5)
        request_of = torch.tensor([r for r, m in enumerate(queries) for _ in range(m)], dtype=torch.int32)
        positions = torch.tensor([contexts[r] - queries[r] + i for r in range(requests) for i in range(queries[r])], dtype=torch.int32)
        starts = torch.tensor([sum(queries[:i]) for i in range(requests + 1)], dtype=torch.int32)
        host = [q.cpu(), cache.cpu(), tables, request_of, positions, starts, torch.tensor(contexts, dtype=torch.int32)]
        out, want = torch.empty((n, heads, rank), dtype=dtype).cuda(), torch.empty((n, heads, rank), dtype=torch.float64)
        scale = 1.5 * (rank + rot) ** -0.5
        kernels.latent_attention(*[t.cuda() for t in host], max(queries), max(contexts), rank, scale, window, out)
        plain_ops.latent_attention(*host, max(queries), max(contexts), rank, scale, window, want)
        assert close(out, want, dtype)


# --------------------------------------------------------------------------- parts alone


def mixer_part(entry, width, eps=1e-5):
    """The mixer of one layer (tensor names under ``l0.mix.``), built as the architecture builds it."""
    import miniserve_b200  # noqa: F401
    from miniserve_b200.architectures.venarax import build_venarax_spec
    from miniserve_b200.config import VenaraxConfig
    from miniserve_b200.parts import MIXERS

    raw = vh.model(50, width, eps, None, [dict(entry, mlp=None)])
    return MIXERS.build(build_venarax_spec(VenaraxConfig.from_dict(raw)).layers[0].mixer, prefix="l0.")


def part_weights(part, dtype, seed, std=0.15):
    w = {}
    for i, spec in enumerate(part.param_specs()):
        if spec.name.endswith("norm"):
            value = 1 + rand(spec.shape, torch.float32, seed + i, 0.2)
        elif spec.name.endswith("sink"):
            value = torch.linspace(-1.0, 2.0, spec.shape[0]).cuda()
        else:
            value = rand(spec.shape, torch.float32, seed + i, std)
        w[spec.name] = value.to(dtype)
    return w


def run_plain(entry, w, x):
    return plain.MIXERS[entry["type"]](x, w, "l0.mix.", entry["mixer"], 1e-5)


ALONE = [(96, vh.VENARAX_A["layers"][0]), (96, vh.VENARAX_A["layers"][1]), (96, vh.VENARAX_A["layers"][2]), (96, vh.VENARAX_A["layers"][3]),
         (72, vh.VENARAX_B["layers"][0]), (72, vh.VENARAX_B["layers"][1]), (128, vh.VENARAX_C["layers"][0]), (128, vh.VENARAX_C["layers"][1]),
         (128, vh.VENARAX_C["layers"][2]), (128, vh.VENARAX_C["layers"][3]), (44, vh.VENARAX_D["layers"][0]), (44, vh.VENARAX_D["layers"][1]),
         (64, vh.layer(vh.latent(18, 16, 16, 24, 96, 0.2, 300.0, 64), None)), (64, vh.layer(vh.sink(16, 1, 32, 48, 0.2, 0.2, 10), None))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(ALONE)))
def test_mixers_in_portions_and_pages_used_again(dtype, case):
    """A sequence in portions down to one and two tokens and then token by token, a second beside it in the same steps, and a
    third on the pages that the first gave back."""
    width, entry = ALONE[case]
    part = mixer_part(entry, width)
    w = part_weights(part, dtype, 70)
    part.load(w)
    wd = {k: v.double().cpu() for k, v in w.items()}
    harness = Harness([part.cache_need()], dtype, page_size=8, num_pages=40, max_seqs=2, max_len=512)
    first, second, third = rand((170, width), dtype, 80), rand((131, width), dtype, 81), rand((90, width), dtype, 82)
    cuts = [0, 1, 3, 5, 62, 64, 150] + list(range(151, len(first) + 1))
    got_first, got_second, at = [], [], 0
    for start, end in zip(cuts[:-1], cuts[1:]):
        portions = {"a": end - start}
        take = min(len(second) - at, 1 if end - start > 20 else 17)
        if take:
            portions["b"] = take
        ctx = harness.context(portions)
        ctx.dtype = dtype
        batch = torch.cat([first[start:end], second[at:at + take]]).contiguous()
        out = part.forward(batch, ctx, harness.view(ctx, 0))
        got_first.append(out[:end - start].clone())
        got_second.append(out[end - start:].clone())
        at += take
    for got, x in ((got_first, first), (got_second, second)):
        assert close(torch.cat(got), run_plain(entry, wd, x.double().cpu()), dtype)
    harness.manager.release("a")
    ctx = harness.context({"c": len(third)})
    ctx.dtype = dtype
    assert close(part.forward(third, ctx, harness.view(ctx, 0)), run_plain(entry, wd, third.double().cpu()), dtype)


def loud_latent(w, x, m, loud):
    """Queries read a constant input column into a head's last unrotated entry, the latent's first entry reads it with the other
    sign and is that entry's key: every score is pushed far down, but for the tokens in ``loud``, whose column has the other
    sign: their keys take the softmax's weight wherever they are seen."""
    q = w["l0.mix.q"].view(m["heads"], m["dim"] + m["rot_dim"], -1)
    q[:, m["dim"] - 1, 0] = 6.0
    w["l0.mix.dkv"][0] = 0.0
    w["l0.mix.dkv"][0, 0] = -6.0
    uk = w["l0.mix.uk"].view(m["heads"], m["dim"], -1)
    uk[:, m["dim"] - 1] = 0.0
    uk[:, m["dim"] - 1, 0] = 1.0
    x[:, 0] = 1.0
    for token in loud:
        x[token, 0] = -5.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rot_dim,vdim,kv_rank,window", [(5, 12, 4, 10, 24, 13), (4, 32, 16, 32, 64, 64), (3, 16, 8, 8, 40, 50),
                                                                   (2, 24, 16, 16, 128, 96), (20, 8, 16, 8, 96, 33)])
def test_latent_part_at_the_windows_edges(dtype, heads, dim, rot_dim, vdim, kv_rank, window):
    """Loud keys placed so that the last query that sees one and the first that does not fall inside a prompt portion for one key
    and are single decoded tokens for another, and for a third inside a portion of two tokens; a window one longer or shorter
    gives other rows among the portions and among the decoded tokens (checked on the plain side)."""
    width, total, decode_from = 64, 300, 262
    entry = vh.latent(heads, dim, rot_dim, vdim, kv_rank, 0.5, 10000.0, window)
    part = mixer_part(entry, width)
    w = part_weights(part, dtype, 30, 0.12)
    x = rand((total, width), dtype, 50)
    in_prompt, in_pair, in_decode = 150 - window, 201 - window, decode_from + 10 - window
    loud_latent(w, x, entry["mixer"], (in_prompt, in_pair, in_decode))
    part.load(w)
    harness = Harness([part.cache_need()], dtype, page_size=8, num_pages=48, max_seqs=2, max_len=512)
    cuts = [(0, 3), (3, 5), (5, 130), (130, 131), (131, 200), (200, 202), (202, decode_from)] + [(i, i + 1) for i in range(decode_from, total)]
    got = []
    for start, end in cuts:
        ctx = harness.context({"r": end - start})
        ctx.dtype = dtype
        got.append(part.forward(x[start:end].contiguous(), ctx, harness.view(ctx, 0)).clone())
    xd, wd = x.double().cpu(), {k: v.double().cpu() for k, v in w.items()}
    expected = run_plain(entry, wd, xd)
    scale = float(expected.abs().max())
    assert close(torch.cat(got), expected, dtype)
    for other in (window + 1, window - 1):
        shifted = run_plain(vh.latent(heads, dim, rot_dim, vdim, kv_rank, 0.5, 10000.0, other), wd, xd)
        apart = (shifted - expected).abs().amax(dim=1)
        assert float(apart[131:200].max()) > 0.05 * scale and float(apart[decode_from:].max()) > 0.05 * scale
        assert float(apart[200:202].max()) > 0.05 * scale


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 16, 24), (8, 2, 64, 64), (3, 1, 48, 32), (2, 2, 128, 128)])
def test_a_far_key_and_the_sink_decide(dtype, heads, kv_heads, dim, vdim):
    """Attention over the whole sequence with most scores far below the sink: a loud key near the start takes the weight of every
    later query, in a prompt portion and in tokens decoded 300 positions on, where the query's temperature has grown; without
    the sink, or with the temperature left out, the rows would be others."""
    width, total, decode_from = 64, 320, 300
    entry = vh.sink(heads, kv_heads, dim, vdim, 1.5 * dim ** -0.5, 0.3, 16)
    part = mixer_part(entry, width)
    w = part_weights(part, dtype, 31, 0.05)
    x = rand((total, width), dtype, 51)
    for name, factor in (("l0.mix.q", 1.0), ("l0.mix.k", -1.0)):
        w[name].view(-1, dim, width)[:, -2:, 0] = 2.0 * factor
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
    no_sink = dict(wd, **{"l0.mix.sink": torch.full((heads,), -1e4, dtype=plain.F64)})
    assert float((run_plain(entry, no_sink, quiet)[decode_from:] - run_plain(entry, wd, quiet)[decode_from:]).abs().max()) > 0.02 * scale
    cold = dict(entry, mixer=dict(entry["mixer"], q_temp=None))
    assert float((run_plain(cold, wd, xd)[decode_from:] - expected[decode_from:]).abs().max()) > 0.01 * scale


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [44, 96, 256])
@pytest.mark.parametrize("rows", [1, 6, 150])
def test_transition_and_two_norm_block(dtype, width, rows):
    """The mix with the embedding output, entered twice with one and two outputs pending, followed by the norms that receive
    its vector; the norms of a parallel block as one kernel."""
    from types import SimpleNamespace

    from miniserve_b200.parts import BLOCKS, NORMS, TRANSITIONS, PartSpec, StreamVector
    from miniserve_b200.parts.context import StepContext

    part = TRANSITIONS.build(PartSpec("reinjection", dict(hidden_size=width, times=2, in_name="in", step_name="step")))
    w = {"in": rand((width, 2 * width), dtype, 1, (2 * width) ** -0.5), "step": rand((2, width), torch.float32, 2)}
    part.load(w)
    wd = {f"loop.{k}": v.double().cpu() for k, v in w.items()}
    memo = {}
    ctx = SimpleNamespace(memo=memo, device=torch.device("cuda"), dtype=dtype, n_tokens=rows)
    ctx.buffer = lambda *args: StepContext.buffer(ctx, *args)
    norms = [NORMS.build(PartSpec("layer", dict(name=f"n{i}", size=width, eps=1e-5))) for i in range(2)]
    for i, norm in enumerate(norms):
        norm.load({f"n{i}": 1 + rand((width,), dtype, 3 + i, 0.3), f"n{i}.b": rand((width,), dtype, 5 + i, 0.3)})
    seen = []
    mixer = SimpleNamespace(forward=lambda x, ctx, cache: seen.append(x.clone()) or x)
    feed_forward = SimpleNamespace(forward=lambda x, ctx: seen.append(x.clone()) or x)
    block = BLOCKS.build(PartSpec("parallel_two_norms"), mixer=mixer, feed_forward=feed_forward, mixer_norm=norms[0], feed_forward_norm=norms[1])
    stream = rand((rows, width), torch.float32, 9)
    embedded = stream.double().cpu()
    part.remember(stream, ctx)
    a, b = rand((rows, width), dtype, 10), rand((rows, width), dtype, 11)
    x = embedded
    for number, pending in ((0, a), (1, (a, b))):
        plain_pending = a.double().cpu() if number == 0 else a.double().cpu() + b.double().cpu()
        x = plain.enter_pass(x + plain_pending, embedded, wd, number)
        handed = part.enter(stream, pending, ctx, number)
        assert isinstance(handed, StreamVector)
        seen.clear()
        out = block.forward(stream, handed, ctx, None)
        assert isinstance(out, tuple) and len(out) == 2
        assert close(stream, x, dtype)
        x = stream.double().cpu()                   # (go on from the engine's own stream)
        for got, norm in zip(seen, norms):
            assert close(got, plain.layer_norm(x, norm.weight.double().cpu(), norm.bias.double().cpu(), 1e-5), dtype)


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
        config, weights = vh.load_folder(folder)
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
# lengths at the borders of pages of 8 and 16 tokens, of key tiles of 32 and of the windows of 9, 13, 22, 37 and 50 tokens; a
# single token; a few hundred
LENGTHS = (1, 9, 10, 13, 14, 16, 17, 23, 33, 38, 51, 64, 65, 150, 230)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,page_size", [("a", 8), ("b", 16), ("c", 16), ("b", 4), ("c", 64), ("d", 8)])
@pytest.mark.parametrize("cutting", list(CUTTINGS))
def test_cuttings_against_plain(tmp_path, request, dtype, name, page_size, cutting):
    """Whole prompts; last tokens decoded one by one; portions down to two tokens; unequal requests batched together in a pool
    so small that pages and slots are used again: always the logits of the plain whole-sequence computation."""
    folder = vh.make_folder(tmp_path, name, seed=11)
    vocab = vh.CONFIGS[name]["vocab"]
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
    import random

    rng = random.Random(100 + seed)
    config = vh.random_config(rng)
    folder = vh.make_folder(tmp_path, f"random{seed}", seed=3, config=config)
    requests = {f"r{i}": helpers.random_tokens(config["vocab"], n, seed=40 + i) for i, n in enumerate((1, 7, 18, 40, 90))}
    steps = CUTTINGS[rng.choice(["tail", "portions", "mixed"])](requests)
    page_size = rng.choice([4, 8, 16, 32])
    runtime = build(folder, dtype, helpers.max_live_tokens(steps, granule=64) // page_size, page_size)
    check(folder, dtype, requests, helpers.collect(steps, replay(runtime, steps)))


@pytest.mark.parametrize("name,page_size", [("a", 8), ("c", 16)])
def test_float32_logits_do_not_depend_on_cutting_or_batch(tmp_path, name, page_size):
    folder = vh.make_folder(tmp_path, name, seed=16)
    vocab = vh.CONFIGS[name]["vocab"]
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
                assert float((results[cutting][rid][position] - alone).abs().max()) <= 2e-6 * scale, (rid, position, cutting)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_prefill_against_decoding_every_token(tmp_path, dtype, name):
    """The same sequence as one prompt and token by token from its first token on: a long decode over many pages, every window
    passed, pages given back and taken again."""
    folder = vh.make_folder(tmp_path, name, seed=12)
    tokens = helpers.random_tokens(vh.CONFIGS[name]["vocab"], 230, seed=500)
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
    """Seven requests live at once, decoded in steps of single tokens whose live set changes (captured graphs with padding rows
    when graphs are on)."""
    folder = vh.make_folder(tmp_path, "c", seed=13)
    vocab = vh.CONFIGS["c"]["vocab"]
    prompt_lens = {f"m{i}": n for i, n in enumerate((3, 1, 17, 40, 9, 64, 25))}
    requests = {rid: helpers.random_tokens(vocab, n + 11, seed=600 + i) for i, (rid, n) in enumerate(prompt_lens.items())}
    steps = helpers.cut_many_live(requests, prompt_lens, seed=2)
    runtime = build(folder, dtype, 7 * 6, 16, max_seqs=7, execution=execution)
    got = helpers.collect(steps, replay(runtime, steps))
    if execution == "cuda_graph":
        assert runtime.step_function.graph_replays > 0
    check(folder, dtype, requests, got, {rid: range(prompt_lens[rid] - 1, len(requests[rid])) for rid in requests})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("execution", ["eager", "cuda_graph"])
def test_greedy_generation_through_the_scheduler(tmp_path, dtype, execution):
    """``LLM.generate``: the engine's own entry point, scheduler (chunked prompts, a token budget that forces portions, more
    prompts than state slots) and sampler; every generated token is the plain implementation's choice, or as good as it
    within rounding."""
    from miniserve_b200.engine.llm import LLM
    from miniserve_b200.sampling import SamplingParams

    folder = vh.make_folder(tmp_path, "a", seed=14)
    config, weights = vh.load_folder(folder)
    prompts = [helpers.random_tokens(config["vocab"], n, seed=700 + n) for n in (1, 5, 30, 77)]
    llm = LLM(str(folder), dtype=dtype, kv_block_size=8, num_kv_blocks=48, max_num_seqs=3, max_num_batched_tokens=24,
              decode_execution=execution)
    results = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=24))
    for prompt, result in zip(prompts, results):
        assert len(result.token_ids) == 24                     # (past both windows, whatever the prompt)
        sequence = list(prompt) + list(result.token_ids)
        logits = plain.forward(sequence, weights, config)
        for at, produced in enumerate(result.token_ids):
            row = logits[len(prompt) + at - 1]
            best = int(torch.argmax(row))
            assert produced == best or float(row[best] - row[produced]) <= 2 * bound_of(dtype, row), (produced, best)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program_and_command_line(tmp_path, dtype):
    """``bin/trace_run`` and ``python -m miniserve_b200.generate`` on a Venarax folder, as a user runs them."""
    folder = vh.make_folder(tmp_path, "d", seed=15)
    vocab = vh.CONFIGS["d"]["vocab"]
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
