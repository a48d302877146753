"""Small Parunex configurations for the tests, with weights made so that every tensor of the design moves its formula: alphas, weights
and biases of the norms away from their neutral values, sinks between -1.5 and 2.5, biases of the size of the projections, shares of
the kept values some of them negative, decays that remember a dozen tokens or more and differ from channel to channel, and
routers whose choices are clear whatever the rounding."""

from __future__ import annotations

import json
from pathlib import Path

import torch


def rot(base, dims, scaling=None):
    out = dict(base=base, dims=dims)
    if scaling:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def attention(heads, kv_heads, dim, vdim, scale, rotation, softcap, v_mix=True):
    mixer = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=rotation, v_mix=v_mix)
    if softcap is not None:
        mixer["softcap"] = softcap
    return dict(type="attention", mixer=mixer)


def gla(heads, dim, vdim, tau, rank):
    """``rank`` is what the tensors of ``l<i>.mix.a1`` and ``.a2`` say; a checkpoint's ``config.json`` need not carry it."""
    return dict(type="gla", mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=tau, rank=rank))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, scale, count=1, keep=1):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale, groups=dict(count=count, keep=keep)))


def layer(mix, mlp):
    return dict(mix, mlp=mlp)


def model(vocab, width, scale, eps, layers):
    return dict(architecture="Parunex", vocab=vocab, width=width, embedding=dict(scale=scale), norm=dict(eps=eps), layers=layers)


# Sizes that differ from one another everywhere; three attention layers of which the last two take the first one's values (as four
# heads of 12 in one of them and as two of 24 in the others); frequencies of all three kinds; a layer without a feed-forward.  (The
# recurrence's first output is (q . k) v, which the norm over a head brings back to size: with a tiny eps a product near zero
# would magnify every rounding before it.)
PARUNEX_A = model(203, 96, 3.0, 1e-2, [
    layer(attention(4, 2, 16, 24, 0.3, rot(500.0, 12, (4.0, 1.0, 4.0, 64)), 1.5), moe(6, 2, 20, 1.7, 3, 2)),
    layer(gla(3, 20, 12, 16.0, 5), dense(56)),
    layer(attention(8, 4, 20, 12, 0.25, rot(10000.0, 20), 2.0), None),
    layer(gla(2, 12, 28, 4.0, 9), moe(8, 3, 24, 0.6, 2, 1)),
    layer(attention(6, 2, 24, 24, 0.2, rot(300.0, 8, (2.0, 2.0, 5.0, 40)), None), dense(44)),
])
# One head everywhere, one group, one expert per token, all experts, no rotation, no soft cap, values that are not mixed (two layers
# with values of other sizes), tau of one, a recurrence first and last.
PARUNEX_B = model(157, 72, 1.0, 1e-6, [
    layer(gla(1, 10, 14, 1.0, 1), moe(4, 1, 12, 2.0)),
    layer(attention(1, 1, 12, 6, 0.4, rot(100.0, 0), None, False), dense(20)),
    layer(attention(5, 5, 6, 10, 0.35, rot(20000.0, 2), 2.0, False), moe(3, 3, 10, 1.0, 3, 3)),
    layer(gla(5, 6, 7, 9.0, 12), None),
])
# Sizes of the kind real models have in small: heads of 64 and 128 (the tensor-core attention kernels), keys of 128 over values of 48
# (the kernel for any size), eight query heads per key head, keys of 64 and 128 in the recurrences.
PARUNEX_C = model(300, 128, 4.0, 5e-3, [
    layer(gla(4, 64, 32, 16.0, 16), dense(256)),
    layer(attention(8, 1, 64, 64, 0.125, rot(1000000.0, 64, (8.0, 1.0, 4.0, 128)), 20.0), moe(16, 4, 32, 2.5, 4, 2)),
    layer(attention(4, 2, 128, 32, 0.09, rot(10000.0, 64), 30.0), dense(128)),
    layer(gla(2, 128, 64, 8.0, 8), moe(8, 2, 48, 1.5, 2, 1)),
    layer(attention(4, 1, 96, 64, 0.1, rot(50000.0, 32, (4.0, 1.0, 4.0, 256)), 50.0), moe(12, 3, 32, 2.0, 4, 3)),
])
# Widths and inner sizes that are no multiple of eight, odd head sizes, attention alone.
PARUNEX_D = model(120, 44, 2.5, 1e-5, [
    layer(attention(3, 3, 7, 9, 0.35, rot(50.0, 4), 4.0), dense(30)),
    layer(attention(3, 1, 9, 27, 0.3, rot(80.0, 6, (3.0, 1.0, 3.0, 30)), 6.0), moe(5, 2, 18, 1.3)),
    layer(attention(6, 3, 11, 9, 0.3, rot(2000.0, 10), 8.0), None),
])
# Recurrences alone (no pages are needed, only state slots).
PARUNEX_E = model(131, 64, 2.0, 1e-4, [
    layer(gla(4, 16, 24, 16.0, 6), dense(48)),
    layer(gla(2, 36, 8, 2.0, 3), moe(9, 2, 16, 1.1, 3, 1)),
    layer(gla(3, 5, 40, 30.0, 8), dense(24)),
])
CONFIGS = {"a": PARUNEX_A, "b": PARUNEX_B, "c": PARUNEX_C, "d": PARUNEX_D, "e": PARUNEX_E}


def random_config(rng) -> dict:
    """A configuration drawn from ``rng`` (a ``random.Random``): one to five layers of either kind in any order, every size and constant
    drawn independently of one another (values that are mixed have one total size)."""
    width = rng.choice([56, 64, 72, 100])
    layers, marked = [], 0
    for _ in range(rng.choice([1, 2, 3, 4, 5])):
        if rng.random() < 0.55:
            kv = rng.choice([1, 2, 4])
            dims = rng.choice([0, 2, 4])
            scaling = rng.choice([None, (rng.choice([2.0, 8.0]), 1.0, rng.choice([2.0, 4.0]), rng.choice([16, 100]))]) if dims else None
            mix = attention(kv * rng.choice([1, 2, 3]), kv, rng.choice([4, 6, 9, 16, 32]), 16 // kv, rng.uniform(0.1, 0.5),
                            rot(rng.choice([30.0, 10000.0]), dims, scaling), rng.choice([None, 1.5, 4.0, 30.0]), rng.random() < 0.8)
        else:
            mix = gla(rng.choice([1, 2, 3, 5]), rng.choice([4, 7, 16, 36]), rng.choice([4, 5, 12, 16]), rng.choice([1.0, 3.0, 16.0]),
                      rng.choice([1, 4, 11]))
        kind = rng.random()
        if kind < 0.2:
            mlp = None
        elif kind < 0.5 or marked > 20:
            mlp = dense(rng.choice([16, 24, 50]))
        else:
            count, size = rng.choice([1, 2, 3]), rng.choice([1, 2, 4])
            keep = rng.randrange(1, count + 1)
            mlp = moe(count * size, rng.randrange(1, min(3, keep * size) + 1), rng.choice([8, 20, 26]), rng.uniform(0.5, 3.0), count, keep)
            marked += count * size
        layers.append(layer(mix, mlp))
    return model(rng.choice([50, 131]), width, rng.choice([1.0, 2.5]), rng.choice([1e-2, 0.1]), layers)


def _normal(shape, seed, std, mean=0.0):
    return mean + std * torch.randn(shape, generator=torch.Generator().manual_seed(seed))


def shape_weights(tensors: dict, config: dict) -> None:
    """In place, see the head of this file.  Every routed layer has columns of its own in the stream: a token's embedding carries
    descending marks in the columns of the experts id, id + 1, ... (mod the number of experts), as many as the layer chooses, and nothing in
    the layer's other columns; no sublayer writes there, the norms before the feed-forwards leave those columns to the tanh
    alone, and the router reads only its own (so unmarked experts tie exactly, which the lower index wins)."""
    width, vocab = config["width"], config["vocab"]

    def put(name, value):
        tensors[name] = value.to(tensors[name].dtype)

    embed = _normal((vocab, width), 5, 1.0 / config["embedding"]["scale"])
    ids, column, marks = torch.arange(vocab), 0, []
    for index, entry in enumerate(config["layers"]):
        p, m, seed = f"l{index}.", entry["mixer"], 100 * index
        for k, name in enumerate(("norm1", "norm2")):
            if p + name in tensors:
                put(p + name, _normal((width,), seed + 2 * k + 1, 0.3, 1.0))
                put(p + name + ".b", _normal((width,), seed + 2 * k + 2, 0.3))
                put(p + name + ".alpha", torch.tensor(0.45 + 0.2 * k + 0.07 * (index % 3)))
        if entry["type"] == "attention":
            put(p + "mix.sink", torch.linspace(-1.5, 2.5, m["heads"]) if m["heads"] > 1 else torch.tensor([0.8]))
            for k, name in enumerate("qkv"):
                put(p + f"mix.{name}.b", _normal(tuple(tensors[p + f"mix.{name}.b"].shape), seed + 10 + k, 0.4))
            put(p + "mix.g", _normal(tuple(tensors[p + "mix.g"].shape), seed + 14, width ** -0.5))
            if p + "mix.vmix" in tensors:
                put(p + "mix.vmix", torch.tensor([0.6, -0.2, 0.8][index % 3]))
        else:
            put(p + "mix.norm", _normal((m["vdim"],), seed + 20, 0.3, 1.0))
            put(p + "mix.a1", _normal(tuple(tensors[p + "mix.a1"].shape), seed + 21, width ** -0.5))
            put(p + "mix.a2", _normal(tuple(tensors[p + "mix.a2"].shape), seed + 22, 1.5 * m["rank"] ** -0.5))
            # decays around 0.93: a dozen tokens are remembered whatever tau is
            keep = 0.93 ** m["tau"]
            put(p + "mix.a2.b", _normal(tuple(tensors[p + "mix.a2.b"].shape), seed + 23, 0.7, float(torch.logit(torch.tensor(keep)))))
        if entry["mlp"] and entry["mlp"]["kind"] == "moe":
            router = entry["mlp"]["router"]
            total, top = router["experts"], router["top"]
            embed[:, column:column + total] = 0.0
            for choice in range(top):
                embed[ids, column + (ids + choice) % total] = 2.4 * 0.6 ** choice / config["embedding"]["scale"]
            weight = torch.zeros(total, width)
            weight[:, column:column + total] = 3.0 * torch.eye(total)
            put(p + "mlp.router", weight)
            marks.append((p, column, column + total))
            column += total
    if column > width - 8:
        raise ValueError("the width is too small for the marks of all routed layers")
    for name in tensors:
        if name.endswith((".mix.o", ".down")):
            tensors[name][:column] = 0.0
    for p, start, stop in marks:
        tensors[p + "norm2"][start:stop] = 1.0
        tensors[p + "norm2.b"][start:stop] = 0.0
    put("embed", embed)
    put("final.norm.b", _normal((width,), 7, 0.2))
    put("final.norm.alpha", torch.tensor(0.6))


def make_folder(tmp_path, name: str, seed: int = 0, stored_dtype: str = "bfloat16", matrix_std: float = 0.12, config=None) -> Path:
    import miniserve_b200  # noqa: F401
    from miniserve_b200.weights import random_tensors
    from safetensors.torch import save_file

    folder = Path(tmp_path) / f"parunex_{name}_{seed}_{stored_dtype}"
    if not folder.exists():
        folder.mkdir(parents=True)
        config = CONFIGS[name] if config is None else config
        tensors = random_tensors(config, seed, stored_dtype, matrix_std)
        shape_weights(tensors, config)
        stored = json.loads(json.dumps(config))
        for entry in stored["layers"]:
            entry["mixer"].pop("rank", None)            # (left to the tensors' shapes)
        (folder / "config.json").write_text(json.dumps(stored, indent=1))
        save_file({k: v.contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))
    return folder


def load_folder(folder):
    from safetensors.torch import load_file

    config = json.loads((Path(folder) / "config.json").read_text())
    weights = {k: v.to(torch.float64) for k, v in load_file(str(Path(folder) / "model.safetensors")).items()}
    return config, weights
