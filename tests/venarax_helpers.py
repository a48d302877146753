"""Small Venarax configurations for the tests, with weights made so that every vector of the design moves its formula: biases and
weights of the layer norms away from their neutral values, sinks between -1.5 and 2.5, pass vectors that tell the passes apart, a
mixing matrix that keeps part of the stream."""

from __future__ import annotations

import json
from pathlib import Path

import torch


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, window):
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
                                                    rot=dict(base=base, dims=rot_dim), mask=dict(size=window)))


def sink(heads, kv_heads, dim, vdim, scale, coef, every):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale,
                                             q_temp=dict(coef=coef, every=every)))


def layer(mix, ff, limit=1.0):
    return dict(mix, mlp=None if ff is None else dict(kind="dense", ff=ff, limit=limit))


def model(vocab, width, eps, loop, layers):
    return dict(architecture="Venarax", vocab=vocab, width=width, norm=dict(eps=eps),
                loop=None if loop is None else dict(start=loop[0], stop=loop[1], times=loop[2]), layers=layers)


# Sizes that differ from one another everywhere: values of another size than keys in both mixers, windows that are no multiple of
# a page, query heads over fewer key heads, a temperature that steps every 7 positions, limits above and below the usual values,
# a layer without feed-forward, two layers in the middle repeated three times.
VENARAX_A = model(203, 96, 1e-5, (1, 3, 3), [
    layer(sink(4, 2, 16, 24, 0.3, 0.4, 7), 56, 0.7),
    layer(latent(5, 12, 4, 10, 24, 0.28, 500.0, 13), None),
    layer(sink(6, 3, 20, 12, 0.25, 0.15, 11), 40, 2.5),
    layer(latent(2, 24, 8, 16, 40, 0.2, 20000.0, 22), 64, 1.3),
])
# One head everywhere, a window of one token (a token sees itself alone) and one that no request of the tests outgrows, a
# temperature that steps at every position and one whose factor falls, a rotation of one pair, a single pass over everything.
VENARAX_B = model(157, 72, 1e-6, (0, 4, 1), [
    layer(latent(1, 10, 2, 14, 12, 0.4, 100.0, 1), 20, 0.4),
    layer(sink(1, 1, 12, 6, 0.4, 0.7, 1), None),
    layer(latent(3, 6, 6, 6, 30, 0.3, 10000.0, 1000), 18, 1.0),
    layer(sink(5, 5, 6, 6, 0.17, -0.1, 5), 24, 5.0),
])
# Sizes of the kind real models have in small: latents of 64 and 128 with a rotated part of 16 and 32 (the tensor-core latent kernels),
# heads of 64 and 128 (the tensor-core attention kernels), keys of 64 over values of 32 (the kernel for any size), eight query
# heads per key head; the last two layers repeated.
VENARAX_C = model(300, 128, 1e-6, (2, 4, 2), [
    layer(latent(8, 32, 16, 64, 64, 0.15, 10000.0, 50), 256, 1.0),
    layer(sink(8, 1, 64, 64, 0.125, 0.3, 32), 128, 0.8),
    layer(sink(4, 2, 128, 128, 0.09, 0.25, 16), None),
    layer(latent(4, 64, 32, 32, 128, 0.1, 1000000.0, 37), 192, 1.5),
])
# Widths that are no multiple of eight, head sizes that are odd, an inner size that is no multiple of eight, no repeated run.
VENARAX_D = model(120, 44, 1e-5, None, [
    layer(latent(3, 7, 2, 5, 18, 0.33, 2000.0, 9), 30, 0.9),
    layer(sink(3, 3, 7, 9, 0.35, 0.5, 4), 18, 1.1),
    layer(latent(2, 9, 4, 11, 21, 0.3, 50.0, 30), 12, 2.0),
])
CONFIGS = {"a": VENARAX_A, "b": VENARAX_B, "c": VENARAX_C, "d": VENARAX_D}


def random_config(rng) -> dict:
    """A configuration drawn from ``rng`` (a ``random.Random``): one to five layers of either kind in any order, every size, window,
    temperature and limit and the repeated run drawn independently of one another."""
    width = rng.choice([20, 40, 64, 72])
    layers = []
    for _ in range(rng.choice([1, 2, 3, 4, 5])):
        ff, limit = rng.choice([None, 16, 24, 50]), rng.choice([0.3, 1.0, 4.0])
        if rng.random() < 0.5:
            layers.append(layer(latent(rng.choice([1, 2, 3, 5]), rng.choice([4, 6, 9, 16]), rng.choice([2, 4, 6, 16]),
                                       rng.choice([4, 5, 12, 16]), rng.choice([8, 16, 21, 40]), rng.uniform(0.1, 0.5),
                                       rng.choice([30.0, 10000.0]), rng.choice([1, 2, 5, 8, 16, 17, 33, 500])), ff, limit))
        else:
            kv = rng.choice([1, 2, 3])
            layers.append(layer(sink(kv * rng.choice([1, 2, 4]), kv, rng.choice([4, 6, 9, 16]), rng.choice([4, 5, 8, 12]),
                                     rng.uniform(0.1, 0.5), rng.uniform(-0.2, 0.8), rng.choice([1, 3, 8, 64])), ff, limit))
    loop = None
    if rng.random() < 0.8:
        start = rng.randrange(0, len(layers))
        loop = (start, rng.randrange(start + 1, len(layers) + 1), rng.choice([1, 2, 3]))
    return model(rng.choice([50, 131]), width, rng.choice([1e-5, 1e-6]), loop, layers)


def _normal(shape, seed, std, mean=0.0):
    return mean + std * torch.randn(shape, generator=torch.Generator().manual_seed(seed))


def shape_weights(tensors: dict, config: dict) -> None:
    """In place, see the head of this file."""
    width = config["width"]

    def put(name, value):
        tensors[name] = value.to(tensors[name].dtype)

    for index, entry in enumerate(config["layers"]):
        p, seed = f"l{index}.", 100 * index
        for k, name in enumerate(("norm1", "norm2")):
            if p + name in tensors:
                put(p + name, _normal((width,), seed + 2 * k + 1, 0.3, 1.0))
                put(p + name + ".b", _normal((width,), seed + 2 * k + 2, 0.3))
        if entry["type"] == "attention":
            heads = entry["mixer"]["heads"]
            put(p + "mix.sink", torch.linspace(-1.5, 2.5, heads) if heads > 1 else torch.tensor([0.8]))
            for k, name in enumerate(("q.norm", "k.norm")):
                put(p + "mix." + name, _normal(tuple(tensors[p + "mix." + name].shape), seed + 10 + k, 0.3, 1.0))
    put("embed", _normal(tuple(tensors["embed"].shape), 5, 1.0))
    put("final.norm.b", _normal((width,), 7, 0.2))
    if "loop.in" in tensors:
        mix = _normal((width, 2 * width), 8, 0.4 / (2 * width) ** 0.5)
        mix[:, :width] += 0.6 * torch.eye(width)
        put("loop.in", mix)
        put("loop.step", _normal(tuple(tensors["loop.step"].shape), 9, 0.5))


def make_folder(tmp_path, name: str, seed: int = 0, stored_dtype: str = "bfloat16", matrix_std: float = 0.1, config=None) -> Path:
    import miniserve_b200  # noqa: F401
    from miniserve_b200.weights import random_tensors
    from safetensors.torch import save_file

    folder = Path(tmp_path) / f"venarax_{name}_{seed}_{stored_dtype}"
    if not folder.exists():
        folder.mkdir(parents=True)
        config = CONFIGS[name] if config is None else config
        tensors = random_tensors(config, seed, stored_dtype, matrix_std)
        shape_weights(tensors, config)
        (folder / "config.json").write_text(json.dumps(config, indent=1))
        save_file({k: v.contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))
    return folder


def load_folder(folder):
    from safetensors.torch import load_file

    config = json.loads((Path(folder) / "config.json").read_text())
    weights = {k: v.to(torch.float64) for k, v in load_file(str(Path(folder) / "model.safetensors")).items()}
    return config, weights
