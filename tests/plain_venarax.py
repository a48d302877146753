"""A plain, slow restatement of the Venarax decoder in float64 torch on the CPU: one function per mechanism, whole sequences,
every key and value of every head formed, softmax position by position.  It shares no code with the package; the tests
compare the engine with it.

Notation: ``x`` is the residual stream ``[T, width]``, ``h`` a mixer's input, ``w`` maps tensor names to float64 tensors,
``config`` is the ``config.json`` mapping.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def layer_norm(x, weight, bias, eps):
    """The mean taken off, divided by the root of the mean squared deviation (eps inside the root), weight and bias."""
    centered = x - x.mean(dim=-1, keepdim=True)
    return centered / torch.sqrt((centered * centered).mean(dim=-1, keepdim=True) + eps) * weight + bias


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def rotate_pairs(x, rot, first_position=0):
    """Neighbouring entries 2i and 2i + 1 (i < dims / 2) of the last dimension turn by p * base^(-2i / dims) at position p
    (``x [T, ..., d]``, row t at position ``first_position + t``); the entries behind ``dims`` stay."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = (first_position + t) * base ** (-2.0 * i / dims)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[t, ..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def softmax_rows(scores, sink=None):
    """Softmax over one row of scores; ``sink``: one more term exp(sink) in the denominator that has no value."""
    peak = float(scores.max()) if sink is None else max(float(scores.max()), float(sink))
    e = torch.exp(scores - peak)
    total = e.sum() if sink is None else e.sum() + math.exp(float(sink) - peak)
    return e / total


def latent_attention(h, w, prefix, m, eps):
    T = h.shape[0]
    H, dim, rot_dim, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[prefix + "q"].T).view(T, H, dim + rot_dim)
    q_plain, q_rot = q[..., :dim], rotate_pairs(q[..., dim:], m["rot"])
    down = h @ w[prefix + "dkv"].T
    latent = rms_norm(down[:, :rank], w[prefix + "dkv.norm"], eps)
    k_rot = rotate_pairs(down[:, rank:], m["rot"])
    k_plain = (latent @ w[prefix + "uk"].T).view(T, H, dim)
    values = (latent @ w[prefix + "uv"].T).view(T, H, vdim)
    window = (m.get("mask") or {}).get("size") or T
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for i in range(T):
        first = max(0, i - window + 1)
        for head in range(H):
            s = (k_plain[first:i + 1, head] @ q_plain[i, head] + k_rot[first:i + 1] @ q_rot[i, head]) * m["scale"]
            out[i, head] = softmax_rows(s) @ values[first:i + 1, head]
    gated = out.reshape(T, H * vdim) * torch.sigmoid(h @ w[prefix + "g"].T)
    return gated @ w[prefix + "o"].T


def query_temperature(position, temp):
    """The factor of the queries at a position: steps up by the logarithm of how many times ``every`` tokens came before."""
    return 1.0 + temp["coef"] * math.log(math.floor((position + 1) / temp["every"]) + 1.0)


def sink_attention(h, w, prefix, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(h @ w[prefix + "q"].T, w[prefix + "q.norm"], eps).view(T, H, d)       # all heads normed as one row
    k = rms_norm(h @ w[prefix + "k"].T, w[prefix + "k.norm"], eps).view(T, G, d)
    v = (h @ w[prefix + "v"].T).view(T, G, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for i in range(T):
        warm = query_temperature(i, m["q_temp"]) if m.get("q_temp") else 1.0
        for head in range(H):
            g = head // (H // G)
            s = (k[:i + 1, g] @ (warm * q[i, head])) * m["scale"]
            out[i, head] = softmax_rows(s, w[prefix + "sink"][head]) @ v[:i + 1, g]
    return out.reshape(T, H * dv) @ w[prefix + "o"].T


MIXERS = {"latent_attention": latent_attention, "attention": sink_attention}


def feed_forward(h, w, prefix, mlp):
    limit = mlp["limit"]
    g = torch.minimum(h @ w[prefix + "gate"].T, torch.tensor(limit, dtype=h.dtype))
    u = (h @ w[prefix + "up"].T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[prefix + "down"].T


def layer(x, w, index, entry, eps):
    """Both sublayers read the same stream, each through a norm of its own, and are added together."""
    p = f"l{index}."
    update = MIXERS[entry["type"]](layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps), w, p + "mix.", entry["mixer"], eps)
    if entry.get("mlp"):
        update = update + feed_forward(layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps), w, p + "mlp.", entry["mlp"])
    return x + update


def layer_order(config):
    """The layers in the order they run, each with the number of the pass that it opens (None: it opens none)."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def enter_pass(x, embedded, w, t):
    """What comes ahead of pass t: the stream and the embedding output through one matrix, and the pass's own vector."""
    return torch.cat([x, embedded], dim=-1) @ w["loop.in"].T + w["loop.step"][t]


def forward(tokens, w, config, return_layers=False):
    eps = config["norm"]["eps"]
    embedded = w["embed"][tokens]
    x, streams = embedded, []
    for index, opens in layer_order(config):
        if opens is not None:
            x = enter_pass(x, embedded, w, opens)
        x = layer(x, w, index, config["layers"][index], eps)
        streams.append(x)
    logits = layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
    return (logits, torch.stack(streams)) if return_layers else logits
