"""A plain, slow restatement of the Parunex decoder in float64 torch on the CPU: one function per mechanism, whole sequences,
softmax position by position, the recurrence walked token by token.  It shares no code with the package; the tests compare the
engine with it.

Notation: ``x`` is the residual stream ``[T, width]``, ``h`` a sublayer's input, ``w`` maps tensor names to float64 tensors,
``m`` is a mixer's section of the ``config.json`` mapping ``config``.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def dynamic_tanh(x, alpha, weight, bias):
    """The norm of this design: entry by entry, no statistics of the row."""
    return torch.tanh(alpha * x) * weight + bias


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def frequencies(rot):
    """``base^(-2i / dims)``; with ``scaling`` slow turns are slowed down further by ``factor``: wavelengths below original / high
    stay, those above original / low are divided, and between the two the frequency is a mix whose share runs from 0 to 1."""
    dims, base, scaling = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            factor, low, high, original = (float(scaling[key]) for key in ("factor", "low", "high", "original"))
            wavelength = 2.0 * math.pi / f
            if wavelength > original / low:
                f = f / factor
            elif wavelength >= original / high:
                share = (original / wavelength - low) / (high - low)
                f = (1.0 - share) * f / factor + share * f
        out.append(f)
    return out


def rotate_halves(x, rot, first_position=0):
    """Entries i and i + dims / 2 (i < dims / 2) of the last dimension turn together; entries behind ``dims`` stay
    (``x [T, ..., d]``, row t at position ``first_position + t``)."""
    half = int(rot["dims"]) // 2
    out = x.clone()
    for i, f in enumerate(frequencies(rot)):
        for t in range(x.shape[0]):
            a = (first_position + t) * f
            u, v = x[t, ..., i], x[t, ..., i + half]
            out[t, ..., i] = u * math.cos(a) - v * math.sin(a)
            out[t, ..., i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def capped(score, cap):
    return score if not cap else cap * torch.tanh(score / cap)


def softmax_rows(scores, sink):
    """Softmax over one row of scores with one more term ``exp(sink)`` in the denominator that has no value."""
    peak = max(float(scores.max()), float(sink))
    e = torch.exp(scores - peak)
    return e / (e.sum() + math.exp(float(sink) - peak))


def mixed_values(v, first, share):
    """What a layer attends to where an earlier layer's values of the same tokens are mixed in."""
    return v if first is None else (1.0 - share) * v + share * first


def attention(h, w, p, m, eps, shared):
    """``shared``: the values of the first layer that mixes them, once it has run (key ``first_values``)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def project(name):
        return h @ w[p + name].T + w[p + name + ".b"]

    q = rotate_halves(project("q").view(T, H, d), m["rot"])
    k = rotate_halves(project("k").view(T, G, d), m["rot"])
    v = project("v")
    if m.get("v_mix"):
        if "first_values" in shared:
            v = mixed_values(v, shared["first_values"], w[p + "vmix"])
        else:
            shared["first_values"] = v
    v = v.view(T, G, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for i in range(T):
        for head in range(H):
            g = head // (H // G)
            s = capped((k[:i + 1, g] @ q[i, head]) * m["scale"], m.get("softcap"))
            out[i, head] = softmax_rows(s, w[p + "sink"][head]) @ v[:i + 1, g]
    out = out * torch.sigmoid(h @ w[p + "g"].T)[..., None]
    return out.reshape(T, H * dv) @ w[p + "o"].T


def key_decays(h, w, p, m):
    """One decay per head and key channel, ``sigmoid(z)^(1 / tau)``."""
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return torch.sigmoid(z).pow(1.0 / m["tau"]).view(h.shape[0], m["heads"], m["dim"])


def gated_linear_attention(h, w, p, m, eps, shared=None):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    decay = key_decays(h, w, p, m)
    S = torch.zeros(H, d, dv, dtype=h.dtype)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    out = rms_norm(out, w[p + "norm"], eps).reshape(T, H * dv)
    return (out * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"attention": attention, "gla": gated_linear_attention}


def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def chosen_experts(scores, router):
    """The experts one token uses, best first: groups are ranked by the sum of their two largest scores."""
    experts, top = router["experts"], router["top"]
    groups = router.get("groups") or dict(count=1, keep=1)
    size = experts // groups["count"]
    rank = [sum(sorted((float(s) for s in scores[g * size:(g + 1) * size]), reverse=True)[:2]) for g in range(groups["count"])]
    kept = sorted(range(groups["count"]), key=lambda g: (-rank[g], g))[:groups["keep"]]
    open_ = [e for e in range(experts) if e // size in kept]
    return sorted(open_, key=lambda e: (-float(scores[e]), e))[:top]


def mixture(h, w, p, mlp):
    router = mlp["router"]
    scores = torch.sigmoid(h @ w[p + "router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = chosen_experts(scores[t], router)
        total = sum(scores[t, e] for e in chosen) + 1e-20
        for e in chosen:
            out[t] += scores[t, e] / total * router["scale"] * expert(h[t], w, f"{p}e{e}.")
    return out


def feed_forward(h, w, p, mlp):
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp)


def norm_of(x, w, name):
    return dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])


def layer(x, w, index, entry, eps, shared):
    p = f"l{index}."
    x = x + MIXERS[entry["type"]](norm_of(x, w, p + "norm1"), w, p + "mix.", entry["mixer"], eps, shared)
    if entry.get("mlp"):
        x = x + feed_forward(norm_of(x, w, p + "norm2"), w, p + "mlp.", entry["mlp"])
    return x


def forward(tokens, w, config, return_layers=False):
    x = w["embed"][tokens] * config["embedding"]["scale"]
    streams, shared = [], {}
    for index, entry in enumerate(config["layers"]):
        x = layer(x, w, index, entry, config["norm"]["eps"], shared)
        streams.append(x)
    logits = norm_of(x, w, "final.norm") @ w["head"].T
    return (logits, torch.stack(streams)) if return_layers else logits
