"""Parunex: a decoder whose layers, in an order that ``config.json`` gives, carry grouped-query attention (biases, a half-split rotation
whose frequencies are scaled by wavelength, scores with a soft cap, a learned sink and a gate per head, values mixed along the
depth) or gated linear attention (a matrix per head with a decay per key channel), and a feed-forward that is a gated layer with
the tanh form of GELU or a mixture of gated experts (sigmoid scores, groups ranked by their two best, weights that add up to a
constant).  The norms are dynamic tanhs: no statistics, entry by entry.  Embeddings are scaled.

Tensor names: ``embed``, ``final.norm``, ``head`` and, for layer i, ``l<i>.norm1``, ``l<i>.norm2`` (each norm with ``.alpha`` and ``.b``
beside it), ``l<i>.mix.{q,q.b,k,k.b,v,v.b,vmix,sink,g,o}`` or ``l<i>.mix.{q,k,v,g,o,norm,a1,a2,a2.b}``, and
``l<i>.mlp.{gate,up,down}`` or ``l<i>.mlp.{router,e<j>.gate,e<j>.up,e<j>.down}``.
"""

from __future__ import annotations

from ..config.model_config import ParunexConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerRun, LayerSpec, ModelSpec, PartSpec

# The design gives positions no upper limit; this is the engine's own bound on a request's length (it sizes the block
# tables of captured decode steps), which `max_model_len` lowers.
NOMINAL_MAX_POSITIONS = 131072


def _attention(m, width: int, eps: float, value_mix) -> PartSpec:
    position = PartSpec("none") if m.rot.dims == 0 else PartSpec("rope", dict(
        head_dim=m.dim, theta=m.rot.base, rotary_dim=m.rot.dims, scaling=m.rot.scaling_dict(), frequencies="float64"))
    return PartSpec("attention", dict(
        hidden_size=width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, qk_norm=False, eps=eps,
        position=position, scale=m.scale, score_softcap=m.softcap, sink="learned", output_gate=True, bias="qkv", value_mix=value_mix,
        q_name="mix.q", k_name="mix.k", v_name="mix.v", o_name="mix.o", gate_name="mix.g", sink_name="mix.sink", mix_name="mix.vmix"))


def _gated_linear_attention(m, width: int, eps: float, where: str) -> PartSpec:
    if m.rank is None:
        raise ValueError(f"{where}mixer: the inner size of the decay's two-step projection comes from 'rank' or from the shapes of "
                         "the checkpoint's tensors; neither was given")
    return PartSpec("gated_linear_attention", dict(
        hidden_size=width, heads=m.heads, head_dim=m.dim, value_dim=m.vdim, rank=m.rank, tau=m.tau, eps=eps, q_name="mix.q",
        k_name="mix.k", v_name="mix.v", g_name="mix.g", o_name="mix.o", norm_name="mix.norm", a_name="mix.a"))


def _feed_forward(mlp, width: int):
    if mlp is None:
        return None
    if mlp.kind == "dense":
        return PartSpec("gated_mlp", dict(hidden_size=width, intermediate_size=mlp.ff, activation="gelu_tanh", gate_name="mlp.gate",
                                          up_name="mlp.up", down_name="mlp.down"))
    return PartSpec("routed_experts", dict(
        hidden_size=width, experts=mlp.experts, top=mlp.top, expert_size=mlp.ff, router_bias=False, activation="silu_glu",
        scoring="sigmoid", groups=(mlp.group_count, mlp.group_keep), group_score="two_largest", normalize=1e-20,
        weight_scale=mlp.scale, router_name="mlp.router", expert_name="mlp.e{index}."))


def build_parunex_spec(config: ParunexConfig) -> ModelSpec:
    width, eps = config.width, config.eps

    def norm(name: str) -> PartSpec:
        return PartSpec("dynamic_tanh", dict(name=name, size=width))

    layers, unused, kept = [], [], False
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        if layer.type == "attention":
            value_mix = None if not layer.mixer.v_mix else "mix" if kept else "keep"
            kept = kept or value_mix is not None
            if value_mix != "mix":
                unused.append(prefix + "mix.vmix")      # a checkpoint may carry it although nothing reads it
            mixer = _attention(layer.mixer, width, eps, value_mix)
        else:
            mixer = _gated_linear_attention(layer.mixer, width, eps, f"layers[{index}].")
        feed_forward = _feed_forward(layer.mlp, width)
        if feed_forward is None:
            unused += [prefix + "norm2", prefix + "norm2.b", prefix + "norm2.alpha"]      # likewise
        layers.append(LayerSpec(prefix=prefix, mixer=mixer, feed_forward=feed_forward, mixer_norm=norm("norm1"),
                                feed_forward_norm=None if feed_forward is None else norm("norm2")))
    return ModelSpec(
        vocab_size=config.vocab, hidden_size=width, embedding_name="embed", layers=tuple(layers),
        order=tuple(LayerRun(index) for index in range(len(layers))), final_norm=norm("final.norm"), output_name="head",
        max_positions=NOMINAL_MAX_POSITIONS, nominal_max_positions=True, optional_names=tuple(unused),
        embedding_scale=config.embedding_scale)


register_architecture("Parunex", ParunexConfig, build_parunex_spec)
