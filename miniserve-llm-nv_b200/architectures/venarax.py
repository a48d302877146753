"""Venarax: a decoder whose layers, in an order that ``config.json`` gives, carry latent attention (an interleaved rotation of a key
part that all heads share, a sliding window, a gate per entry) or grouped-query attention without rotation (queries and keys normed
over the whole projection, a temperature of the queries that grows with the position, a learned sink per head).  Mixer and
feed-forward (a clamped gated activation) read the same stream, each through a layer norm of its own, and are added together.  A
run of layers is repeated (``loop``): before each pass the stream is mixed with the embedding output by one matrix and receives
the pass's vector.

Tensor names: ``embed``, ``loop.in``, ``loop.step``, ``final.norm``, ``final.norm.b``, ``head`` and, for layer i,
``l<i>.norm1``, ``l<i>.norm1.b``, ``l<i>.norm2``, ``l<i>.norm2.b``, ``l<i>.mlp.{gate,up,down}`` and
``l<i>.mix.{q,dkv,dkv.norm,uk,uv,g,o}`` or ``l<i>.mix.{q,k,v,q.norm,k.norm,sink,o}``.
"""

from __future__ import annotations

from ..config.model_config import VenaraxConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerRun, LayerSpec, ModelSpec, PartSpec

# The design gives positions no upper limit; this is the engine's own bound on a request's length (it sizes the block
# tables of captured decode steps), which `max_model_len` lowers.
NOMINAL_MAX_POSITIONS = 131072


def _mixer(kind: str, m, width: int, eps: float) -> PartSpec:
    if kind == "latent_attention":
        position = PartSpec("rope", dict(head_dim=m.rot_dim, theta=m.rot.base, rotary_dim=m.rot.dims, interleaved=True,
                                         frequencies="float64"))
        return PartSpec("latent_attention", dict(
            hidden_size=width, num_heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, kv_rank=m.kv_rank, scale=m.scale,
            eps=eps, position=position, output_gate="entry", window=m.window, q_name="mix.q", dkv_name="mix.dkv",
            latent_norm_name="mix.dkv.norm", uk_name="mix.uk", uv_name="mix.uv", gate_name="mix.g", o_name="mix.o"))
    return PartSpec("attention", dict(
        hidden_size=width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, qk_norm="row", eps=eps,
        position=PartSpec("none"), scale=m.scale, sink="learned", query_temperature=m.temperature, q_name="mix.q", k_name="mix.k",
        v_name="mix.v", o_name="mix.o", q_norm_name="mix.q.norm", k_norm_name="mix.k.norm", sink_name="mix.sink"))


def build_venarax_spec(config: VenaraxConfig) -> ModelSpec:
    width, eps = config.width, config.eps

    def norm(name: str) -> PartSpec:
        return PartSpec("layer", dict(name=name, size=width, eps=eps))

    layers, unused = [], []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        feed_forward = None if layer.mlp is None else PartSpec("gated_mlp", dict(
            hidden_size=width, intermediate_size=layer.mlp.ff, activation="clamped_glu", limit=layer.mlp.limit, gate_name="mlp.gate",
            up_name="mlp.up", down_name="mlp.down"))
        layers.append(LayerSpec(prefix=prefix, mixer=_mixer(layer.type, layer.mixer, width, eps), feed_forward=feed_forward,
                                mixer_norm=norm("norm1"), feed_forward_norm=None if feed_forward is None else norm("norm2"),
                                block=PartSpec("parallel_two_norms")))
        if feed_forward is None:
            unused += [prefix + "norm2", prefix + "norm2.b"]      # a checkpoint may carry them although nothing reads them
    n, transitions = len(layers), ()
    if config.loop is None:
        order = [LayerRun(index) for index in range(n)]
        unused += ["loop.in", "loop.step"]
    else:
        start, stop, times = config.loop
        transitions = (PartSpec("reinjection", dict(hidden_size=width, times=times, in_name="loop.in", step_name="loop.step")),)
        order = [LayerRun(index) for index in range(start)]
        for number in range(times):
            order += [LayerRun(index, enters=(0, number) if index == start else None) for index in range(start, stop)]
        order += [LayerRun(index) for index in range(stop, n)]
    return ModelSpec(
        vocab_size=config.vocab, hidden_size=width, embedding_name="embed", layers=tuple(layers), order=tuple(order),
        final_norm=norm("final.norm"), output_name="head", max_positions=NOMINAL_MAX_POSITIONS, nominal_max_positions=True,
        optional_names=tuple(unused), transitions=transitions)


register_architecture("Venarax", VenaraxConfig, build_venarax_spec)
