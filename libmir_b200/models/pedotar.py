"""Pedotar: a decoder with a layer norm before and behind every sublayer, selective state-space mixers, latent attention,
attention within runs of positions whose heads' weights are mixed, and a run of layers that repeats:
config.json -> ModelSpec.

config.json:
    architecture  "Pedotar"
    vocab, width, norm.eps
    loop          {start, stop, times}: layers start .. stop - 1 run `times` times in a row with the same weights, every
                  pass with a cache or state of its own; before every pass but the first the embedding's output is added
                  to the residual
    layers[i]     {type, mixer, mlp}; tensors of layer i start with "l<i>."
        type "mamba1"            {inner, state, dt_rank, conv}: a selective scan behind a short convolution with a bias
        type "latent_attention"  {heads, dim, rot_dim, vdim, kv_rank, scale, rot {dims, base}}: queries by one
                                 projection, keys and values through one latent per token, half-split rotation of the
                                 rot_dim part; causal
        type "attention"         {heads, kv_heads, dim, vdim, scale, mask {size}}: an RMS norm of every query and key
                                 head (weights q.norm, k.norm), no rotation; a query sees its own run of mask.size
                                 positions; the heads' softmax weights are mixed by a stored matrix (talk [heads, heads])
        mlp       {kind "dense", ff}: down(silu(gate x) * up x), or null
Every norm of the residual and of a sublayer's result is a layer norm with weight and bias (eps = norm.eps).
Tensor names: embed (also the output head), l<i>.norm1(.b), l<i>.norm1b(.b), l<i>.norm2(.b), l<i>.norm2b(.b), l<i>.mix.*,
l<i>.mlp.*, final.norm(.b).
"""

from __future__ import annotations

from typing import Mapping, Optional

from ..config.spec import (EmbeddingSpec, HeadSpec, LatentAttentionSpec, LayerNormSpec, LayerSpec, LoopSpec, ModelSpec,
                           RotarySpec, ScheduleEntry, SelectiveScanSpec, SoftmaxAttentionSpec, SwiGluSpec)
from ..errors import ConfigError
from ..registry import register_architecture

LAYER_NAMES = {"mixer_norm": "norm1", "mixer_out_norm": "norm1b", "feed_forward_norm": "norm2",
               "feed_forward_out_norm": "norm2b", "mixer": "mix.", "feed_forward": "mlp."}
ATTENTION_NAMES = (("q_proj.weight", "q"), ("k_proj.weight", "k"), ("v_proj.weight", "v"), ("o_proj.weight", "o"),
                   ("q_norm.weight", "q.norm"), ("k_norm.weight", "k.norm"), ("head_mix", "talk"))
FEED_FORWARD_NAMES = (("gate_proj.weight", "gate"), ("up_proj.weight", "up"), ("down_proj.weight", "down"))


def _need(table, key: str, where: str):
    if not isinstance(table, Mapping) or key not in table:
        raise ConfigError(f"Pedotar config: {where} needs `{key}`")
    return table[key]


def _size(table, key: str, where: str) -> int:
    value = int(_need(table, key, where))
    if value <= 0:
        raise ConfigError(f"Pedotar config: {where}.{key} must be above zero, got {value}")
    return value


def _selective_scan(mixer: Mapping, width: int, where: str) -> SelectiveScanSpec:
    return SelectiveScanSpec(hidden_size=width, inner=_size(mixer, "inner", where), state=_size(mixer, "state", where),
                             dt_rank=_size(mixer, "dt_rank", where), conv_taps=_size(mixer, "conv", where))


def _latent_attention(mixer: Mapping, width: int, eps: float, where: str) -> LatentAttentionSpec:
    rotary_dim = int(mixer.get("rot_dim", 0))
    position = None
    if rotary_dim:
        rot = _need(mixer, "rot", where)
        dims = int(_need(rot, "dims", where + ".rot"))
        if dims != rotary_dim or rotary_dim < 0 or rotary_dim % 2:
            raise ConfigError(f"Pedotar config: {where}: rot.dims {dims} must equal rot_dim {rotary_dim}, an even number")
        position = RotarySpec(head_dim=rotary_dim, rotary_dim=rotary_dim, theta=float(_need(rot, "base", where + ".rot")),
                              layout="half")
    return LatentAttentionSpec(
        hidden_size=width, heads=_size(mixer, "heads", where), head_dim=_size(mixer, "dim", where), rotary_dim=rotary_dim,
        value_dim=_size(mixer, "vdim", where), q_rank=0, kv_rank=_size(mixer, "kv_rank", where),
        scale=float(_need(mixer, "scale", where)), norm_eps=eps, gate=False, position=position)


def _attention(mixer: Mapping, width: int, eps: float, where: str) -> SoftmaxAttentionSpec:
    heads, kv_heads, dim = (_size(mixer, key, where) for key in ("heads", "kv_heads", "dim"))
    if heads % kv_heads:
        raise ConfigError(f"Pedotar config: {where}: heads must be a multiple of kv_heads")
    return SoftmaxAttentionSpec(
        hidden_size=width, heads=heads, kv_heads=kv_heads, head_dim=dim, value_head_dim=_size(mixer, "vdim", where),
        scale=float(_need(mixer, "scale", where)), qk_norm=True, qk_norm_eps=eps, names=ATTENTION_NAMES, position=None,
        chunk=_size(_need(mixer, "mask", where), "size", where + ".mask"), head_mix=True)


def _feed_forward(mlp: Mapping, width: int, where: str) -> SwiGluSpec:
    if mlp.get("kind") != "dense":
        raise ConfigError(f"Pedotar config: {where} has kind {mlp.get('kind')!r}; known: dense")
    return SwiGluSpec(hidden_size=width, intermediate_size=_size(mlp, "ff", where), names=FEED_FORWARD_NAMES)


def build(config: Mapping, catalog: Optional[Mapping[str, tuple]] = None) -> ModelSpec:
    width, vocab = _size(config, "width", "the model"), _size(config, "vocab", "the model")
    eps = float(_need(_need(config, "norm", "the model"), "eps", "norm"))
    norm = LayerNormSpec(size=width, eps=eps, tensor="", bias_tensor=".b")
    layers = []
    for index, layer in enumerate(_need(config, "layers", "the model")):
        where = f"layers[{index}]"
        kind, mixer = _need(layer, "type", where), _need(layer, "mixer", where)
        inside = where + ".mixer"
        if kind == "mamba1":
            mixer_spec = _selective_scan(mixer, width, inside)
        elif kind == "latent_attention":
            mixer_spec = _latent_attention(mixer, width, eps, inside)
        elif kind == "attention":
            mixer_spec = _attention(mixer, width, eps, inside)
        else:
            raise ConfigError(f"Pedotar config: {where} has type {kind!r}; known: mamba1, latent_attention, attention")
        mlp = layer.get("mlp")
        feed_forward = _feed_forward(mlp, width, where + ".mlp") if mlp is not None else None
        second = norm if feed_forward is not None else None
        layers.append(LayerSpec(prefix=f"l{index}.", mixer=mixer_spec, feed_forward=feed_forward, mixer_norm=norm,
                                feed_forward_norm=second, mixer_out_norm=norm, feed_forward_out_norm=second,
                                names=LAYER_NAMES, arrangement="sandwich"))
    count = len(layers)
    loop_config, loop = config.get("loop"), None
    if loop_config:
        start, stop, times = (int(_need(loop_config, key, "loop")) for key in ("start", "stop", "times"))
        if not 0 <= start <= stop <= count or times < 1:
            raise ConfigError(f"Pedotar config: loop {start}..{stop} x {times} does not fit {count} layers")
        schedule = [ScheduleEntry(layer=i) for i in range(start)]
        for number in range(times):
            schedule += [ScheduleEntry(layer=i, opens_pass=number if i == start else None) for i in range(start, stop)]
        schedule += [ScheduleEntry(layer=i) for i in range(stop, count)]
        loop = LoopSpec(passes=times, step_tensor=None, add_embedding=True)
    else:
        schedule = [ScheduleEntry(layer=i) for i in range(count)]
    return ModelSpec(
        architecture="Pedotar", hidden_size=width, vocab_size=vocab,
        max_positions=int(config.get("max_positions", 1 << 30)), embedding=EmbeddingSpec("embed", vocab, width, 1.0),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm, final_norm_name="final.norm",
        head=HeadSpec("embed", vocab, width, tied=True), loop=loop)


register_architecture("Pedotar", build)
