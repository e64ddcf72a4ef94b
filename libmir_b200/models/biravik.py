"""Biravik: a decoder whose norms stand behind the sums, x = norm1(alpha x + mixer(x)), then x = norm2(alpha x + ff(x)),
with softmax attention beside lightning attention in one layer, windowed attention whose values are its keys, and wkv
mixers: config.json -> ModelSpec.

config.json:
    architecture  "Biravik"
    vocab, width, norm.eps, embedding.scale, postln_alpha (alpha)
    layers[i]     {type, mixer, mlp}; tensors of layer i start with "l<i>."
        type "parallel"   mixer {left, left_scale, right, right_scale}: left_scale * left(x) + right_scale * right(x)
            left   {heads, kv_heads, dim, vdim, scale, q_temp {coef, every}}: grouped softmax attention without rotation;
                   an RMS norm of every query and key head (weights q.norm, k.norm), queries times 1 + coef ln(floor((p + 1)
                   / every) + 1) at position p, a bias that falls linearly with the distance (slope 2^(-8 (h + 1) / heads) of
                   head h), one sink per query head, a sigmoid gate on the concatenated heads; causal
            right  {heads, dim, vdim, decay [one per head]}: linear attention with a fixed decay per head on silu of its
                   projections, one RMS norm over all heads together (weight `norm`), a sigmoid gate
        type "attention"  mixer {heads, kv_heads, dim, vdim, scale, rot {dims, base, scaling {factor, original, fast, slow}},
                          mask {size, keep_first}}: the values are the keys as projected (no value tensor, vdim equals dim);
                          q/k norm, interleaved rotation of the first rot.dims dims with YaRN scaling, a sliding window with
                          kept first tokens, sinks, gate
        type "wkv"        mixer {heads, dim}: time mixing with a matrix state per head; the rank of the decay's low-rank
                          pair is the shape of `w1`
        mlp       {kind "dense", ff} (up, squared relu, down), {kind "moe", expert {ff}, router {experts, top}} (gated
                  experts, weights by softmax over the chosen logits) or null
Norm weights of the layers and of the model are stored around zero (the norm multiplies by 1 + w); the norms inside mixers
have plain weights.
Tensor names: embed, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.*, final.norm, head.
"""

from __future__ import annotations

from typing import Mapping, Optional

from ..config.spec import (EmbeddingSpec, GeluMlpSpec, HeadSpec, LayerSpec, ModelSpec, QueryTemperature, RetentionSpec,
                           RmsNormSpec, RotarySpec, RoutedExpertsSpec, ScheduleEntry, SideBySideSpec,
                           SoftmaxAttentionSpec, WkvSpec, YarnScaling)
from ..errors import ConfigError
from ..registry import register_architecture

LAYER_NAMES = {"mixer_norm": "norm1", "feed_forward_norm": "norm2", "mixer": "mix.", "feed_forward": "mlp."}
ATTENTION_NAMES = (("q_proj.weight", "q"), ("k_proj.weight", "k"), ("v_proj.weight", "v"), ("o_proj.weight", "o"),
                   ("q_norm.weight", "q.norm"), ("k_norm.weight", "k.norm"), ("g_proj.weight", "g"), ("sinks", "sink"))
DEFAULT_DECAY_RANK = 16      # of the decay's low-rank pair, when no checkpoint is at hand to take it from


def _need(table, key: str, where: str):
    if not isinstance(table, Mapping) or key not in table:
        raise ConfigError(f"Biravik config: {where} needs `{key}`")
    return table[key]


def _size(table, key: str, where: str) -> int:
    value = int(_need(table, key, where))
    if value <= 0:
        raise ConfigError(f"Biravik config: {where}.{key} must be above zero, got {value}")
    return value


def _grouped_heads(mixer: Mapping, where: str) -> tuple:
    heads, kv_heads, dim = (_size(mixer, key, where) for key in ("heads", "kv_heads", "dim"))
    if heads % kv_heads:
        raise ConfigError(f"Biravik config: {where}: heads must be a multiple of kv_heads")
    return heads, kv_heads, dim


def _rotation(mixer: Mapping, dim: int, where: str) -> Optional[RotarySpec]:
    rot = mixer.get("rot")
    if not rot:
        return None
    dims = int(_need(rot, "dims", where + ".rot"))
    if dims == 0:
        return None
    if dims % 2 or not 0 < dims <= dim:
        raise ConfigError(f"Biravik config: {where}.rot.dims {dims} must be even and at most dim {dim}")
    scaling = rot.get("scaling")
    yarn = YarnScaling(*(float(_need(scaling, key, where + ".rot.scaling"))
                         for key in ("factor", "original", "fast", "slow"))) if scaling else None
    return RotarySpec(head_dim=dim, rotary_dim=dims, theta=float(_need(rot, "base", where + ".rot")), scaling=yarn,
                      layout="interleaved")


def _biased_attention(mixer: Mapping, width: int, eps: float, where: str) -> SoftmaxAttentionSpec:
    heads, kv_heads, dim = _grouped_heads(mixer, where)
    temperature = mixer.get("q_temp")
    if temperature:
        every = float(_need(temperature, "every", where + ".q_temp"))
        if every <= 0:
            raise ConfigError(f"Biravik config: {where}.q_temp.every must be above zero, got {every}")
        temperature = QueryTemperature(float(_need(temperature, "coef", where + ".q_temp")), every)
    return SoftmaxAttentionSpec(
        hidden_size=width, heads=heads, kv_heads=kv_heads, head_dim=dim, value_head_dim=int(mixer.get("vdim", dim)),
        scale=float(_need(mixer, "scale", where)), qk_norm=True, qk_norm_eps=eps, names=ATTENTION_NAMES, sinks=True,
        gate=True, slopes=tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)), temperature=temperature or None)


def _lightning(mixer: Mapping, width: int, eps: float, where: str) -> RetentionSpec:
    heads, dim = _size(mixer, "heads", where), _size(mixer, "dim", where)
    decays = tuple(float(d) for d in _need(mixer, "decay", where))
    if len(decays) != heads:
        raise ConfigError(f"Biravik config: {where}.decay lists {len(decays)} numbers for {heads} heads")
    return RetentionSpec(hidden_size=width, heads=heads, key_dim=dim, value_dim=int(mixer.get("vdim", dim)), decays=decays,
                         norm_eps=eps, key_scale=1.0, activated=True, norm_span="all", norm_weight=True, gate="sigmoid")


def _parallel(mixer: Mapping, width: int, eps: float, where: str) -> SideBySideSpec:
    left = _biased_attention(_need(mixer, "left", where), width, eps, where + ".left")
    right = _lightning(_need(mixer, "right", where), width, eps, where + ".right")
    return SideBySideSpec(hidden_size=width, branches=(("left", left), ("right", right)),
                          scales=tuple(float(_need(mixer, key, where)) for key in ("left_scale", "right_scale")))


def _key_value_attention(mixer: Mapping, width: int, eps: float, where: str) -> SoftmaxAttentionSpec:
    heads, kv_heads, dim = _grouped_heads(mixer, where)
    if int(mixer.get("vdim", dim)) != dim:
        raise ConfigError(f"Biravik config: {where}: the values are the keys, so vdim must equal dim")
    mask = mixer.get("mask") or {}
    window = _size(mask, "size", where + ".mask") if mask else None
    return SoftmaxAttentionSpec(
        hidden_size=width, heads=heads, kv_heads=kv_heads, head_dim=dim, scale=float(_need(mixer, "scale", where)),
        qk_norm=True, qk_norm_eps=eps, names=ATTENTION_NAMES, sinks=True, gate=True, values_from_keys=True, window=window,
        keep_first=int(mask.get("keep_first", 0)), position=_rotation(mixer, dim, where))


def _wkv(mixer: Mapping, width: int, eps: float, where: str, catalog, prefix: str) -> WkvSpec:
    name = prefix + "w1"
    rank = int(catalog[name][0]) if catalog is not None and name in catalog else int(mixer.get("decay_rank", DEFAULT_DECAY_RANK))
    return WkvSpec(hidden_size=width, heads=_size(mixer, "heads", where), head_dim=_size(mixer, "dim", where),
                   decay_rank=rank, norm_eps=eps)


def _feed_forward(mlp: Mapping, width: int, where: str):
    kind = mlp.get("kind")
    if kind == "dense":
        return GeluMlpSpec(hidden_size=width, intermediate_size=_size(mlp, "ff", where), activation="relu2")
    if kind == "moe":
        router = _need(mlp, "router", where)
        experts, top = (_size(router, key, where + ".router") for key in ("experts", "top"))
        if top > experts:
            raise ConfigError(f"Biravik config: {where}.router chooses {top} of {experts} experts")
        # (the softmax over all logits, divided by its sum over the chosen, is the softmax over the chosen)
        return RoutedExpertsSpec(hidden_size=width, expert_size=_size(_need(mlp, "expert", where), "ff", where + ".expert"),
                                 experts=experts, top=top, correction=False, score="softmax", group_score="max")
    raise ConfigError(f"Biravik config: {where} has kind {kind!r}; known: dense, moe")


def build(config: Mapping, catalog: Optional[Mapping[str, tuple]] = None) -> ModelSpec:
    width, vocab = _size(config, "width", "the model"), _size(config, "vocab", "the model")
    eps = float(_need(_need(config, "norm", "the model"), "eps", "norm"))
    alpha = float(_need(config, "postln_alpha", "the model"))
    norm = RmsNormSpec(size=width, eps=eps, offset=1.0, tensor="")
    layers = []
    for index, layer in enumerate(_need(config, "layers", "the model")):
        where = f"layers[{index}]"
        prefix = f"l{index}."
        kind, mixer = _need(layer, "type", where), _need(layer, "mixer", where)
        inside = where + ".mixer"
        if kind == "parallel":
            mixer_spec = _parallel(mixer, width, eps, inside)
        elif kind == "attention":
            mixer_spec = _key_value_attention(mixer, width, eps, inside)
        elif kind == "wkv":
            mixer_spec = _wkv(mixer, width, eps, inside, catalog, prefix + "mix.")
        else:
            raise ConfigError(f"Biravik config: {where} has type {kind!r}; known: parallel, attention, wkv")
        mlp = layer.get("mlp")
        feed_forward = _feed_forward(mlp, width, where + ".mlp") if mlp is not None else None
        layers.append(LayerSpec(prefix=prefix, mixer=mixer_spec, feed_forward=feed_forward, mixer_norm=norm,
                                feed_forward_norm=norm if feed_forward is not None else None, names=LAYER_NAMES,
                                arrangement="post_norm", residual_alpha=alpha))
    return ModelSpec(
        architecture="Biravik", hidden_size=width, vocab_size=vocab,
        max_positions=int(config.get("max_positions", 1 << 30)),
        embedding=EmbeddingSpec("embed", vocab, width, float((config.get("embedding") or {}).get("scale", 1.0))),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(layer=i) for i in range(len(layers))),
        final_norm=norm, final_norm_name="final.norm", head=HeadSpec("head", vocab, width, tied=False))


register_architecture("Biravik", build)
