"""Dogotar as a list of parts.

Embedding: the token row.  Layers in the order config.json lists them; in each the mixer and the feed-forward read the same
stream through layer norms of their own and their results join it together (the ``parallel_rows`` arrangement: one product for
the last matrices of all of them).  Mixers: ``attention`` is ``head_norm_attention`` with a rotation of halves (linearly scaled
frequencies), a window, an output gate and, where the configuration says so, values mixed with the first such layer's;
``parallel`` is ``side_by_side_sum`` over a ``head_norm_attention`` without positions whose mask is a chunk and a
``matrix_memory``, each with its factor.  Feed-forward: dense with the tanh form of GELU.  Final layer norm; the head is the
embedding table.

The design has no position limit of its own: ``max_positions`` is only a bound for the engine.
"""

from __future__ import annotations

import re

from ..config.dogotar import ARCHITECTURE, CappedAttentionConfig, DogotarConfig, PairConfig
from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerSpec, ModelSpec, part, sequential_schedule

MAX_POSITIONS = 1 << 20


def _attention_spec(cfg: DogotarConfig, m: CappedAttentionConfig, **more):
    return part("head_norm_attention", hidden_size=cfg.width, num_heads=m.heads, num_kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim,
                scale=m.scale, eps=cfg.norm_eps, softcap=m.softcap, bias=True, **more)


def _mixer_spec(cfg: DogotarConfig, index: int):
    m = cfg.layers[index].mixer
    if isinstance(m, CappedAttentionConfig):
        position = None
        if m.rot is not None:
            scaling = None if m.rot.factor is None else {"kind": "linear", "factor": m.rot.factor}
            position = part("rope", head_dim=m.dim, rotary_dim=m.rot.dims, theta=m.rot.base, scaling=scaling, layout="half")
        mix = None if not m.v_mix else ("source" if index == cfg.value_source() else "mixed")
        return _attention_spec(cfg, m, window=m.reach, position=position, value_mix=mix, output_gate=True)
    if isinstance(m, PairConfig):
        r = m.right
        left = _attention_spec(cfg, m.left, chunk=m.left.reach, out_scale=m.left_scale)
        right = part("matrix_memory", hidden_size=cfg.width, num_heads=r.heads, dim=r.dim, vdim=r.vdim, gate_cap=r.gate_cap,
                     eps=cfg.norm_eps, out_scale=m.right_scale)
        return part("side_by_side_sum", hidden_size=cfg.width, names=("left", "right"), branches=(left, right))
    raise TypeError(f"no mixer for {type(m).__name__}")


def dogotar_spec(cfg: DogotarConfig) -> ModelSpec:
    norm = part("layer", size=cfg.width, eps=cfg.norm_eps)
    layers = []
    for i, layer in enumerate(cfg.layers):
        ffn = None if layer.ff is None else part("mlp", hidden_size=cfg.width, intermediate_size=layer.ff, activation="gelu_tanh")
        layers.append(LayerSpec(mixer=_mixer_spec(cfg, i), ffn=ffn, mixer_norm=norm, ffn_norm=None if ffn is None else norm,
                                arrangement="parallel_rows"))
    return ModelSpec(
        architecture=ARCHITECTURE,
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_positions=MAX_POSITIONS,
        embedding=part("token_embedding", vocab_size=cfg.vocab, hidden_size=cfg.width),
        layers=tuple(layers),
        schedule=sequential_schedule(len(layers)),
        final_norm=norm,
        head=part("lm_head", vocab_size=cfg.vocab, hidden_size=cfg.width, tied=True),
        stop_token_ids=cfg.stop_token_ids,
    )


_LAYER = re.compile(r"^layers\.(\d+)\.(.+)$")
_ATTENTION = {"q_proj": "q", "q_bias": "q.b", "q_norm": "q.norm", "k_proj": "k", "k_bias": "k.b", "k_norm": "k.norm",
              "v_proj": "v", "v_bias": "v.b", "value_share": "vmix", "gate_proj": "g", "o_proj": "o"}
_MEMORY = {"q_proj": "q", "k_proj": "k", "v_proj": "v", "gate_proj": "g", "input_proj": "i", "input_bias": "i.b", "forget_proj": "f",
           "forget_bias": "f.b", "out_norm": "norm", "o_proj": "o"}
_IN_LAYER = {
    "mixer_norm.weight": "norm1", "mixer_norm.bias": "norm1.b",
    "ffn_norm.weight": "norm2", "ffn_norm.bias": "norm2.b",
    "ffn.up_proj": "mlp.up", "ffn.down_proj": "mlp.down",
}
_IN_LAYER.update({f"mixer.{local}": f"mix.{name}" for local, name in _ATTENTION.items()})
_IN_LAYER.update({f"mixer.left.{local}": f"mix.left.{name}" for local, name in _ATTENTION.items()})
_IN_LAYER.update({f"mixer.right.{local}": f"mix.right.{name}" for local, name in _MEMORY.items()})
_TOP = {"embedding.weight": "embed", "final_norm.weight": "final.norm", "final_norm.bias": "final.norm.b"}


def dogotar_tensor_name(path: str) -> str:
    if path in _TOP:
        return _TOP[path]
    m = _LAYER.match(path)
    if m and m.group(2) in _IN_LAYER:
        return f"l{m.group(1)}.{_IN_LAYER[m.group(2)]}"
    raise KeyError(f"{ARCHITECTURE} has no tensor for part path {path!r}")


def _without_reader(cfg: DogotarConfig, name: str) -> bool:
    """What a checkpoint may carry although its layer has no use for it: the norm in front of a feed-forward that is not there,
    the share of a layer that does not mix values."""
    m = re.match(r"^l(\d+)\.(norm2|norm2\.b|mix\.vmix)$", name)
    if not m or int(m.group(1)) >= len(cfg.layers):
        return False
    layer = cfg.layers[int(m.group(1))]
    return not getattr(layer.mixer, "v_mix", False) if m.group(2) == "mix.vmix" else layer.ff is None


DOGOTAR = Architecture(
    name=ARCHITECTURE,
    model_types=("dogotar",),
    read_config=DogotarConfig.from_dicts,
    to_spec=dogotar_spec,
    tensor_name=dogotar_tensor_name,
    ignorable=_without_reader,
)

register_architecture(DOGOTAR, replace=True)
