"""Typed configuration of Kezunex, a decoder that mixes three kinds of layers: softmax attention and a state-space mixer side
by side, a recurrent block with a real-gated linear recurrent unit, and a matrix memory with exponential gates; layer norms
before and after every sub-block, a scale per channel on its way into the stream, gelu-gated dense feed-forwards, and a group
of layers that runs several times with the embedding output added again.  The token table doubles as the output head.

config.json of this design, key by key:

    architecture        "Kezunex"
    vocab, width        sizes of the token table and of the residual stream
    embedding.scale     the looked-up row is multiplied by it
    norm.eps            eps of every norm of the model: the layer norms, the per-head norms of queries and keys, the output
                        norms of the recurrent mixers
    layers[i]           type, mixer, mlp:
      type "parallel"   mixer: left (heads, kv_heads, dim, vdim, scale, q_temp: coef and every, optional), left_scale,
                        right (heads, vdim, state, groups, conv: taps, norm_groups), right_scale
      type "rglru"      mixer: width, blocks, conv (taps)
      type "mlstm"      mixer: heads, dim, vdim, gate_cap
      mlp               null, or kind "dense" with ff
    loop                optional: layers start .. stop - 1 run `times` times in a row with the same weights (each pass with a
                        cache and state of its own); right before pass t the embedding output (t > 0) and row t of tensor
                        loop.step are added to the stream
    max_positions       optional: longest sequence the block tables are made for

Tensor names: embed, loop.step, l<i>.norm1 / norm1b / norm2 / norm2b / ls1 / ls2, l<i>.mix.*, l<i>.mlp.gate / up / down, final.norm.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .errors import ConfigError
from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

DEFAULT_MAX_POSITIONS = 1 << 17
MIXER_TYPES = ("parallel", "rglru", "mlstm")
HEAD_MAX = 256                # the attention kernels take head widths up to 256
STATE_ROWS_MAX = 512          # the matrix recurrence holds up to this many rows of a state
DECAY_FACTOR = 8.0            # the recurrent unit's log decay is at most this times softplus(lam)


def _need(mapping: Mapping[str, Any], key: str, where: str):
    if not isinstance(mapping, Mapping) or key not in mapping:
        raise ConfigError(f"config.json lacks {where}{key}")
    return mapping[key]


def _sizes(m: Mapping[str, Any], at: str, *keys: str) -> list:
    values = [int(_need(m, key, at)) for key in keys]
    if min(values) <= 0:
        raise ConfigError(f"{at}: {', '.join(keys)} must be positive")
    return values


@dataclass(frozen=True)
class KezunexConfig:
    raw: Mapping[str, Any]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "KezunexConfig":
        config = cls(dict(raw))
        config.to_spec()          # every refusal is raised here, before any weight is read
        return config

    def to_dict(self) -> dict:
        return dict(self.raw)

    # ---------------------------------------------------------------- mixers
    @staticmethod
    def _attention(m, at: str, width: int, eps: float) -> PartSpec:
        heads, kv_heads, dim, vdim = _sizes(m, at, "heads", "kv_heads", "dim", "vdim")
        if heads % kv_heads:
            raise ConfigError(f"{at}heads must be a multiple of kv_heads")
        if max(dim, vdim) > HEAD_MAX:
            raise ConfigError(f"{at}: heads wider than {HEAD_MAX} are not supported by the attention kernels")
        temp = m.get("q_temp")
        if temp:
            temp = (float(_need(temp, "coef", at + "q_temp.")), float(_need(temp, "every", at + "q_temp.")))
            if not temp[1] > 0:
                raise ConfigError(f"{at}q_temp.every must be positive")
        return PartSpec("windowed_attention", {
            "hidden_size": width, "num_heads": heads, "num_kv_heads": kv_heads, "key_dim": dim, "value_dim": vdim, "position": PartSpec("none", {}),
            "scale": float(_need(m, "scale", at)), "window": None, "sink": None, "qk_norm": "head", "q_temp": temp or None, "eps": eps, "bias": ()})

    @staticmethod
    def _state_space(m, at: str, width: int, eps: float) -> PartSpec:
        heads, vdim, state, groups, conv, parts = _sizes(m, at, "heads", "vdim", "state", "groups", "conv", "norm_groups")
        if heads % groups or (heads * vdim) % parts:
            raise ConfigError(f"{at}: groups must divide heads, norm_groups must divide heads * vdim")
        if state > STATE_ROWS_MAX:
            raise ConfigError(f"{at}state {state} is not supported: the recurrence holds up to {STATE_ROWS_MAX} rows")
        return PartSpec("state_space", {"hidden_size": width, "num_heads": heads, "value_dim": vdim, "state_dim": state, "groups": groups,
                                        "conv": conv, "norm_groups": parts, "eps": eps})

    def _mixer(self, layer: Mapping[str, Any], where: str, width: int, eps: float) -> PartSpec:
        kind = _need(layer, "type", where)
        if kind not in MIXER_TYPES:
            raise ConfigError(f"{where}type {kind!r} is not a mixer of this design; known: {', '.join(MIXER_TYPES)}")
        m, at = _need(layer, "mixer", where), where + "mixer."
        if kind == "parallel":
            return PartSpec("parallel", {
                "left": self._attention(_need(m, "left", at), at + "left.", width, eps), "left_scale": float(_need(m, "left_scale", at)),
                "right": self._state_space(_need(m, "right", at), at + "right.", width, eps), "right_scale": float(_need(m, "right_scale", at))})
        if kind == "rglru":
            inner, blocks, conv = _sizes(m, at, "width", "blocks", "conv")
            if inner % blocks:
                raise ConfigError(f"{at}blocks must divide width")
            return PartSpec("rglru", {"hidden_size": width, "width": inner, "blocks": blocks, "conv": conv, "factor": DECAY_FACTOR})
        heads, dim, vdim = _sizes(m, at, "heads", "dim", "vdim")
        cap = float(_need(m, "gate_cap", at))
        if not cap > 0:
            raise ConfigError(f"{at}gate_cap must be positive")
        if dim > STATE_ROWS_MAX:
            raise ConfigError(f"{at}dim {dim} is not supported: the recurrence holds up to {STATE_ROWS_MAX} rows")
        return PartSpec("matrix_memory", {"hidden_size": width, "num_heads": heads, "key_dim": dim, "value_dim": vdim, "gate_cap": cap, "eps": eps})

    @staticmethod
    def _feed_forward(layer: Mapping[str, Any], where: str, width: int) -> Optional[PartSpec]:
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        at = where + "mlp."
        if _need(mlp, "kind", at) != "dense":
            raise ConfigError(f"{at}kind {mlp['kind']!r} is not a feed-forward of this design (dense only)")
        (ff,) = _sizes(mlp, at, "ff")
        return PartSpec("swiglu", {"hidden_size": width, "intermediate_size": ff, "activation": "gelu_tanh",
                                   "names": {"gate": "gate", "up": "up", "down": "down"}})

    # ---------------------------------------------------------------- the model
    def run_list(self, n_layers: int):
        loop = self.raw.get("loop")
        if not loop:
            return tuple(RunEntry(layer=i) for i in range(n_layers)), 0
        start, stop, times = int(_need(loop, "start", "loop.")), int(_need(loop, "stop", "loop.")), int(_need(loop, "times", "loop."))
        if not 0 <= start < stop <= n_layers or times < 1:
            raise ConfigError("loop: need 0 <= start < stop <= number of layers and times >= 1")
        run = [RunEntry(layer=i) for i in range(start)]
        for t in range(times):
            for i in range(start, stop):
                run.append(RunEntry(layer=i, pass_step=t if i == start else None, add_embedding=i == start and t > 0))
        run += [RunEntry(layer=i) for i in range(stop, n_layers)]
        return tuple(run), times

    def to_spec(self) -> ModelSpec:
        raw = self.raw
        if raw.get("architecture") != "Kezunex":
            raise ConfigError(f"architecture {raw.get('architecture')!r} is not Kezunex")
        vocab, width = _sizes(raw, "", "vocab", "width")
        eps = float(_need(_need(raw, "norm", ""), "eps", "norm."))
        if not eps > 0:
            raise ConfigError("norm.eps must be positive")
        layer_list = _need(raw, "layers", "")
        if not layer_list:
            raise ConfigError("a model needs at least one layer")
        norm = PartSpec("layer_norm", {"size": width, "eps": eps, "weight_name": ""})
        scale = PartSpec("channel_scale", {"size": width})
        names = {"mixer": "mix.", "mixer_norm": "norm1", "mixer_out_norm": "norm1b", "mixer_scale": "ls1", "feed_forward": "mlp.",
                 "feed_forward_norm": "norm2", "feed_forward_out_norm": "norm2b", "feed_forward_scale": "ls2"}
        layers = []
        for i, layer in enumerate(layer_list):
            where = f"layers[{i}]."
            ffn = self._feed_forward(layer, where, width)
            extras = {"mixer_out_norm": norm, "mixer_scale": scale}
            if ffn is not None:
                extras |= {"feed_forward_out_norm": norm, "feed_forward_scale": scale}
            layers.append(LayerSpec(prefix=f"l{i}.", mixer=self._mixer(layer, where, width, eps), mixer_norm=norm, feed_forward=ffn,
                                    feed_forward_norm=norm if ffn is not None else None, arrangement="pre_post_norm_scaled", names=names,
                                    extras=extras))
        run, times = self.run_list(len(layers))
        spec = ModelSpec(
            hidden_size=width, vocab_size=vocab, max_positions=int(raw.get("max_positions", DEFAULT_MAX_POSITIONS)),
            embedding=PartSpec("token_embedding", {"vocab_size": vocab, "hidden_size": width, "weight_name": "",
                                                   "scale": float(_need(_need(raw, "embedding", ""), "scale", "embedding."))}),
            embedding_prefix="embed", layers=tuple(layers), run=run, final_norm=norm, final_norm_prefix="final.norm",
            head=PartSpec("linear_head", {"vocab_size": vocab, "hidden_size": width, "tied_to": "embed", "weight_name": ""}),
            head_prefix="head",
            pass_steps=PartSpec("pass_vectors", {"count": times, "hidden_size": width, "weight_name": ""}) if times else None,
            pass_steps_prefix="loop.step",
            stream=PartSpec("post_norm", {"keep_embedding": times > 1}))
        spec.validate()
        return spec


register_architecture("Kezunex", KezunexConfig)
