"""Typed configuration of Tekezen, a decoder that alternates latent attention behind a short window with grouped attention
behind a longer window that keeps the sequence's first tokens; norms on the sub-blocks' outputs only; dense and routed
clamped gated feed-forwards; an embedding that adds a row for each pair of neighbouring tokens; the token table doubles
as the output head.

config.json of this design, key by key:

    architecture        "Tekezen"
    vocab, width        sizes of the token table and of the residual stream
    embedding.bigram    optional: buckets, mul_prev, mul_cur.  Row (token before * mul_prev + token * mul_cur) mod buckets of
                        the tensor `bigram` joins the token's row; a sequence's first token takes the row behind the buckets
    norm.eps            eps of every RMS norm (the outputs' and the final norm, whose weights are offsets from one; the latent's
                        norm and the norms of the whole query and key projections, whose weights are factors)
    layers[i]           type, mixer, mlp:
      type "latent_attention"   mixer: heads, dim (unrotated), rot_dim, vdim, kv_rank, scale, rot (base, dims = rot_dim,
                                optional scaling: factor, original, fast, slow), mask.size (optional window); one output
                                gate per head
      type "attention"          mixer: heads, kv_heads, dim, vdim, scale, softcap (optional), rot (base, dims, optional
                                scaling: factor), mask (optional): size, keep_first; v_mix: the layer shares values, the
                                first such layer hands its own on and the others blend them into theirs
      mlp                       null, or kind "dense" with ff and limit, or kind "moe" with expert.ff / limit,
                                router.experts / top and, optional, shared.ff / limit
    max_positions       optional: longest sequence the block tables are made for

Tensor names: embed, bigram, l<i>.norm1 / norm2, l<i>.mix.*, l<i>.mlp.*, final.norm.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional

from .errors import ConfigError
from .registry import register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

DEFAULT_MAX_POSITIONS = 1 << 17
MIXER_TYPES = ("latent_attention", "attention")
HEAD_STEP, HEAD_MAX = 16, 512        # the attention kernels take rows that are multiples of 16 up to 512
LATENT_NAMES = {"q": "q", "kv_down": "dkv", "kv_norm": "dkv.norm", "k_up": "uk", "v_up": "uv", "gate": "g", "out": "o"}
EXPERT_NAMES = {"router": "router", "gate": "e{}.gate", "up": "e{}.up", "down": "e{}.down", "shared_gate": "shared.gate",
                "shared_up": "shared.up", "shared_down": "shared.down"}


def _need(mapping: Mapping[str, Any], key: str, where: str):
    if not isinstance(mapping, Mapping) or key not in mapping:
        raise ConfigError(f"config.json lacks {where}{key}")
    return mapping[key]


def _rotation(rot: Mapping[str, Any], at: str, kind: str) -> PartSpec:
    """The rotary encoding of a mixer: coordinates paired across the halves of the turned part, frequencies changed by the
    mixer's own rule where `scaling` is given ("linear" for the grouped attention, "yarn" for the latent)."""
    dims, base = int(_need(rot, "dims", at)), float(_need(rot, "base", at))
    if dims <= 0 or dims % 2 or not base > 0:
        raise ConfigError(f"{at}: dims must be positive and even, base positive")
    params = {"theta": base, "dim": dims}
    scaling = rot.get("scaling")
    if scaling:
        keys = ("factor",) if kind == "linear" else ("factor", "original", "fast", "slow")
        params["scaling"] = {"kind": kind, **{key: float(_need(scaling, key, at + "scaling.")) for key in keys}}
        if not all(value > 0 for key, value in params["scaling"].items() if key != "kind"):
            raise ConfigError(f"{at}scaling: the numbers must be positive")
    return PartSpec("rotary_half", params)


def _window(m: Mapping[str, Any], at: str) -> tuple:
    """(window or None, kept first tokens) of a mixer's mask."""
    mask = m.get("mask") or {}
    window = int(mask["size"]) if mask.get("size") is not None else None
    keep = int(mask.get("keep_first") or 0)
    if window is not None and window < 1 or keep < 0:
        raise ConfigError(f"{at}mask: size must be at least 1, keep_first not negative")
    return window, keep


@dataclass(frozen=True)
class TekezenConfig:
    raw: Mapping[str, Any]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "TekezenConfig":
        config = cls(dict(raw))
        config.to_spec()          # every refusal is raised here, before any weight is read
        return config

    def to_dict(self) -> dict:
        return dict(self.raw)

    # ---------------------------------------------------------------- mixers
    @staticmethod
    def _latent(m, at: str, width: int, eps: float) -> PartSpec:
        heads, dim, rot_dim = int(_need(m, "heads", at)), int(_need(m, "dim", at)), int(_need(m, "rot_dim", at))
        vdim, kv_rank = int(_need(m, "vdim", at)), int(_need(m, "kv_rank", at))
        if min(heads, dim, rot_dim, vdim, kv_rank) <= 0:
            raise ConfigError(f"{at}: sizes must be positive")
        position = _rotation(_need(m, "rot", at), at + "rot.", "yarn")
        if position["dim"] != rot_dim:
            raise ConfigError(f"{at}rot.dims must equal rot_dim")
        if -(-(kv_rank + rot_dim) // HEAD_STEP) * HEAD_STEP > HEAD_MAX:
            raise ConfigError(f"{at}kv_rank + rot_dim = {kv_rank + rot_dim} is not supported: the attention kernels take cache rows up to {HEAD_MAX} wide")
        window, keep = _window(m, at)
        if keep:
            raise ConfigError(f"{at}mask.keep_first: latent attention keeps no first tokens")
        return PartSpec("latent_attention", {
            "hidden_size": width, "num_heads": heads, "plain_dim": dim, "rot_dim": rot_dim, "value_dim": vdim, "kv_rank": kv_rank,
            "q_rank": 0, "gate": "head", "position": position, "scale": float(_need(m, "scale", at)), "eps": eps, "window": window,
            "sink": False, "shared_kv": False, "names": LATENT_NAMES})

    @staticmethod
    def _attention(m, at: str, width: int, eps: float, values: Optional[str]) -> PartSpec:
        heads, kv_heads = int(_need(m, "heads", at)), int(_need(m, "kv_heads", at))
        dim, vdim = int(_need(m, "dim", at)), int(_need(m, "vdim", at))
        if min(heads, kv_heads, dim, vdim) <= 0 or heads % kv_heads:
            raise ConfigError(f"{at}: sizes must be positive and heads a multiple of kv_heads")
        if max(dim, vdim) > HEAD_MAX:
            raise ConfigError(f"{at}: heads of {max(dim, vdim)} are not supported: the attention kernels take up to {HEAD_MAX}")
        position = _rotation(_need(m, "rot", at), at + "rot.", "linear")
        if position["dim"] > dim:
            raise ConfigError(f"{at}rot.dims must not exceed dim")
        softcap = m.get("softcap")
        if softcap is not None and not float(softcap) > 0:
            raise ConfigError(f"{at}softcap must be positive")
        window, keep = _window(m, at)
        return PartSpec("windowed_attention", {
            "hidden_size": width, "num_heads": heads, "num_kv_heads": kv_heads, "key_dim": dim, "value_dim": vdim, "position": position,
            "scale": float(_need(m, "scale", at)), "softcap": softcap, "window": window, "keep_first": keep, "qk_norm": "whole", "eps": eps,
            "values": values})

    def _mixers(self, layers, width: int, eps: float) -> list:
        out, first = [], None        # first: the layer whose values the later sharing layers take
        for i, layer in enumerate(layers):
            where = f"layers[{i}]."
            kind = _need(layer, "type", where)
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{where}type {kind!r} is not a mixer of this design; known: {', '.join(MIXER_TYPES)}")
            m, at = _need(layer, "mixer", where), where + "mixer."
            if kind == "latent_attention":
                out.append(self._latent(m, at, width, eps))
                continue
            values = None
            if m.get("v_mix"):
                values = "give" if first is None else "take"
                sizes = tuple(int(_need(m, key, at)) for key in ("kv_heads", "vdim"))
                if first is None:
                    first = (i, sizes[0] * sizes[1])
                elif sizes[0] * sizes[1] != first[1]:
                    raise ConfigError(f"{at}v_mix: the values of layer {first[0]} have another size")
            out.append(self._attention(m, at, width, eps, values))
        return out

    # ---------------------------------------------------------------- feed-forwards
    @staticmethod
    def _feed_forward(layer: Mapping[str, Any], where: str, width: int) -> Optional[PartSpec]:
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        at = where + "mlp."
        kind = _need(mlp, "kind", at)

        def sized(part, at) -> tuple:
            ff, limit = int(_need(part, "ff", at)), float(_need(part, "limit", at))
            if ff <= 0 or not limit > 0:
                raise ConfigError(f"{at}: ff and limit must be positive")
            return ff, limit

        if kind == "dense":
            ff, limit = sized(mlp, at)
            return PartSpec("swiglu", {"hidden_size": width, "intermediate_size": ff, "activation": "gated_clamp", "limit": limit,
                                       "names": {"gate": "gate", "up": "up", "down": "down"}})
        if kind != "moe":
            raise ConfigError(f"{at}kind {kind!r} is not a feed-forward of this design; known: dense, moe")
        router = _need(mlp, "router", at)
        experts, top = int(_need(router, "experts", at + "router.")), int(_need(router, "top", at + "router."))
        ff, limit = sized(_need(mlp, "expert", at), at + "expert.")
        if min(experts, top) <= 0 or top > experts:
            raise ConfigError(f"{at}router: experts and top must be positive and top at most experts")
        shared = None
        if mlp.get("shared"):
            size, shared_limit = sized(mlp["shared"], at + "shared.")
            shared = {"size": size, "limit": shared_limit, "scaled": False}
        # the softmax over the chosen logits alone is the softmax over all of them, renormalised over the chosen
        return PartSpec("routed_experts", {
            "hidden_size": width, "expert_size": ff, "experts": experts, "top": top, "scores": "softmax", "renormalize": True,
            "route_scale": 1.0, "activation": "gated_clamp", "limit": limit, "shared": shared, "names": EXPERT_NAMES})

    # ---------------------------------------------------------------- the model
    def to_spec(self) -> ModelSpec:
        raw = self.raw
        if raw.get("architecture") != "Tekezen":
            raise ConfigError(f"architecture {raw.get('architecture')!r} is not Tekezen")
        vocab, width = int(_need(raw, "vocab", "")), int(_need(raw, "width", ""))
        eps = float(_need(_need(raw, "norm", ""), "eps", "norm."))
        if vocab <= 0 or width <= 0 or not eps > 0:
            raise ConfigError("vocab, width and norm.eps must be positive")
        pairs, bigram = None, (raw.get("embedding") or {}).get("bigram")
        if bigram:
            at = "embedding.bigram."
            pairs = {**{key: int(_need(bigram, key, at)) for key in ("buckets", "mul_prev", "mul_cur")}, "weight_name": "bigram"}
            if not 0 < pairs["buckets"] < 1 << 31:
                raise ConfigError(f"{at}buckets must be positive and fit 31 bits")
        layer_list = _need(raw, "layers", "")
        if not layer_list:
            raise ConfigError("a model needs at least one layer")
        norm = PartSpec("rms_norm_offset", {"size": width, "eps": eps, "weight_name": ""})
        names = {"mixer": "mix.", "mixer_out_norm": "norm1", "feed_forward": "mlp.", "feed_forward_out_norm": "norm2"}
        layers = []
        for i, (layer, mixer) in enumerate(zip(layer_list, self._mixers(layer_list, width, eps))):
            ffn = self._feed_forward(layer, f"layers[{i}].", width)
            extras = {"mixer_out_norm": norm} | ({"feed_forward_out_norm": norm} if ffn is not None else {})
            layers.append(LayerSpec(prefix=f"l{i}.", mixer=mixer, mixer_norm=None, feed_forward=ffn, feed_forward_norm=None,
                                    arrangement="pre_post_norm_scaled", names=names, extras=extras))
        spec = ModelSpec(
            hidden_size=width, vocab_size=vocab, max_positions=int(raw.get("max_positions", DEFAULT_MAX_POSITIONS)),
            embedding=PartSpec("token_embedding", {"vocab_size": vocab, "hidden_size": width, "weight_name": "embed", "pairs": pairs}),
            embedding_prefix="", layers=tuple(layers), run=tuple(RunEntry(layer=i) for i in range(len(layers))),
            final_norm=norm, final_norm_prefix="final.norm",
            head=PartSpec("linear_head", {"vocab_size": vocab, "hidden_size": width, "tied_to": "embed", "weight_name": ""}),
            head_prefix="head", stream=PartSpec("post_norm"))
        spec.validate()
        return spec


register_architecture("Tekezen", TekezenConfig)
