"""Typed configuration of the Dabilorn architecture, read from ``config.json``.

A Dabilorn model is a list of layers (``layers``) with layer norms (a weight, no bias) on the sublayers' outputs, each followed by
a stored vector: x <- x + ls1 * norm1(mixer(x + canon1(x))), then x <- x + ls2 * norm2(ff(x)), canon1 a causal convolution over
time on every channel with ``canon.taps`` taps.  A layer's ``type`` names its mixer:

* ``latent_attention``: queries through a normed latent of ``q_rank`` numbers; a cache of one normed latent of ``kv_rank`` numbers
  and one rotated key part of ``rot_dim`` numbers per token; ``heads`` heads with ``dim`` unrotated and ``rot_dim`` rotated query
  and key numbers and values of ``vdim``; ``scale``; interleaved rotary pairs (``rot.base``, ``rot.dims``), stretched when
  ``rot.scaling`` is given (``factor``, ``original``, ``fast``, ``slow``); every earlier token is visible; the heads' outputs are
  gated number by number;
* ``attention``: ``heads`` query and ``kv_heads`` key/value heads of ``dim`` and ``vdim``, q and k RMS-normed over their whole
  rows, half-split rotation of the first ``rot.dims`` numbers (``rot.base``), ``scale``, weights sigmoid(score + a stored number
  per head) that are not normalised, chunks of ``mask.size`` positions, the heads' outputs gated number by number;
* ``wkv``: RWKV-style time mixing with ``heads`` memories of ``dim`` x ``dim``; the decay's inner size is its tensor's and is
  read from there.

``mlp`` is null or ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}, "shared": {"ff"} or null}``: the ``top`` experts
with the largest sigmoid scores, each run on its score times the token's row, experts down(relu(up x)^2); a shared expert of the
same form runs for every token, times a sigmoid of one number per token.  Around the layers: ``vocab``, ``width``, ``norm.eps``; the
embedding rows go through a layer norm (``embed.norm``), the output projection is the embedding table behind ``final.norm``.
Optional keys this engine adds: ``max_position`` (default 1,048,576: the design has no position limit), ``bos_token_id``,
``eos_token_id``, and in a wkv layer's ``mixer`` ``decay_rank`` for a model without tensors to read it from.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Optional, Tuple

from .kolodra import _get, _pos_int
from .lasupel import _under
from .model_spec import ModelSpec, ScheduleEntry
from .qwen3 import ConfigError

MIXER_TYPES = ("latent_attention", "attention", "wkv")


@dataclass(frozen=True)
class DabilornMlp:
    ff: int                         # an expert's size
    experts: int
    top: int
    shared_ff: int = 0              # 0: no shared expert


@dataclass(frozen=True)
class DabilornLayer:
    type: str
    mixer: Tuple[Tuple[str, object], ...]     # the mixer's sizes and constants
    mlp: Optional[DabilornMlp]

    def m(self, key: str):
        return dict(self.mixer)[key]


def _rotation(m: dict, w: str, most: int, stretched: bool) -> dict:
    """The rotation's keys; without ``rot`` nothing turns."""
    rot = m.get("rot")
    if rot is None:
        return {"rot_dims": 0, "rot_base": 1.0, "stretch": None}
    dims, base = _under(w, _get, m, "rot.dims", int), float(_under(w, _get, m, "rot.base"))
    if dims < 0 or dims % 2 or dims > most:
        raise ConfigError(f"config.json: {w}: 'rot.dims' = {dims} must be even and at most {most}")
    if dims and not base > 0:
        raise ConfigError(f"config.json: {w}: 'rot.base' must be positive")
    stretch = None
    if rot.get("scaling") is not None:
        if not stretched:
            raise ConfigError(f"config.json: {w}: 'rot.scaling' belongs to latent attention")
        stretch = tuple(float(_under(w, _get, m, "rot.scaling." + k)) for k in ("factor", "original", "fast", "slow"))
        if not all(v > 0 for v in stretch) or not base > 1:
            raise ConfigError(f"config.json: {w}: 'rot.scaling' needs positive factor, original, fast and slow, and a 'rot.base' above 1")
    return {"rot_dims": dims, "rot_base": base, "stretch": stretch}


def _mixer(kind: str, m: dict, w: str) -> Tuple[Tuple[str, object], ...]:
    w = w + ".mixer"

    def fail(msg):
        raise ConfigError(f"config.json: {w}: {msg}")

    if kind == "wkv":
        out = {k: _under(w, _pos_int, m, k) for k in ("heads", "dim")}
        if out["dim"] > 512:
            fail(f"'dim' = {out['dim']} (at most 512)")
        out["decay_rank"] = _under(w, _pos_int, m, "decay_rank")
    elif kind == "latent_attention":
        out = {k: _under(w, _pos_int, m, k) for k in ("heads", "vdim", "kv_rank", "q_rank")}
        for k in ("dim", "rot_dim"):
            v = _under(w, _get, m, k, int)
            if v < 0:
                fail(f"'{k}' must not be negative")
            out[k] = v
        if out["dim"] + out["rot_dim"] <= 0:
            fail("'dim' + 'rot_dim' must be positive")
        if out["kv_rank"] > 512:
            fail(f"'kv_rank' = {out['kv_rank']} (at most 512)")
        out["scale"] = float(_under(w, _get, m, "scale"))
        out.update(_rotation(m, w, out["rot_dim"], stretched=True))
    else:
        out = {k: _under(w, _pos_int, m, k) for k in ("heads", "kv_heads", "dim", "vdim")}
        if out["heads"] % out["kv_heads"]:
            fail(f"'heads' ({out['heads']}) must be a multiple of 'kv_heads' ({out['kv_heads']})")
        if out["dim"] > 256 or out["vdim"] > 256:
            fail(f"'dim' = {out['dim']} and 'vdim' = {out['vdim']} may be at most 256")
        out["scale"] = float(_under(w, _get, m, "scale"))
        out["chunk"] = _under(w, _pos_int, m, "mask.size") if m.get("mask") is not None else None
        out.update(_rotation(m, w, out["dim"], stretched=False))
    return tuple(sorted(out.items(), key=lambda kv: kv[0]))


def _mlp(mlp, w: str) -> Optional[DabilornMlp]:
    if mlp is None:
        return None
    w = w + ".mlp"
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {w}.kind = {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} (moe or null)")
    experts, top = _under(w, _pos_int, mlp, "router.experts"), _under(w, _pos_int, mlp, "router.top")
    if top > experts:
        raise ConfigError(f"config.json: {w}.router: {top} experts cannot be chosen among {experts}")
    return DabilornMlp(_under(w, _pos_int, mlp, "expert.ff"), experts, top,
                       _under(w, _pos_int, mlp, "shared.ff") if mlp.get("shared") is not None else 0)


@dataclass(frozen=True)
class DabilornConfig:
    vocab: int
    width: int
    norm_eps: float
    taps: int
    layers: Tuple[DabilornLayer, ...]
    max_position: int = 1 << 20
    bos_token_id: Optional[int] = None
    stop_token_ids: Tuple[int, ...] = ()

    architecture = "Dabilorn"

    @classmethod
    def from_dict(cls, d: dict, tensor_shapes: Optional[dict] = None) -> "DabilornConfig":
        entries = d.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(entries):
            w = f"layers[{i}]"
            if not isinstance(e, dict):
                raise ConfigError(f"config.json: {w} must be an object")
            if e.get("type") not in MIXER_TYPES:
                raise ConfigError(f"config.json: {w}.type = {e.get('type')!r} (this design has {', '.join(MIXER_TYPES)})")
            if not isinstance(e.get("mixer"), dict):
                raise ConfigError(f"config.json: {w}.mixer must be an object")
            mixer = e["mixer"]
            if e["type"] == "wkv" and "decay_rank" not in mixer:
                shape = (tensor_shapes or {}).get(f"l{i}.mix.w1")
                if shape is None or len(shape) != 2:
                    raise ConfigError(f"config.json: {w}: the inner size of the decay is not known (mixer.decay_rank, or the rows of the "
                                      f"checkpoint's matrix 'l{i}.mix.w1')")
                mixer = dict(mixer, decay_rank=int(shape[0]))
            layers.append(DabilornLayer(e["type"], _mixer(e["type"], mixer, w), _mlp(e.get("mlp"), w)))
        eps = float(_get(d, "norm.eps"))
        if not eps > 0:
            raise ConfigError("config.json: 'norm.eps' must be positive")
        eos = d.get("eos_token_id")
        stops = (eos,) if isinstance(eos, int) and not isinstance(eos, bool) else tuple(int(x) for x in eos) if isinstance(eos, list) else ()
        return cls(vocab=_pos_int(d, "vocab"), width=_pos_int(d, "width"), norm_eps=eps, taps=_pos_int(d, "canon.taps"), layers=tuple(layers),
                   max_position=_pos_int(d, "max_position") if "max_position" in d else 1 << 20,
                   bos_token_id=d.get("bos_token_id") if isinstance(d.get("bos_token_id"), int) else None, stop_token_ids=stops)

    @classmethod
    def from_dir(cls, model_dir: str) -> "DabilornConfig":
        from ..weights.loader import tensor_shapes

        with open(os.path.join(model_dir, "config.json")) as f:
            d = json.load(f)
        return cls.from_dict(d, tensor_shapes(model_dir))

    # ------------------------------------------------------------------- spec
    def _mixer_spec(self, l: DabilornLayer, p: str):
        from ..parts.attention import AttentionSpec
        from ..parts.latent_attention import LatentAttentionSpec
        from ..parts.rotary import RotarySpec, RotaryStretch
        from ..parts.wkv import WkvSpec

        if l.type == "wkv":
            return WkvSpec(prefix=p, hidden_size=self.width, num_heads=l.m("heads"), head_dim=l.m("dim"), decay_rank=l.m("decay_rank"),
                           norm_eps=self.norm_eps)
        if l.type == "latent_attention":
            st = l.m("stretch")
            position = RotarySpec(rotary_dim=l.m("rot_dims"), theta=l.m("rot_base"), pairing="interleaved",
                                  stretch=RotaryStretch(*st) if st is not None else None) if l.m("rot_dims") else None
            return LatentAttentionSpec(prefix=p, hidden_size=self.width, num_heads=l.m("heads"), nope_dim=l.m("dim"), rope_dim=l.m("rot_dim"),
                                       value_dim=l.m("vdim"), kv_rank=l.m("kv_rank"), scale=l.m("scale"), norm_eps=self.norm_eps,
                                       position=position, window=None, q_rank=l.m("q_rank"), out_gate=True)
        return AttentionSpec(
            prefix=p, hidden_size=self.width, num_heads=l.m("heads"), num_kv_heads=l.m("kv_heads"), head_dim=l.m("dim"), scale=l.m("scale"),
            qk_norm_eps=self.norm_eps, qk_norm="row", value_dim=l.m("vdim"), chunk=l.m("chunk"), weights="sigmoid", out_gate=True,
            position=RotarySpec(rotary_dim=l.m("rot_dims"), theta=l.m("rot_base"), pairing="half") if l.m("rot_dims") else None,
            names=(("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_norm", "q.norm"), ("k_norm", "k.norm"), ("gate", "g"), ("score_bias", "pb")))

    def _mlp_spec(self, mlp: DabilornMlp, p: str):
        from ..parts.mlp import UngatedMlpSpec
        from ..parts.moe import RoutedExpertsSpec

        shared = UngatedMlpSpec(prefix=p + "shared.", hidden_size=self.width, intermediate_size=mlp.shared_ff, activation="square_relu",
                                names=("up", "down")) if mlp.shared_ff else None
        return RoutedExpertsSpec(prefix=p, hidden_size=self.width, num_experts=mlp.experts, top=mlp.top, expert_ff=mlp.ff, correction=False,
                                 shared=shared, shared_gate=shared is not None, activation="square_relu", gated=False, weight_on="input")

    def to_model_spec(self) -> ModelSpec:
        from ..parts.block import OutputNormBlockSpec
        from ..parts.norm import LayerNormSpec

        blocks, schedule, ignored = [], [], []
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            if l.mlp is None:               # a layer without a feed-forward has no use for its norm and scale, should they be stored
                ignored += [p + "norm2", p + "ls2"]
            blocks.append(OutputNormBlockSpec(
                mixer_norm=LayerNormSpec(p + "norm1", self.width, self.norm_eps, scale_name=p + "ls1"), mixer=self._mixer_spec(l, p + "mix."),
                ffn_norm=LayerNormSpec(p + "norm2", self.width, self.norm_eps, scale_name=p + "ls2") if l.mlp is not None else None,
                ffn=self._mlp_spec(l.mlp, p + "mlp.") if l.mlp is not None else None,
                conv_taps=self.taps, conv_name=p + "canon1", conv_size=self.width))
            schedule.append(ScheduleEntry(i))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, blocks=tuple(blocks), schedule=tuple(schedule),
            final_norm=LayerNormSpec("final.norm", self.width, self.norm_eps), embed_name="embed", head_name=None,
            embed_norm=LayerNormSpec("embed.norm", self.width, self.norm_eps), max_position=self.max_position,
            stop_token_ids=self.stop_token_ids, bos_token_id=self.bos_token_id, ignored_tensors=tuple(ignored))
