"""Typed configuration of the Virorax architecture, read from ``config.json``.

A Virorax model adds a learned vector per position to the embedding row and then runs a list of layers (``layers``) with RMS
norms on the sublayers' inputs and a constant factor on their outputs (``residual_mult``): x <- x + m mixer(norm1(x)), then
x <- x + m ff(norm2(x)).  With ``loop`` the layers start .. stop - 1 run ``times`` times in a row with the same weights, each pass
with a cache and states of its own; before every pass but the first, the embedding output is added to x once more.  A layer's
``type`` names its mixer:

* ``attention``: grouped-query attention (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``) with biases on q, k and v; q and k are
  RMS-normed per head with a weight shared by the heads, then the first ``rot.dims`` numbers of a head are rotated (half-split
  pairs, ``rot.base``); a sliding window ``mask.size``; a learned sink score per head in the softmax's denominator; every head's
  output times the sigmoid of one number per head;
* ``retention``: linear attention with one constant ``decay`` per head (``heads``, ``dim``, ``vdim``); q and k are rotated the same way,
  k is scaled by dim^(-1/2), each head's output is brought to unit root mean square without a weight and the heads together are
  gated number by number with silu.

``mlp`` is null or ``{"kind": "dense", "ff"}``: down(relu(up x)^2).  Around the layers: ``vocab``, ``width``, ``norm.eps``,
``max_positions`` (rows of the position table; taken from the table when the key is absent); the output projection is the embedding
table behind ``final.norm``, its logits capped by ``logit_softcap`` (c tanh(z / c)).  ``mask``, ``rot``, ``loop`` and ``logit_softcap``
may be absent.  Optional keys this engine adds: ``bos_token_id``, ``eos_token_id``.
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

MIXER_TYPES = ("attention", "retention")


@dataclass(frozen=True)
class ViroraxLayer:
    type: str
    mixer: Tuple[Tuple[str, object], ...]     # the mixer's sizes and constants
    ff: int                                   # 0: no feed-forward

    def m(self, key: str):
        return dict(self.mixer)[key]


@dataclass(frozen=True)
class ViroraxLoop:
    start: int
    stop: int
    times: int


def _number(d: dict, key: str, where: str = "") -> float:
    v = _under(where, _get, d, key) if where else _get(d, key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or v != v or v in (float("inf"), float("-inf")):
        raise ConfigError(f"config.json: {where + '.' if where else ''}{key} = {v!r} must be a number")
    return float(v)


def _mixer(kind: str, m: dict, w: str) -> Tuple[Tuple[str, object], ...]:
    w = w + ".mixer"

    def fail(msg):
        raise ConfigError(f"config.json: {w}: {msg}")

    if kind == "attention":
        out = {k: _under(w, _pos_int, m, k) for k in ("heads", "kv_heads", "dim", "vdim")}
        if out["heads"] % out["kv_heads"]:
            fail(f"'heads' ({out['heads']}) must be a multiple of 'kv_heads' ({out['kv_heads']})")
        if out["dim"] > 256 or out["vdim"] > 256:
            fail(f"'dim' = {out['dim']} and 'vdim' = {out['vdim']} may be at most 256")
        out["scale"] = _number(m, "scale", w)
        out["window"] = _under(w, _pos_int, m, "mask.size") if m.get("mask") is not None else None
    else:
        out = {k: _under(w, _pos_int, m, k) for k in ("heads", "dim", "vdim")}
        if out["dim"] > 512:
            fail(f"'dim' = {out['dim']} (at most 512)")
        decay = m.get("decay")
        if (not isinstance(decay, list) or len(decay) != out["heads"]
                or not all(isinstance(d, (int, float)) and not isinstance(d, bool) and 0.0 <= d < float("inf") for d in decay)):
            fail(f"'decay' must list one number (not negative) for each of the {out['heads']} heads")
        out["decay"] = tuple(float(d) for d in decay)
    rot = m.get("rot")
    dims = _under(w, _get, m, "rot.dims", int) if rot is not None else 0
    if dims < 0 or dims % 2 or dims > out["dim"]:
        fail(f"'rot.dims' = {dims} must be even and at most dim ({out['dim']})")
    out["rot_dims"] = dims
    out["rot_base"] = _number(m, "rot.base", w) if dims else 1.0
    if not out["rot_base"] > 0:
        fail("'rot.base' must be positive")
    return tuple(sorted(out.items(), key=lambda kv: kv[0]))


def _mlp(mlp, w: str) -> int:
    if mlp is None:
        return 0
    if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
        raise ConfigError(f"config.json: {w}.mlp.kind = {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} (dense or null)")
    return _under(w + ".mlp", _pos_int, mlp, "ff")


def _loop(d: dict, layers: int) -> Optional[ViroraxLoop]:
    if d.get("loop") is None:
        return None
    start, stop, times = (_under("loop", _get, d["loop"], k, int) for k in ("start", "stop", "times"))
    if not 0 <= start < stop <= layers or times < 1:
        raise ConfigError(f"config.json: loop: layers {start} .. {stop} ({layers} layers), {times} times: must be a run of layers, at least once")
    return ViroraxLoop(start, stop, times)


@dataclass(frozen=True)
class ViroraxConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    max_positions: int
    layers: Tuple[ViroraxLayer, ...]
    loop: Optional[ViroraxLoop] = None
    logit_softcap: Optional[float] = None
    bos_token_id: Optional[int] = None
    stop_token_ids: Tuple[int, ...] = ()

    architecture = "Virorax"

    @classmethod
    def from_dict(cls, d: dict, tensor_shapes: Optional[dict] = None) -> "ViroraxConfig":
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
            layers.append(ViroraxLayer(e["type"], _mixer(e["type"], e["mixer"], w), _mlp(e.get("mlp"), w)))
        eps = _number(d, "norm.eps")
        if not eps > 0:
            raise ConfigError("config.json: 'norm.eps' must be positive")
        if "max_positions" not in d and len((tensor_shapes or {}).get("pos", ())) == 2:
            d = dict(d, max_positions=int(tensor_shapes["pos"][0]))
        cap = _number(d, "logit_softcap") if d.get("logit_softcap") is not None else None
        if cap is not None and not cap > 0:
            raise ConfigError(f"config.json: 'logit_softcap' = {cap} must be positive")
        eos = d.get("eos_token_id")
        stops = (eos,) if isinstance(eos, int) and not isinstance(eos, bool) else tuple(int(x) for x in eos) if isinstance(eos, list) else ()
        return cls(vocab=_pos_int(d, "vocab"), width=_pos_int(d, "width"), norm_eps=eps, residual_mult=_number(d, "residual_mult"),
                   max_positions=_pos_int(d, "max_positions"), layers=tuple(layers), loop=_loop(d, len(layers)), logit_softcap=cap,
                   bos_token_id=d.get("bos_token_id") if isinstance(d.get("bos_token_id"), int) else None, stop_token_ids=stops)

    @classmethod
    def from_dir(cls, model_dir: str) -> "ViroraxConfig":
        with open(os.path.join(model_dir, "config.json")) as f:
            d = json.load(f)
        if "max_positions" in d:
            return cls.from_dict(d)
        from ..weights.loader import tensor_shapes

        return cls.from_dict(d, tensor_shapes(model_dir))

    # ------------------------------------------------------------------- spec
    def _mixer_spec(self, l: ViroraxLayer, p: str):
        from ..parts.attention import AttentionSpec
        from ..parts.lightning import ConstantDecayAttentionSpec
        from ..parts.rotary import RotarySpec

        position = RotarySpec(rotary_dim=l.m("rot_dims"), theta=l.m("rot_base"), pairing="half") if l.m("rot_dims") else None
        if l.type == "retention":
            return ConstantDecayAttentionSpec(
                prefix=p, hidden_size=self.width, num_heads=l.m("heads"), key_dim=l.m("dim"), value_dim=l.m("vdim"), decay=l.m("decay"),
                norm_eps=self.norm_eps, activation="none", q_scale=float(l.m("dim")) ** -0.5, position=position, norm="head", norm_weight=False,
                gate="silu")
        return AttentionSpec(
            prefix=p, hidden_size=self.width, num_heads=l.m("heads"), num_kv_heads=l.m("kv_heads"), head_dim=l.m("dim"), scale=l.m("scale"),
            qk_norm_eps=self.norm_eps, position=position, window=l.m("window"), qk_norm="head", value_dim=l.m("vdim"), bias=True, out_bias=False,
            stored_sinks=True, head_gate=True,
            names=(("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_norm", "q.norm"), ("k_norm", "k.norm"), ("gate", "g"), ("sink", "sink")))

    def run_order(self) -> Tuple[Tuple[int, bool], ...]:
        """The layer runs: (layer, whether the embedding output joins the residual right before it)."""
        runs = [(i, False) for i in range(len(self.layers))]
        if self.loop is None:
            return tuple(runs)
        lo, hi = self.loop.start, self.loop.stop
        again = [(i, i == lo) for i in range(lo, hi)]
        return tuple(runs[:hi] + again * (self.loop.times - 1) + runs[hi:])

    def to_model_spec(self) -> ModelSpec:
        from ..parts.block import PreNormBlockSpec
        from ..parts.mlp import UngatedMlpSpec
        from ..parts.norm import RmsNormSpec

        blocks, ignored = [], []
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            if not l.ff:                    # a layer without a feed-forward has no use for its norm, should it be stored
                ignored.append(p + "norm2")
            blocks.append(PreNormBlockSpec(
                mixer_norm=RmsNormSpec(p + "norm1", self.width, self.norm_eps), mixer=self._mixer_spec(l, p + "mix."),
                ffn_norm=RmsNormSpec(p + "norm2", self.width, self.norm_eps) if l.ff else None,
                ffn=UngatedMlpSpec(prefix=p + "mlp.", hidden_size=self.width, intermediate_size=l.ff, activation="square_relu",
                                   names=("up", "down")) if l.ff else None))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, blocks=tuple(blocks),
            schedule=tuple(ScheduleEntry(i, add_embedding=again) for i, again in self.run_order()),
            final_norm=RmsNormSpec("final.norm", self.width, self.norm_eps), embed_name="embed", head_name=None, position_name="pos",
            branch_scale=self.residual_mult, logit_cap=self.logit_softcap, max_position=self.max_positions,
            stop_token_ids=self.stop_token_ids, bos_token_id=self.bos_token_id, ignored_tensors=tuple(ignored))
