"""Typed configuration of the Soputar decoder and its description as a
``ModelSpec``.

config.json of this design is nested: ``vocab``, ``width``, ``norm.eps``,
``embedding.scale`` and a list ``layers``; every layer names its mixer
(``type``: ``attention``, ``latent_attention`` or ``delta``) with the mixer's
sizes and constants (``mixer``) and its feed-forward (``mlp``: ``kind``
``dense``, or null for none).  Tensors: ``embed``, ``l<i>.norm1``,
``l<i>.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.

A sublayer reads the residual stream itself and its result is normed before it
joins: x <- x + norm(f(x)).  Every norm of the stream is an RMS norm whose
weight is stored as its distance from one.

Mixers.  ``attention``: grouped-query softmax attention without rotation and
without biases; the whole query row and the whole key row are RMS-normed
before they are split into heads; the query is multiplied by a temperature
1 + coef ln(floor((p + 1) / every) + 1) that grows with its position
(``q_temp``), the scaled score is capped (``softcap``); a layer with
``kv_from`` reads an earlier layer's keys and values.  ``latent_attention``:
keys and values through a normed latent of ``kv_rank`` numbers beside one
rotated key part of ``rot_dim`` dimensions that all heads share (neighbouring
pairs, plain frequencies), queries straight from the stream, a learned sink
per head in the softmax's denominator.  ``delta``: the gated delta rule with a
short convolution (``conv`` taps) and SiLU on q, k and v, unit norms on q and
k, a decay and a step size per head, a gated norm per head behind it.

Feed-forward ``dense``: g = min(W_gate h, limit), u = clamp(W_up h, +-limit),
W_down (g sigmoid(1.702 g) (u + 1)).
"""

from __future__ import annotations

import copy
import math
from dataclasses import dataclass, field

from ..errors import ConfigError
from .fusasun import _number
from .spec import BlockSpec, LayerCall, ModelSpec, PartSpec, TensorSpec
from .tifapel import _need, _positive_int

_MIXERS = ("attention", "latent_attention", "delta")
# what the design fixes
GATE_SLOPE = 1.702              # the feed-forward's gate: g * sigmoid(GATE_SLOPE * g)
UP_SHIFT = 1.0                  # and the 1 of (u + 1)
UNIT_EPS = 1e-6                 # under the root of the delta rule's unit vectors
NORM_OFFSET = 1.0               # a stream norm's gain is this plus its stored weight
# random weights: a stored norm weight lies around zero, a convolution's taps around zero, decays of a few per cent
NORM_INIT = (0.0, 0.1)
CONV_INIT = (0.0, 0.5)
A_LOG_INIT = (0.0, 0.5)
DT_BIAS_INIT = (-3.0, 0.5)
SINK_INIT = (0.0, 1.0)


@dataclass
class SoputarConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: list                       # as in config.json: dicts with type / mixer / mlp
    max_positions: int = 1 << 20       # the design has no limit of its own; the cache's size is the limit
    torch_dtype: str = "bfloat16"
    extra: dict = field(default_factory=dict)
    generation: dict = field(default_factory=dict)

    # ---- reading -----------------------------------------------------------

    @classmethod
    def from_dict(cls, d: dict) -> "SoputarConfig":
        norm = _need(d, "norm", "the top level")
        known = {"architecture", "architectures", "vocab", "width", "norm", "embedding", "layers", "max_positions",
                 "torch_dtype"}
        cfg = cls(vocab=_need(d, "vocab", "the top level"), width=_need(d, "width", "the top level"),
                  eps=_number(_need(norm, "eps", "norm"), "norm.eps"),
                  embedding_scale=_number(_need(_need(d, "embedding", "the top level"), "scale", "embedding"),
                                          "embedding.scale"),
                  layers=copy.deepcopy(_need(d, "layers", "the top level")),
                  max_positions=int(d.get("max_positions") or (1 << 20)),
                  torch_dtype=d.get("torch_dtype") or "bfloat16",
                  extra={k: v for k, v in d.items() if k not in known})
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        d = dict(self.extra)
        d.update(architecture="Soputar", vocab=self.vocab, width=self.width, norm={"eps": self.eps},
                 embedding={"scale": self.embedding_scale}, layers=copy.deepcopy(self.layers),
                 torch_dtype=self.torch_dtype)
        if self.max_positions != 1 << 20:
            d["max_positions"] = self.max_positions
        return d

    # ---- checks ------------------------------------------------------------

    def validate(self) -> None:
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        if not self.eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.eps!r}")
        if not isinstance(self.layers, list) or not self.layers:
            raise ConfigError("'layers' must be a non-empty list")
        if self.torch_dtype not in ("bfloat16", "float32"):
            raise ConfigError(f"torch_dtype {self.torch_dtype!r}: supported are bfloat16 and float32")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"{where}.type {kind!r}: this design has {', '.join(_MIXERS)}")
            m = _need(layer, "mixer", where)
            if kind == "attention":
                self._check_attention(i, m, where + ".mixer")
            elif kind == "latent_attention":
                self._check_latent(m, where + ".mixer")
            else:
                self._check_delta(m, where + ".mixer")
            mlp = layer.get("mlp")
            if mlp is not None:
                kind = _need(mlp, "kind", where + ".mlp")
                if kind != "dense":
                    raise ConfigError(f"{where}.mlp.kind {kind!r}: 'dense' (or null for no feed-forward)")
                _positive_int(_need(mlp, "ff", where + ".mlp"), where + ".mlp.ff")
                if not _number(_need(mlp, "limit", where + ".mlp"), where + ".mlp.limit") > 0:
                    raise ConfigError(f"{where}.mlp.limit must be positive")

    @staticmethod
    def _check_heads(m: dict, where: str, keys) -> None:
        for key in keys:
            _positive_int(_need(m, key, where), f"{where}.{key}")
        if "kv_heads" in keys and m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv_heads")

    def _check_attention(self, i: int, m: dict, where: str) -> None:
        self._check_heads(m, where, ("heads", "kv_heads", "dim", "vdim"))
        _number(_need(m, "scale", where), where + ".scale")
        if m.get("softcap") is not None and not _number(m["softcap"], where + ".softcap") > 0:
            raise ConfigError(f"{where}.softcap must be positive")
        temp = m.get("q_temp")
        if temp is not None:
            _number(_need(temp, "coef", where + ".q_temp"), where + ".q_temp.coef")
            _positive_int(_need(temp, "every", where + ".q_temp"), where + ".q_temp.every")
        if m.get("kv_from") is not None:
            j = m["kv_from"]
            if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < i:
                raise ConfigError(f"{where}.kv_from {j!r}: an earlier layer's index")
            owner = self.layers[j]
            if owner.get("type") != "attention" or owner["mixer"].get("kv_from") is not None:
                raise ConfigError(f"{where}.kv_from {j}: layer {j} has no keys and values of its own")
            for key in ("kv_heads", "dim", "vdim"):
                if owner["mixer"].get(key) != m[key]:
                    raise ConfigError(f"{where}.{key} {m[key]} differs from layer {j}'s {owner['mixer'].get(key)}")

    @classmethod
    def _check_latent(cls, m: dict, where: str) -> None:
        cls._check_heads(m, where, ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        _number(_need(m, "scale", where), where + ".scale")
        rot = _need(m, "rot", where)
        dims = _positive_int(_need(rot, "dims", where + ".rot"), where + ".rot.dims")
        if dims % 2 or dims != m["rot_dim"]:
            raise ConfigError(f"{where}.rot.dims {dims} must be even and equal rot_dim {m['rot_dim']}")
        if not _number(_need(rot, "base", where + ".rot"), where + ".rot.base") > 0:
            raise ConfigError(f"{where}.rot.base must be positive")

    @classmethod
    def _check_delta(cls, m: dict, where: str) -> None:
        cls._check_heads(m, where, ("heads", "kv_heads", "dim", "vdim", "conv"))

    # ---- derived ----------------------------------------------------------------

    def n_params(self) -> int:
        return sum(math.prod(t.shape) for t in self.to_spec().tensors())

    def summary(self) -> str:
        kinds = "".join(layer["type"][0] for layer in self.layers)
        return (f"soputar: {len(self.layers)} layers ({kinds}), width {self.width}, vocab {self.vocab}, "
                f"eps {self.eps:g}, {self.n_params() / 1e6:.1f} M params, {self.torch_dtype}")

    # ---- description as parts ------------------------------------------------

    def _mixer(self, p: str, kind: str, m: dict):
        """(mixer, position) of one layer whose tensors start with ``p``."""
        d, eps = self.width, self.eps
        matrix = lambda name, *shape: TensorSpec(p + "mix." + name, shape)
        vector = lambda name, n, init=None: TensorSpec(p + "mix." + name, (n,), "vector", init)
        H, Dv = m["heads"], m["vdim"]
        if kind == "attention":
            G, D = m["kv_heads"], m["dim"]
            own = m.get("kv_from") is None
            tensors = dict(q=matrix("q", H * D, d), q_norm=vector("q.norm", H * D), o=matrix("o", d, H * Dv))
            if own:
                tensors.update(k=matrix("k", G * D, d), v=matrix("v", G * Dv, d), k_norm=vector("k.norm", G * D))
            temp = m.get("q_temp")
            return PartSpec("gqa_attention", dict(
                hidden_size=d, n_heads=H, n_kv_heads=G, head_dim=D, v_head_dim=Dv, scale=float(m["scale"]), window=None,
                qk_norm_eps=eps, qk_norm="rows", own_kv=own,
                softcap=None if m.get("softcap") is None else float(m["softcap"]),
                q_temp=None if temp is None else (float(temp["coef"]), int(temp["every"]))), tensors), None
        if kind == "latent_attention":
            D, R, rank = m["dim"], m["rot_dim"], m["kv_rank"]
            tensors = dict(q=matrix("q", H * (D + R), d), dkv=matrix("dkv", rank + R, d),
                           dkv_norm=vector("dkv.norm", rank), uk=matrix("uk", H * D, rank), uv=matrix("uv", H * Dv, rank),
                           sink=vector("sink", H, SINK_INIT), o=matrix("o", d, H * Dv))
            mixer = PartSpec("latent_attention", dict(
                hidden_size=d, n_heads=H, head_dim=D, rot_dim=R, v_head_dim=Dv, q_rank=0, kv_rank=rank, eps=eps,
                scale=float(m["scale"]), window=None, out_gate=None, cache="latent"), tensors)
            return mixer, PartSpec("rope_neox", dict(n_rot=R, base=float(m["rot"]["base"]), angles="float32",
                                                     pairing="neighbours"))
        G, D, taps = m["kv_heads"], m["dim"], m["conv"]
        conv = lambda name, n: TensorSpec(p + "mix." + name + ".conv", (n, taps), "vector", CONV_INIT)
        tensors = dict(q=matrix("q", G * D, d), k=matrix("k", G * D, d), v=matrix("v", H * Dv, d),
                       q_conv=conv("q", G * D), k_conv=conv("k", G * D), v_conv=conv("v", H * Dv),
                       b=matrix("b", H, d), a=matrix("a", H, d), a_log=vector("A_log", H, A_LOG_INIT),
                       dt_bias=vector("dt_bias", H, DT_BIAS_INIT), norm=vector("norm", Dv), g=matrix("g", H * Dv, d),
                       o=matrix("o", d, H * Dv))
        return PartSpec("gated_delta", dict(
            hidden_size=d, n_heads=H, n_kv_heads=G, head_dim=D, v_head_dim=Dv, conv_taps=taps, eps=eps,
            unit_eps=UNIT_EPS, q_scale=float(D) ** -0.5), tensors), None

    def _feed_forward(self, p: str, mlp):
        if mlp is None:
            return PartSpec("none", {}, {})
        d, ff = self.width, mlp["ff"]
        return PartSpec("gated_mlp", dict(
            hidden_size=d, intermediate_size=ff,
            activation=("clamped_swish", GATE_SLOPE, float(mlp["limit"]), UP_SHIFT)),
            dict(gate=TensorSpec(p + "mlp.gate", (ff, d)), up=TensorSpec(p + "mlp.up", (ff, d)),
                 down=TensorSpec(p + "mlp.down", (d, ff))))

    def to_spec(self) -> ModelSpec:
        d, eps = self.width, self.eps
        norm = lambda name: PartSpec("rms_norm", dict(size=d, eps=eps, gain_offset=NORM_OFFSET),
                                     dict(gain=TensorSpec(name, (d,), "vector", NORM_INIT)))
        blocks, schedule, entry_of = [], [], {}
        for i, layer in enumerate(self.layers):
            p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
            mixer, position = self._mixer(p, layer["type"], m)
            norms = dict(mixer_post=norm(p + "norm1"))
            if mlp is not None:
                norms.update(feed_forward_post=norm(p + "norm2"))
            blocks.append(BlockSpec("post_norm", mixer, self._feed_forward(p, mlp), norms, position))
            j = m.get("kv_from") if layer["type"] == "attention" else None
            if j is None:
                entry_of[i] = len(entry_of)
                schedule.append(LayerCall(layer=i, cache=entry_of[i]))
            else:
                schedule.append(LayerCall(layer=i, cache=entry_of[j], writes_cache=False))
        return ModelSpec(
            architecture="Soputar", hidden_size=d, vocab_size=self.vocab,
            embedding=PartSpec("gather", dict(scale=self.embedding_scale), dict(table=TensorSpec("embed", (self.vocab, d)))),
            blocks=tuple(blocks), schedule=tuple(schedule), final_norm=norm("final.norm"),
            head=PartSpec("linear", dict(softcap=None), dict(weight=TensorSpec("head", (self.vocab, d)))),
            max_positions=self.max_positions, stop_ids=(), storage_dtype=self.torch_dtype, default_sampling={},
        )
