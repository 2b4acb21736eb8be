"""The Levolix decoder: its typed configuration and its model description.

A Levolix ``config.json`` names the design in ``architecture`` and nests its sizes::

    {"architecture": "Levolix", "vocab": V, "width": d, "norm": {"eps": e},
     "layers": [{"type": "parallel",
                 "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}, "rot": {"base", "dims"}},
                           "right": {"heads", "kv_heads", "dim", "vdim", "conv": taps}, "left_scale", "right_scale"},
                 "mlp": null | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "identity", "top"}}},
                {"type": "retention",
                 "mixer": {"heads", "dim", "vdim", "decay": [one a head], "rot": {"base", "dims"}}, "mlp": ...}]}

The model (``parts/layer.py`` ``SandwichLayer`` without front norms): x <- x + N1(mixer(x)), then x <- x + N2(experts(x)), N an
RMS norm whose gain is stored less one. Mixers: ``retention`` = linear attention with a fixed decay a head and rotated halves;
``parallel`` = an attention inside fixed chunks of positions (biases, one norm over the whole query and the whole key
projection, neighbouring channels rotated, a one in the softmax denominator, a sigmoid gate per channel) beside a gated delta
rule (short convolutions, unit-length queries and keys), joined with two scales (``parts/attention.py``, ``parts/recurrent.py``,
``parts/side_by_side.py``). Feed-forward: silu experts and identity experts chosen by softmax score plus a correction, weights
the scores themselves (``parts/moe.py``). The output matrix is the embedding table.

Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.<q|k|v|g|o>``, ``l<i>.mix.left.<q|k|v|q.b|k.b|v.b|q.norm|k.norm|g|o>``,
``l<i>.mix.right.<q|k|v|q.conv|k.conv|v.conv|b|a|A_log|dt_bias|norm|g|o>``, ``l<i>.mlp.<router|correction|e<k>.gate|e<k>.up|
e<k>.down>``, ``final.norm``.
"""

from __future__ import annotations

from dataclasses import dataclass

from ..parts.spec import (AttentionSpec, EmbeddingSpec, GatedDeltaSpec, HeadSpec, LayerSpec, ModelSpec, NormSpec, PositionSpec,
                          RetentionSpec, RoutedExpertsSpec, SideBySideSpec, straight_schedule)
from .base import ConfigError, read_fields

UNIT_EPS = 1e-6             # inside the root of the delta rule's unit vectors


@dataclass(frozen=True)
class _Rot:
    base: float
    dims: int


@dataclass(frozen=True)
class _Mask:
    size: int


@dataclass(frozen=True)
class _Attention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: dict
    mask: dict


@dataclass(frozen=True)
class _Delta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class _Pair:
    left: dict
    right: dict
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class _Retention:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: dict


@dataclass(frozen=True)
class _Expert:
    ff: int


@dataclass(frozen=True)
class _Router:
    experts: int
    top: int
    identity: int = 0


@dataclass(frozen=True)
class _Moe:
    kind: str
    expert: dict
    router: dict


@dataclass(frozen=True)
class _Layer:
    type: str
    mixer: dict
    mlp: dict | None = None


@dataclass(frozen=True)
class _Norm:
    eps: float


MIXERS = ("parallel", "retention")


def _strict(cls, d, where):
    obj, unread = read_fields(cls, d, where)
    if unread:
        raise ConfigError(f"{where}: unknown key(s) {unread}")
    return obj


@dataclass(frozen=True)
class LevolixConfig:
    vocab: int
    width: int
    layers: tuple[dict, ...]
    norm: dict
    architecture: str = "Levolix"
    max_positions: int = 1 << 20        # the design sets no limit; tables are built for what the engine is asked to hold
    eos_token_id: int | tuple[int, ...] | None = None

    def __post_init__(self):
        def need(cond, msg):
            if not cond:
                raise ConfigError("config.json: " + msg)

        need(self.vocab > 0 and self.width > 0, f"vocab ({self.vocab}) and width ({self.width}) must be positive")
        need(len(self.layers) > 0, "layers is empty")
        object.__setattr__(self, "eps", _strict(_Norm, self.norm, "config.json: norm").eps)
        need(self.eps > 0, f"norm.eps must be positive, got {self.eps}")
        parsed = []
        for i, raw in enumerate(self.layers):
            where = f"config.json: layers[{i}]"
            L = _strict(_Layer, raw, where)
            need(L.type in MIXERS, f"layers[{i}].type {L.type!r} is not a known mixer {list(MIXERS)}")

            def rotation(d, dim, w):
                rot = _strict(_Rot, d, w + ".rot")
                need(0 <= rot.dims <= dim and rot.dims % 2 == 0 and rot.base > 0, f"{w}.rot: dims {rot.dims} of {dim} (even), base {rot.base}")
                return rot

            if L.type == "retention":
                m = _strict(_Retention, L.mixer, where + ".mixer")
                need(m.heads > 0 and 0 < m.dim <= 256 and m.vdim > 0, f"layers[{i}].mixer: heads {m.heads}, dim {m.dim} (at most 256), vdim {m.vdim}")
                need(len(m.decay) == m.heads and all(d >= 0.0 for d in m.decay),
                     f"layers[{i}].mixer.decay: {len(m.decay)} values for {m.heads} heads, none of them negative")
                mixer = (m, rotation(m.rot, m.dim, where + ".mixer"))
            else:
                pair = _strict(_Pair, L.mixer, where + ".mixer")
                a = _strict(_Attention, pair.left, where + ".mixer.left")
                need(a.heads > 0 and a.kv_heads > 0 and a.heads % a.kv_heads == 0, f"layers[{i}].mixer.left: heads {a.heads}, kv_heads {a.kv_heads}")
                need(0 < a.dim <= 256 and a.dim % 2 == 0 and 0 < a.vdim <= 256 and a.scale > 0,
                     f"layers[{i}].mixer.left: dim {a.dim} (even, at most 256), vdim {a.vdim} (at most 256), scale {a.scale}")
                mask = _strict(_Mask, a.mask, where + ".mixer.left.mask")
                need(mask.size > 0, f"layers[{i}].mixer.left.mask.size must be positive")
                d = _strict(_Delta, pair.right, where + ".mixer.right")
                need(d.heads > 0 and d.kv_heads > 0 and d.heads % d.kv_heads == 0 and 0 < d.dim <= 256 and d.vdim > 0 and 1 <= d.conv <= 16,
                     f"layers[{i}].mixer.right: heads {d.heads}, kv_heads {d.kv_heads}, dim {d.dim} (at most 256), vdim {d.vdim}, conv {d.conv} (1 to 16)")
                mixer = (pair, a, rotation(a.rot, a.dim, where + ".mixer.left"), mask, d)
            f = None
            if L.mlp is not None:
                moe = _strict(_Moe, L.mlp, where + ".mlp")
                need(moe.kind == "moe", f"layers[{i}].mlp.kind {moe.kind!r} is not 'moe'")
                ex, ro = _strict(_Expert, moe.expert, where + ".mlp.expert"), _strict(_Router, moe.router, where + ".mlp.router")
                need(ex.ff > 0 and ro.experts > 0 and ro.identity >= 0 and 0 < ro.top <= ro.experts + ro.identity, f"layers[{i}].mlp: {L.mlp}")
                f = (ex, ro)
            parsed.append((L.type, mixer, f))
        object.__setattr__(self, "parsed_layers", tuple(parsed))

    @property
    def stop_ids(self) -> tuple[int, ...]:
        if self.eos_token_id is None:
            return ()
        return (self.eos_token_id,) if isinstance(self.eos_token_id, int) else tuple(self.eos_token_id)


def _position(rot: _Rot, dim: int, pairing: str) -> PositionSpec:
    if rot.dims == 0:
        return PositionSpec(head_dim=dim, kind="none")
    return PositionSpec(head_dim=dim, theta=rot.base, rotary_dim=rot.dims, pairing=pairing, precise=True)


def levolix_model_spec(cfg: LevolixConfig, tensor_names=None) -> ModelSpec:
    d, eps = cfg.width, cfg.eps
    norm = NormSpec(d, eps, gain_offset=1.0)
    layers = []
    for i, (kind, m, f) in enumerate(cfg.parsed_layers):
        p = f"l{i}."
        names = {"post1.weight": p + "norm1"}
        if kind == "retention":
            r, rot = m
            mixer = RetentionSpec(hidden=d, heads=r.heads, head_dim=r.dim, value_dim=r.vdim, decay=r.decay,
                                  position=_position(rot, r.dim, "halves"), eps=eps)
            names.update({f"mixer.{n}.weight": p + "mix." + n for n in ("q", "k", "v", "g", "o")})
        else:
            pair, a, rot, mask, r = m
            lp, rp = p + "mix.left.", p + "mix.right."
            left = AttentionSpec(hidden=d, heads=a.heads, kv_heads=a.kv_heads, head_dim=a.dim, value_dim=a.vdim,
                                 position=_position(rot, a.dim, "neighbours"), qk_norm=True, qk_norm_eps=eps, qk_norm_span="projection",
                                 qkv_bias=True, scale=a.scale, chunk=mask.size, unit_sink=True, gate="channel")
            for n in ("q", "k", "v"):
                names[f"mixer.left.{n}_proj.weight"], names[f"mixer.left.{n}_proj.bias"] = lp + n, lp + n + ".b"
            for n in ("q", "k"):
                names[f"mixer.left.{n}_norm.weight"] = lp + n + ".norm"
            names["mixer.left.g_proj.weight"], names["mixer.left.o_proj.weight"] = lp + "g", lp + "o"
            right = GatedDeltaSpec(hidden=d, heads=r.heads, kv_heads=r.kv_heads, head_dim=r.dim, value_dim=r.vdim, conv_taps=r.conv,
                                   unit_eps=UNIT_EPS, eps=eps)
            for n in ("q", "k", "v", "g", "b", "a", "o", "norm"):
                names[f"mixer.right.{n}.weight"] = rp + n
            for n in ("q.conv", "k.conv", "v.conv", "A_log", "dt_bias"):
                names["mixer.right." + n] = rp + n
            mixer = SideBySideSpec(hidden=d, left=left, right=right, combine="scaled", left_scale=pair.left_scale,
                                   right_scale=pair.right_scale, eps=eps)
        ffn = None
        if f is not None:
            ex, ro = f
            names["post2.weight"] = p + "norm2"
            ffn = RoutedExpertsSpec(hidden=d, intermediate=ex.ff, experts=ro.experts, identity=ro.identity, top=ro.top, router_bias=False,
                                    scoring="softmax", choice_bias=True)
            names["ffn.router.weight"], names["ffn.correction"] = p + "mlp.router", p + "mlp.correction"
            for e in range(ro.experts):
                for n in ("gate", "up", "down"):
                    names[f"ffn.e{e}.{n}.weight"] = p + f"mlp.e{e}.{n}"
        layers.append(LayerSpec(mixer=mixer, ffn=ffn, norm1=None, norm2=None, post1=norm, post2=norm if ffn is not None else None,
                                names=names, kind="sandwich"))
    return ModelSpec(
        embedding=EmbeddingSpec(vocab=cfg.vocab, dim=d, name="embed"), layers=tuple(layers), schedule=straight_schedule(len(layers)),
        head=HeadSpec(vocab=cfg.vocab, dim=d, norm=norm, tied=True, norm_name="final.norm"), max_positions=cfg.max_positions)
