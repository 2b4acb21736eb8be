"""The Nirozen decoder: its typed configuration and its model description.

A Nirozen ``config.json`` names the design in ``architecture`` and nests its sizes::

    {"architecture": "Nirozen", "vocab": V, "width": d, "norm": {"eps": e},
     "embedding": {"scale": s, "bigram": {"buckets": n, "mul_prev": a, "mul_cur": b}},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "vdim", "q_rank", "kv_rank", "scale"},
                 "mlp": null | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}, "shared": {"ff"}}}, ...],
     "loop": {"start", "stop", "times"}}

The model: x = E[token] * s + B[(previous token * a + token * b) mod n] (B's last row for a sequence's first token) + a
sinusoidal vector of the token's position (base 10,000; ``parts/ends.py``). A layer is pre-norm (``parts/layer.py``),
x += mixer(norm1 x), x += ff(norm2 x), with RMS norms whose gains are stored less one. The mixer is attention through
low-rank latents without any position of its own (``parts/latent_attention.py``): queries and keys/values each through a
normed latent, a sink per head in the softmax, an output gate per channel. The feed-forward is routed SiLU experts
weighted by the softmax over the chosen logits, plus a shared expert (``parts/moe.py``), or none. Layers ``loop.start ..
loop.stop - 1`` run ``loop.times`` times in a row with the same weights and caches of their own, every pass (the first
too) beginning with the addition of its row of ``loop.step``. Final norm, untied output matrix.

Tensor names: ``embed``, ``bigram``, ``loop.step``, ``l<i>.norm1``, ``l<i>.norm2``,
``l<i>.mix.<dq|dq.norm|uq|dkv|dkv.norm|uk|uv|sink|g|o>``, ``l<i>.mlp.<router|router.b|e<k>.<gate|up|down>|
shared.<gate|up|down>>``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from dataclasses import dataclass

from ..parts.spec import (EmbeddingSpec, GatedMLPSpec, HeadSpec, LatentAttentionSpec, LayerSpec, ModelSpec, NormSpec,
                          PairEmbeddingSpec, PositionSpec, RoutedExpertsSpec, looped_schedule, straight_schedule)
from .base import ConfigError, read_fields


@dataclass(frozen=True)
class _Mixer:
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float


@dataclass(frozen=True)
class _Moe:
    kind: str
    expert: dict
    router: dict
    shared: dict | None = None


@dataclass(frozen=True)
class _ExpertSizes:
    ff: int


@dataclass(frozen=True)
class _Router:
    experts: int
    top: int


@dataclass(frozen=True)
class _Layer:
    type: str
    mixer: dict
    mlp: dict | None = None


@dataclass(frozen=True)
class _Loop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class _Norm:
    eps: float


@dataclass(frozen=True)
class _Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class _Embedding:
    scale: float = 1.0
    bigram: dict | None = None


MIXERS = ("latent_attention",)
POSITION_BASE = 10000.0         # of the sinusoidal position vectors; fixed by the design


def _strict(cls, d, where):
    """``read_fields`` that also refuses keys the class does not name: a key that nobody reads is a part of the model
    that would silently be left out."""
    obj, unread = read_fields(cls, d, where)
    if unread:
        raise ConfigError(f"{where}: unknown key(s) {unread}")
    return obj


@dataclass(frozen=True)
class NirozenConfig:
    vocab: int
    width: int
    layers: tuple[dict, ...]
    norm: dict
    embedding: dict | None = None
    loop: dict | None = None
    architecture: str = "Nirozen"
    max_positions: int = 1 << 20        # the design sets no limit: positions are worked out where they are used
    eos_token_id: int | tuple[int, ...] | None = None

    def __post_init__(self):
        def need(cond, msg):
            if not cond:
                raise ConfigError("config.json: " + msg)

        need(self.vocab > 0 and self.width > 0, f"vocab ({self.vocab}) and width ({self.width}) must be positive")
        need(len(self.layers) > 0, "layers is empty")
        object.__setattr__(self, "eps", _strict(_Norm, self.norm, "config.json: norm").eps)
        need(self.eps > 0, f"norm.eps must be positive, got {self.eps}")
        emb = _strict(_Embedding, self.embedding, "config.json: embedding") if self.embedding is not None else _Embedding()
        bg = _strict(_Bigram, emb.bigram, "config.json: embedding.bigram") if emb.bigram is not None else None
        if bg is not None:
            need(bg.buckets > 0 and bg.mul_prev >= 0 and bg.mul_cur >= 0,
                 f"embedding.bigram: buckets {bg.buckets}, multipliers {bg.mul_prev}, {bg.mul_cur}")
        object.__setattr__(self, "embedding_scale", emb.scale)
        object.__setattr__(self, "bigram", bg)
        parsed = []
        for i, raw in enumerate(self.layers):
            where = f"config.json: layers[{i}]"
            L = _strict(_Layer, raw, where)
            need(L.type in MIXERS, f"layers[{i}].type {L.type!r} is not a known mixer {list(MIXERS)}")
            m = _strict(_Mixer, L.mixer, where + ".mixer")
            for key in ("heads", "dim", "vdim", "q_rank", "kv_rank"):
                need(getattr(m, key) > 0, f"layers[{i}].mixer.{key} must be positive, got {getattr(m, key)}")
            f = None
            if L.mlp is not None:
                moe = _strict(_Moe, L.mlp, where + ".mlp")
                need(moe.kind == "moe", f"layers[{i}].mlp.kind {moe.kind!r} is not 'moe'")
                ex = _strict(_ExpertSizes, moe.expert, where + ".mlp.expert")
                ro = _strict(_Router, moe.router, where + ".mlp.router")
                sh = _strict(_ExpertSizes, moe.shared, where + ".mlp.shared") if moe.shared is not None else None
                need(ex.ff > 0 and 0 < ro.top <= ro.experts and (sh is None or sh.ff > 0),
                     f"layers[{i}].mlp: expert.ff {ex.ff}, router.experts {ro.experts}, router.top {ro.top}, shared {L.mlp.get('shared')}")
                f = (ex, ro, sh)
            parsed.append((m, f))
        object.__setattr__(self, "parsed_layers", tuple(parsed))
        lp = _strict(_Loop, self.loop, "config.json: loop") if self.loop is not None else None
        if lp is not None:
            need(0 <= lp.start <= lp.stop <= len(self.layers) and lp.times >= 1,
                 f"loop {self.loop} does not fit {len(self.layers)} layers")
        object.__setattr__(self, "parsed_loop", lp)

    @property
    def stop_ids(self) -> tuple[int, ...]:
        if self.eos_token_id is None:
            return ()
        return (self.eos_token_id,) if isinstance(self.eos_token_id, int) else tuple(self.eos_token_id)


def nirozen_model_spec(cfg: NirozenConfig, tensor_names=None) -> ModelSpec:
    d, eps = cfg.width, cfg.eps

    def centred():
        return NormSpec(d, eps, gain_offset=1.0)

    layers = []
    for i, (m, f) in enumerate(cfg.parsed_layers):
        p = f"l{i}."
        names = {"norm1.weight": p + "norm1"}
        for local, theirs in (("dq.weight", "dq"), ("dq_norm.weight", "dq.norm"), ("uq.weight", "uq"), ("dkv.weight", "dkv"),
                              ("dkv_norm.weight", "dkv.norm"), ("uk.weight", "uk"), ("uv.weight", "uv"), ("sinks", "sink"),
                              ("g.weight", "g"), ("o.weight", "o")):
            names["mixer." + local] = p + "mix." + theirs
        mixer = LatentAttentionSpec(
            hidden=d, heads=m.heads, plain_dim=m.dim, rot_dim=0, value_dim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank,
            scale=m.scale, norm_eps=eps, sinks=True, position=PositionSpec(head_dim=0, kind="none"))
        ffn = None
        if f is not None:
            ex, ro, sh = f
            ffn = RoutedExpertsSpec(
                hidden=d, intermediate=ex.ff, experts=ro.experts, top=ro.top, activation="silu", router_bias=True,
                shared=GatedMLPSpec(hidden=d, intermediate=sh.ff, activation="silu") if sh is not None else None)
            names.update({"norm2.weight": p + "norm2", "ffn.router.weight": p + "mlp.router", "ffn.router.bias": p + "mlp.router.b"})
            for e in [f"e{k}" for k in range(ro.experts)] + (["shared"] if sh is not None else []):
                for local in ("gate", "up", "down"):
                    names[f"ffn.{e}.{local}.weight"] = p + f"mlp.{e}.{local}"
        layers.append(LayerSpec(mixer=mixer, ffn=ffn, norm1=centred(), norm2=centred() if ffn is not None else None,
                                names=names, kind="prenorm"))
    lp = cfg.parsed_loop
    if lp is not None and lp.stop > lp.start:
        schedule = looped_schedule(len(layers), lp.start, lp.stop, lp.times, entry="row")
        pass_rows, rows, ignored = "loop.step", lp.times, ()
    else:
        schedule, pass_rows, rows, ignored = straight_schedule(len(layers)), None, 0, (r"loop\.step$",)
    bg = cfg.bigram
    if bg is not None:
        embedding = PairEmbeddingSpec(vocab=cfg.vocab, dim=d, buckets=bg.buckets, mul_prev=bg.mul_prev, mul_cur=bg.mul_cur,
                                      scale=cfg.embedding_scale, names={"weight": "embed", "pairs": "bigram"},
                                      sinusoid=POSITION_BASE)
    else:
        embedding = EmbeddingSpec(vocab=cfg.vocab, dim=d, scale=cfg.embedding_scale, name="embed", sinusoid=POSITION_BASE)
    return ModelSpec(
        embedding=embedding, layers=tuple(layers), schedule=schedule,
        head=HeadSpec(vocab=cfg.vocab, dim=d, norm=centred(), tied=False, norm_name="final.norm", name="head"),
        max_positions=cfg.max_positions, pass_rows=pass_rows, pass_rows_count=rows, ignored_tensors=ignored)
