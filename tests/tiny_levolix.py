"""Tiny Levolix configurations of the tests. They differ in every size and option: width, vocabulary, eps; chunks of positions
shorter than a page, of exactly a page, of a page and one, of one token, and longer than any test sequence; 1 to 8 query heads
on 1 to 4 key/value heads; key and value widths equal and unequal, in and out of the tensor-core sizes; whole, partial and no
rotation; delta rules with as many heads as key heads and with several a key head, key widths 8 to 136 (every tiling of the
recurrence's kernels), value widths that are no multiple of 4, convolutions of 1 to 5 taps; retentions with one to five heads and
decays from 0.5 to 1; experts with top 1, 2, 3 and all, one expert, none to five identity experts, and layers without
feed-forward; both orders of the two mixers."""

from __future__ import annotations


def att(heads, kv, dim, vdim, scale, chunk, base, dims):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk}, "rot": {"base": base, "dims": dims}}


def delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts, identity, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}


def par(left, right, ls, rs, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": ls, "right_scale": rs}, "mlp": mlp}


def ret(heads, dim, vdim, decay, base, dims, mlp):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": dims}}, "mlp": mlp}


# odd sizes everywhere (the general kernels); chunks shorter than a page and of a page; a retention first
F = {"architecture": "Levolix", "vocab": 203, "width": 72, "norm": {"eps": 1e-5},
     "layers": [ret(3, 12, 20, [0.9, 1.0, 0.97], 100.0, 8, moe(5, 2, 2, 36)),
                par(att(4, 2, 24, 16, 0.3, 37, 300.0, 16), delta(6, 2, 12, 10, 3), 0.7, 1.2, moe(4, 0, 1, 20)),
                ret(1, 40, 72, [0.999], 50.0, 40, None),
                par(att(3, 3, 16, 40, 0.2, 64, 1000.0, 16), delta(2, 2, 40, 24, 1), 1.1, 0.4, moe(3, 5, 3, 16))]}

# widths that send bfloat16 prompts through the tensor-memory products and single tokens through the weight-streaming kernel,
# attention on the tensor-core kernels (64 and 128 channels), chunks of a page and one and of 200 positions, wide states
H = {"architecture": "Levolix", "vocab": 320, "width": 256, "norm": {"eps": 1e-6},
     "layers": [par(att(8, 4, 64, 64, 0.125, 65, 10000.0, 64), delta(4, 2, 64, 64, 4), 0.9, 0.8, moe(8, 8, 2, 64)),
                ret(4, 64, 128, [0.96875, 0.99, 0.9995, 0.5], 20000.0, 64, moe(6, 2, 8, 64)),
                par(att(4, 1, 128, 96, 0.1, 200, 500.0, 64), delta(3, 1, 96, 48, 5), 1.0, 1.0, None),
                ret(2, 136, 32, [0.98, 0.995], 10000.0, 0, moe(1, 1, 1, 40))]}

# a chunk of one token (a token sees itself alone) and one longer than any test sequence; no rotation; a key
# width beyond the chunked kernels'; every expert an ordinary one, and all chosen
J = {"architecture": "Levolix", "vocab": 150, "width": 96, "norm": {"eps": 2e-5},
     "layers": [par(att(2, 1, 32, 24, 0.25, 1, 100.0, 0), delta(1, 1, 136, 20, 2), 0.5, 1.5, moe(4, 0, 4, 24)),
                ret(5, 8, 16, [0.6, 0.7, 0.9, 0.99, 1.0], 30.0, 4, moe(2, 1, 1, 48)),
                par(att(6, 2, 8, 8, 0.5, 5000, 100.0, 8), delta(4, 4, 8, 12, 4), 1.3, 0.9, moe(1, 5, 2, 8))]}

CONFIGS = {"F": F, "H": H, "J": J}
SEEDS = {"F": 517, "H": 628, "J": 739}
STD = 0.08


def sharpen(folder, steady: bool = False, logit_std: float = 3.0) -> None:
    """Rewrite a written folder so that faults show. The layers have no front norms: the embedding's rows are scaled to the size
    that the closing norms give the sublayers' results. The routers' rows are scaled until their logits have about
    ``logit_std``, and the corrections are large enough to move choices; with ``steady`` they lie so far apart that they alone
    choose (the same experts for every token, the weights still the token's own scores): a bfloat16 run, whose rounding may turn
    a close choice and with it everything behind it, can then be compared row by row. The attention's norms give scores that are
    far from uniform and not dwarfed by the one in the denominator, and the delta rules forget slowly (small step sizes)."""
    from pathlib import Path

    from plain.qwen3_plain import read_safetensors
    from sleuth_b200.weights.safetensors import write_safetensors
    path = Path(folder) / "model.safetensors"
    tensors = read_safetensors(path)
    for name, t in tensors.items():
        if name == "embed":
            tensors[name] = t * (0.3 / STD)
        elif name.endswith(".mlp.router"):
            tensors[name] = t * (logit_std / (float(t.float().std()) * 2.0 * t.shape[1] ** 0.5))
        elif name.endswith(".mlp.correction"):
            tensors[name] = t.argsort().argsort().to(t.dtype) * 2.0 if steady else t
        elif name.endswith(".dt_bias"):
            tensors[name] = t - 2.5
        elif name.endswith((".q.norm", ".k.norm")):
            tensors[name] = t * 1.5
        elif name.endswith((".q.b", ".k.b", ".v.b")):
            tensors[name] = t * 4.0
    write_safetensors(tensors, path, metadata={"format": "pt"})
