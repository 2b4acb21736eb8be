"""Tiny Nirozen configurations of the tests. They differ in every size and option: width (odd, even, multiples of 128),
vocabulary, the pair table's buckets and multipliers, embedding scale, norm eps; 1, 3, 5, 6 and 40 heads, key and value widths
equal and unequal, query ranks below and above the key/value rank, latent ranks that the tensor-core kernels take (multiples
of 16) and ranks they do not, head sizes that the tcgen05 prompt kernel takes and ones it does not; experts with top 1, 2, 3
and all, one expert, with and without a shared expert; layers without a feed-forward; the loop over the first layers three
times, over inner layers twice, over one layer once, over all layers four times, and absent."""

from __future__ import annotations


def attention(heads, dim, vdim, q_rank, kv_rank, scale=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
            "scale": scale if scale is not None else dim ** -0.5}


def moe(experts, top, ff, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def layer(m, f):
    return {"type": "latent_attention", "mixer": m, "mlp": f}


# odd sizes everywhere (the general kernels), an odd width (the last channel of the position vector is a sine), a layer
# without feed-forward inside the loop
S = {"architecture": "Nirozen", "vocab": 211, "width": 75, "norm": {"eps": 1e-6},
     "embedding": {"scale": 11.0, "bigram": {"buckets": 89, "mul_prev": 7, "mul_cur": 13}},
     "layers": [layer(attention(3, 12, 20, 28, 36, scale=0.37), moe(5, 2, 18, shared=26)),
                layer(attention(5, 10, 6, 50, 21), None),
                layer(attention(3, 12, 20, 17, 44), moe(6, 1, 22, shared=10))],
     "loop": {"start": 1, "stop": 3, "times": 2}}

# the loop starts at layer 0 and runs three times; sizes the latent tensor-core kernels take; no shared expert in one layer
T = {"architecture": "Nirozen", "vocab": 259, "width": 128, "norm": {"eps": 2e-5},
     "embedding": {"scale": 9.0, "bigram": {"buckets": 1021, "mul_prev": 1, "mul_cur": 259}},
     "layers": [layer(attention(6, 32, 48, 40, 80), moe(8, 3, 48, shared=64)),
                layer(attention(6, 48, 32, 72, 48, scale=0.2), moe(9, 2, 32))],
     "loop": {"start": 0, "stop": 2, "times": 3}}

# one head and forty heads (more than a tile of sixteen or thirty-two rows); all experts chosen; no loop
U = {"architecture": "Nirozen", "vocab": 203, "width": 64, "norm": {"eps": 1e-5},
     "embedding": {"scale": 14.0, "bigram": {"buckets": 40, "mul_prev": 3, "mul_cur": 2}},
     "layers": [layer(attention(1, 16, 8, 24, 24), moe(4, 4, 16, shared=24)),
                layer(attention(40, 8, 8, 24, 32), moe(7, 3, 24, shared=8)),
                layer(attention(2, 16, 16, 32, 16), None)]}

# sizes that send prompts of 128 tokens and more through the tensor-memory products and, with equal key and value widths of
# 64 and 128, through the tcgen05 attention; single tokens through the weight-streaming kernel; a loop over one layer, once.
# Only the last layer's experts are a choice, so that a close call touches its own token's row and no other
V = {"architecture": "Nirozen", "vocab": 640, "width": 384, "norm": {"eps": 1e-6},
     "embedding": {"scale": 10.0, "bigram": {"buckets": 4099, "mul_prev": 641, "mul_cur": 3}},
     "layers": [layer(attention(5, 64, 64, 192, 128), moe(4, 4, 128, shared=192)),
                layer(attention(3, 128, 128, 160, 272), moe(2, 2, 128, shared=128)),
                layer(attention(6, 32, 64, 128, 96), moe(16, 4, 64, shared=96))],
     "loop": {"start": 2, "stop": 3, "times": 1}}

# one expert of which one is chosen, a loop over all layers four times, pair-table multipliers whose products do not fit 32 bits
W = {"architecture": "Nirozen", "vocab": 150, "width": 96, "norm": {"eps": 1e-5},
     "embedding": {"scale": 8.0, "bigram": {"buckets": 200003, "mul_prev": 1000003, "mul_cur": 999983}},
     "layers": [layer(attention(4, 16, 16, 32, 32), moe(1, 1, 40, shared=24)),
                layer(attention(2, 32, 24, 16, 48), None)],
     "loop": {"start": 0, "stop": 2, "times": 4}}

CONFIGS = {"S": S, "T": T, "U": U, "V": V, "W": W}
SEEDS = {"S": 171, "T": 272, "U": 373, "V": 474, "W": 575}
STD = 0.08


def sharpen(folder, logit_std: float = 3.0) -> None:
    """Rewrite a written folder so that faults show: queries are scaled until attention is far from uniform; the sinks become
    distinct numbers of the size of the scores, so that a sink that is left out, scaled or counted per slice moves the
    result; norm gains lie well away from one; the pair table's rows and the pass vectors are as large as the token rows; the
    routers' rows are scaled until their logits have about ``logit_std`` and the router biases are distinct multiples of 0.7
    in a shuffled order, so that they decide a good part of the choices."""
    from pathlib import Path

    import torch

    from plain.qwen3_plain import read_safetensors
    from sleuth_b200.weights.safetensors import write_safetensors
    path = Path(folder) / "model.safetensors"
    tensors = read_safetensors(path)
    for name, t in tensors.items():
        g = torch.Generator().manual_seed(t.numel() + len(name))
        if name.endswith(".mix.uq"):
            tensors[name] = t * 4.0
        elif name.endswith(".mix.sink"):
            tensors[name] = 0.4 + 2.6 * (torch.randperm(t.numel(), generator=g).to(t.dtype) + 0.5) / t.numel()
        elif name.endswith((".norm1", ".norm2", "final.norm")):
            tensors[name] = t * 4.0
        elif name in ("bigram", "loop.step"):
            tensors[name] = t * 8.0
        elif name.endswith(".mlp.router"):
            tensors[name] = t * (logit_std / (float(t.float().std()) * t.shape[1] ** 0.5)) if t.numel() > 1 else t
        elif name.endswith(".mlp.router.b"):
            tensors[name] = (torch.randperm(t.numel(), generator=g).to(t.dtype) - (t.numel() - 1) / 2) * 0.7
    write_safetensors(tensors, path, metadata={"format": "pt"})
