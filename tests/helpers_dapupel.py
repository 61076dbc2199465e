"""Small Dapupel configurations and model folders for the tests (random weights of the tests' own making)."""
from __future__ import annotations

import json
import tempfile
from pathlib import Path

import torch

from tests import plain_dapupel as plain


def attention(heads, kv_heads, dim, size, conv=4, scale=None, softcap=15.0):
    return "attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, conv=conv, scale=scale or dim ** -0.5, softcap=softcap,
                             mask=dict(size=size))


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, base=10000.0, scale=None, scaling=(4.0, 64, 32.0, 1.0)):
    rot = dict(dims=rot_dim, base=base)
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return "latent_attention", dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank,
                                    scale=scale or (dim + rot_dim) ** -0.5, rot=rot)


def delta(heads, kv_heads, dim, vdim, conv=4, ranks=(5, 6)):
    return "channel_delta", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, ranks=list(ranks))


def moe(experts, top, ff, limit=1.5):
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit))


def layer(mix, mlp):
    return dict(type=mix[0], mixer=mix[1], mlp=mlp)


def config(vocab, width, streams, taps, eps, layers):
    return dict(architecture="Dapupel", vocab=vocab, width=width, streams=streams, canon=dict(taps=taps), norm=dict(eps=eps), layers=layers)


# sizes that are multiples of nothing: odd widths, shared key heads, a window shorter than a page, a layer without a feed-forward
DAP_ODD = config(53, 44, 3, 3, 1e-5, [
    layer(delta(6, 3, 10, 7, conv=2, ranks=(3, 5)), moe(6, 2, 14)),
    layer(attention(4, 2, 6, 9, conv=3, softcap=3.0), moe(5, 5, 10, limit=0.8)),
    layer(latent(3, 10, 6, 9, 14, 11, scaling=(8.0, 32, 16.0, 2.0)), None),
    layer(latent(2, 8, 4, 12, 20, 9, base=500.0, scaling=None), moe(4, 1, 9)),
    layer(attention(3, 1, 14, 70, conv=5), moe(3, 2, 11)),
])
# sizes that the tensor-core kernels and 16-byte paths take
DAP_FAST = config(320, 128, 4, 4, 1e-6, [
    layer(attention(4, 2, 64, 48), moe(8, 2, 64)),
    layer(latent(4, 32, 16, 32, 80, 64), moe(6, 3, 64)),
    layer(delta(4, 2, 32, 64, ranks=(16, 24)), moe(8, 1, 128)),
    layer(latent(8, 64, 32, 64, 96, 128, base=300000.0, scaling=(16.0, 128, 32.0, 1.0)), moe(8, 2, 64)),
    layer(attention(8, 8, 32, 130, softcap=5.0), None),
    layer(delta(3, 3, 64, 32, conv=3, ranks=(8, 8)), moe(8, 4, 64)),
])
# values that a given model may happen to make equal or 1
DAP_ONES = config(31, 32, 1, 1, 1e-5, [
    layer(attention(1, 1, 8, 1, conv=1), moe(1, 1, 8)),
    layer(delta(1, 1, 8, 8, conv=1, ranks=(1, 1)), moe(2, 2, 8)),
    layer(latent(1, 2, 2, 8, 8, 4), moe(2, 1, 8)),
])
# more streams and longer filters than usual, states wider than tall and the reverse, values wider than a single token's kernel takes
DAP_WIDE = config(60, 36, 7, 6, 1e-5, [
    layer(delta(2, 1, 130, 20, conv=6, ranks=(9, 2)), moe(4, 2, 16)),
    layer(delta(2, 2, 20, 140, ranks=(7, 4)), None),
    layer(latent(2, 16, 8, 24, 130, 40), moe(4, 2, 16)),
])

CONFIGS = {"odd": DAP_ODD, "fast": DAP_FAST, "ones": DAP_ONES, "wide": DAP_WIDE}


def make_model_dir(cfg: dict, seed: int, folder=None, store_dtype=torch.float32, weights=None):
    """config.json + model.safetensors with the tests' own random weights; returns the folder and the float32 weights."""
    from qwenforge_b200.weights import save_safetensors

    folder = Path(folder or tempfile.mkdtemp(prefix="dap_model_"))
    folder.mkdir(parents=True, exist_ok=True)
    weights = plain.random_weights(cfg, seed) if weights is None else weights
    (folder / "config.json").write_text(json.dumps(cfg))
    save_safetensors(folder / "model.safetensors", {k: v.to(store_dtype) for k, v in weights.items()})
    return folder, weights


def steady(cfg: dict, weights: dict, seed: int = 0) -> dict:
    """The same weights with routers that choose by clear margins, so that bfloat16 rounding flips (next to) no choice: a few channels
    carry a large number of either sign per token, no sublayer writes to them, the norms saturate there, and the routers read
    nothing else. The logits do not see those channels."""
    gen = torch.Generator().manual_seed(seed)
    n, width = 8, int(cfg["width"])
    w = {k: v.clone() for k, v in weights.items()}
    w["final.norm"][:n] = 0
    w["final.norm.b"][:n] = 0
    sign = lambda *shape: torch.randint(0, 2, shape, generator=gen).float() * 2 - 1
    w["embed"][:, :n] = 16.0 * sign(int(cfg["vocab"]), n)
    for name in list(w):
        if name.endswith("mix.o") or name.endswith(".down"):
            w[name][:n] = 0
        elif name.endswith(".router"):
            experts = w[name].shape[0]
            w[name].zero_()
            w[name][:, :n] = (3.0 * sign(experts, n) * (1.0 + torch.rand(experts, n, generator=gen))).to(torch.bfloat16).float()
        elif name.endswith("canon2"):
            w[name][:n, :-1] *= 0.25
    return w
