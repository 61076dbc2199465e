"""Small Lasonex configurations and model folders for the tests (random weights of the tests' own making)."""
from __future__ import annotations

import json
import tempfile
from pathlib import Path

import torch

from tests import plain_lasonex as plain

STRETCH = dict(factor=4.0, original=64, fast=8.0, slow=0.5)   # frequencies that the blend of both ends reaches at small sizes


def attention(heads, kv_heads, dim, vdim, size, rot_dims, diff=0.35, base=10000.0, scale=None, scaling=None):
    rot = dict(dims=rot_dims, base=base)
    if scaling is not None:
        rot["scaling"] = scaling
    return "attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, diff=diff, mask=dict(size=size), rot=rot)


def retention(heads, dim, vdim, rot_dims, decay=None, base=10000.0):
    return "retention", dict(heads=heads, dim=dim, vdim=vdim, decay=decay or [1.0 - 2.0 ** -(3 + 2 * i) for i in range(heads)],
                             rot=dict(dims=rot_dims, base=base))


def dense(ff, limit=1.5):
    return dict(kind="dense", ff=ff, limit=limit)


def moe(experts, top, ff, groups=None, limit=0.8):
    router = dict(experts=experts, top=top)
    if groups is not None:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(kind="moe", router=router, expert=dict(ff=ff, limit=limit))


def layer(mix, mlp):
    return dict(type=mix[0], mixer=mix[1], mlp=mlp)


def config(vocab, width, eps, scale, layers):
    return dict(architecture="Lasonex", vocab=vocab, width=width, embedding=dict(scale=scale), norm=dict(eps=eps), layers=layers)


# sizes that are multiples of nothing: values wider and narrower than two maps, odd widths, a window shorter than a page
LAS_ODD = config(53, 44, 1e-5, 3.0, [
    layer(attention(4, 2, 10, 14, 7, 6, scaling=STRETCH), moe(6, 2, 14, groups=(3, 2))),
    layer(retention(3, 10, 6, 4), None),
    layer(attention(3, 3, 6, 18, 90, 0, diff=0.6), dense(30)),
    layer(retention(2, 6, 22, 6, decay=[0.5, 0.999]), moe(5, 5, 12)),
    layer(attention(6, 2, 14, 10, 33, 14, base=500.0), moe(4, 1, 9, groups=(4, 1))),
])
# sizes that the tensor-core kernels and 16-byte paths take
LAS_FAST = config(320, 128, 1e-6, 7.0, [
    layer(retention(4, 32, 64, 32), dense(256)),
    layer(attention(6, 2, 32, 64, 48, 32, scaling=STRETCH), moe(6, 2, 64, groups=(3, 1))),
    layer(retention(2, 64, 32, 16, decay=[0.9, 1.0]), moe(8, 3, 64, groups=(4, 2))),
    layer(attention(8, 4, 16, 32, 70, 16), moe(8, 2, 64)),
    layer(attention(4, 1, 48, 80, 130, 32, diff=0.2), dense(128)),
    layer(retention(1, 128, 128, 64, decay=[0.97]), None),
    layer(attention(2, 2, 64, 128, 200, 64, scaling=STRETCH), moe(8, 4, 64, groups=(2, 1))),
])
# values that a given model may happen to make equal or 1
LAS_ONES = config(31, 32, 1e-5, 1.0, [
    layer(attention(1, 1, 16, 16, 1, 16, diff=0.5), moe(1, 1, 8)),
    layer(retention(1, 8, 8, 8, decay=[0.75]), dense(8)),
    layer(attention(2, 2, 8, 16, 64, 8, diff=0.8), moe(2, 2, 8, groups=(1, 1))),
])

CONFIGS = {"odd": LAS_ODD, "fast": LAS_FAST, "ones": LAS_ONES}


def make_model_dir(cfg: dict, seed: int, folder=None, store_dtype=torch.float32, weights=None):
    """config.json + model.safetensors with the tests' own random weights; returns the folder and the float32 weights."""
    from qwenforge_b200.weights import save_safetensors

    folder = Path(folder or tempfile.mkdtemp(prefix="las_model_"))
    folder.mkdir(parents=True, exist_ok=True)
    weights = plain.random_weights(cfg, seed) if weights is None else weights
    (folder / "config.json").write_text(json.dumps(cfg))
    save_safetensors(folder / "model.safetensors", {k: v.to(store_dtype) for k, v in weights.items()})
    return folder, weights


def steady(cfg: dict, weights: dict, seed: int = 0) -> dict:
    """The same weights with routers that choose by clear margins, so that bfloat16 rounding flips (next to) no choice: a few channels
    carry a large number of either sign per token, no sublayer writes to them, and the routers read nothing else. The logits do not
    see those channels."""
    gen = torch.Generator().manual_seed(seed)
    n, scale = 8, float(cfg["embedding"]["scale"])
    w = {k: v.clone() for k, v in weights.items()}
    w["final.norm"][:n] = 0
    sign = lambda *shape: torch.randint(0, 2, shape, generator=gen).float() * 2 - 1
    w["embed"][:, :n] = (2.0 / scale * sign(int(cfg["vocab"]), n)).to(torch.bfloat16).float()
    for name in list(w):
        if name.endswith("mix.o") or name.endswith(".down"):
            w[name][:n] = 0
        elif name.endswith(".router"):
            experts = w[name].shape[0]
            w[name].zero_()
            w[name][:, :n] = (2.0 * sign(experts, n) * (1.0 + torch.rand(experts, n, generator=gen))).to(torch.bfloat16).float()
    return w
