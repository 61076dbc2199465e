"""The Lasonex design on a GPU: each new kernel and kernel option against its plain reference, the model against the plain
implementation (tests/plain_lasonex.py) whole, decoded, cut into portions, in unequal batches, in slots, pages and state rows used
before, and through the engine's own entry point with greedy generation. The tests make their own small configurations
(tests/helpers_lasonex.py) and weights; where random weights would hide a fault (a key at the window's edge, the second map, a token
that only the state still holds), weights or inputs are made so that it shows. In bfloat16 the tests' routers choose by clear margins."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests import kernel_refs as refs
from tests import plain_lasonex as plain
from tests.helpers import max_err, random_tokens
from tests.helpers_lasonex import (CONFIGS, LAS_FAST, LAS_ODD, LAS_ONES, STRETCH, attention, config, dense, layer, make_model_dir, moe,
                                   retention, steady)

pytestmark = pytest.mark.gpu
DEV = "cuda"
BOTH = [torch.float32, torch.bfloat16]


def close(got, want, dtype, what="", f32=3e-5, bf16=1e-2):
    got, want = got.double().cpu(), want.double().cpu()
    bound = (f32 if dtype == torch.float32 else bf16) * (float(want.abs().max()) + 1e-9)
    err = float((got - want).abs().max())
    assert err <= bound, f"{what}: max |diff| {err:.3e} exceeds {bound:.3e}"


def expect(cfg, weights, tokens, margin=0.1):
    """The plain implementation's logits, and which rows' routers chose by a clear margin (of their logits) in every layer."""
    margins = []
    logits = plain.forward(cfg, weights, tokens, margins=margins)
    sure = torch.ones(len(tokens), dtype=torch.bool)
    for m in margins:
        sure &= m >= margin
    return logits, sure


def row_errors(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.square().mean(-1).sqrt() / want.std(-1)


def logits_close(got, want, dtype, what=""):
    """The difference with its mean taken off, root mean square over the vocabulary, against the spread of the logits."""
    want, sure = want if isinstance(want, tuple) else (want, torch.ones(want.shape[0], dtype=torch.bool))
    err = row_errors(got, want)
    if dtype == torch.float32:
        assert float(err.max()) <= 1e-4, f"{what}: worst row {float(err.max()):.3e} exceeds 1e-4"
    else:
        assert len(sure) < 4 or int(sure.sum()) >= len(sure) // 2, f"{what}: too few rows with a sure router to judge by"
        worst = float(err[sure].max()) if bool(sure.any()) else 0.0
        assert float(err.median()) <= 0.05 and worst <= 0.3, f"{what}: median {float(err.median()):.3e}, worst sure row {worst:.3e}"


def rand(g, *shape, dtype=torch.float32, spread=1.0):
    return (spread * torch.randn(*shape, generator=g)).to(dtype).to(DEV)


def ints(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


class Batch:
    """The integers of a step of sequences with the given slots and (start, length) spans."""

    def __init__(self, slots, spans):
        self.slots, self.n_seqs = ints(slots), len(slots)
        cu, seq, pos = [0], [], []
        for s, (start, length) in enumerate(spans):
            cu.append(cu[-1] + length)
            seq += [s] * length
            pos += list(range(start, start + length))
        self.cu_q, self.tok_seq, self.tok_pos, self.n_tokens = ints(cu), ints(seq), ints(pos), cu[-1]
        self.max_q_len = max(length for _, length in spans)


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", BOTH)
def test_embedding_rows_under_a_scale(dtype):
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(1)
    table, ids, err = rand(g, 40, 50, dtype=dtype), ints([3, 39, 0, 7]), ints([0])
    out = torch.empty(4, 50, device=DEV)
    ops.embed_gather(ids, table, out, err, 12.5)
    assert torch.equal(out, table[ids.long()].float() * 12.5)
    token_ids, pos, slots, steps = ints([1, 2, 3, 4]), ints([5, 6, 7, 8]), ints([0, 1, -1, 2]), ints([0] * 4)
    hidden, cursor, ticket = torch.zeros(4, 50, device=DEV), ints([0]), ints([0])
    ops.decode_advance_embed(ints([9, 8, 7, 6]), token_ids, pos, slots, steps, ints([9] * 4), ints([-1]), 1,
                             torch.full((2, 4), -1, dtype=torch.int32, device=DEV), cursor, table, hidden, ticket, err, 12.5)
    assert torch.equal(hidden, table[torch.tensor([9, 8, 3, 6], device=DEV)].float() * 12.5) and int(err) == 0


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("width", [45, 384, 1024, 1500, 2052, 4100, 4098])
def test_two_norms_of_one_stream_with_what_is_pending(dtype, width):
    """One or two outputs pending, none, or expert rows that are still to be summed; two norms, one, none; all rows or named ones."""
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(width)
    n, top = 19, 3
    hidden = rand(g, n, width, spread=3.0)
    a, b, rows = rand(g, n, width, dtype=dtype), rand(g, n, width, dtype=dtype), rand(g, n * top, width, dtype=dtype)
    w1, w2 = ((1 + 0.1 * torch.randn(width, generator=g)).to(dtype).to(DEV) for _ in range(2))
    dest = torch.randperm(n * top, generator=g).to(torch.int32).to(DEV)
    weight = torch.rand(n * top, generator=g).to(DEV)
    cpu = lambda t: t.cpu() if isinstance(t, torch.Tensor) else tuple(cpu(x) for x in t) if isinstance(t, tuple) else t
    cases = [(a, b, None), (a, None, None), (None, None, None), (a, rows, (dest, top, weight)), (None, rows, (dest, top, None)), (None, b, None)]
    for x, y, y_rows in cases:
        h_got, h_ref = hidden.clone(), hidden.clone().cpu()
        out = [torch.empty(n, width, dtype=dtype, device=DEV) for _ in range(2)]
        ref = [torch.empty(n, width, dtype=dtype) for _ in range(2)]
        ops.pair_rms_norm(h_got, x, y, w1, 1e-5, out[0], w2, 1e-3, out[1], b_rows=y_rows)
        refs.pair_rms_norm(h_ref, cpu(x), cpu(y), w1.cpu(), 1e-5, ref[0], w2.cpu(), 1e-3, ref[1], b_rows=cpu(y_rows))
        close(h_got, h_ref, torch.float32, "stream", f32=1e-6)
        close(out[0], ref[0], dtype, "first norm")
        close(out[1], ref[1], dtype, "second norm")
        only = torch.empty_like(out[0])
        h_one = hidden.clone()
        ops.pair_rms_norm(h_one, x, y, w1, 1e-5, only, b_rows=y_rows)
        assert torch.equal(only, out[0]) and torch.equal(h_one, h_got)
        if x is not None or y is not None:
            h_none = hidden.clone()
            ops.pair_rms_norm(h_none, x, y, b_rows=y_rows)
            assert torch.equal(h_none, h_got)
        picked, want = torch.empty(5, width, dtype=dtype, device=DEV), ints([18, 0, 7, 7, 3])
        h_kept = hidden.clone()
        ops.pair_rms_norm(h_kept, x, y, w1, 1e-5, picked, b_rows=y_rows, rows=want)
        assert torch.equal(h_kept, hidden) and torch.equal(picked, out[0][want.long()])
    err = ints([0])
    ops.pair_rms_norm(hidden.clone(), a, b, w1, 1e-5, torch.empty(1, width, dtype=dtype, device=DEV), rows=ints([n]), err=err)
    assert int(err) == ops.ERR_ROW_RANGE


class Site:
    def __init__(self, ops, dtype, kv_heads, head_dim, slots=4, pages=12, per_slot=3):
        self.storage = torch.full((pages, 2, kv_heads, 64, head_dim), 7.0, dtype=dtype, device=DEV)
        table = torch.full((slots, per_slot), -1, dtype=torch.int32)
        for s in range(slots):
            for i in range(per_slot):
                table[s, i] = (5 * (s * per_slot + i) + 1) % pages
        self.args = ops.KvSiteArgs(self.storage, table.to(DEV), kv_heads, head_dim)
        self.table = self.args.table


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,size", [(4, 2, 10, 14, 6, 32), (6, 2, 32, 64, 32, 64), (2, 1, 24, 40, 16, 64), (4, 4, 16, 32, 0, 32),
                                                        (1, 1, 64, 128, 48, 128), (3, 3, 9, 30, 8, 31)])
def test_heads_of_two_maps_into_the_cache(dtype, heads, kv, dim, vdim, rot, size):
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(dim)
    for spans, slots in (([(60, 7), (0, 1), (0, 5)], [2, 0, -1]), ([(130, 1), (5, 1)], [1, 3]), ([(0, 150), (3, 130)], [0, 2])):
        b = Batch(slots, spans)
        qkv = rand(g, b.n_tokens, (heads + kv) * 2 * dim + kv * vdim + 8, dtype=dtype)
        freq = torch.rand(rot // 2, generator=g).to(DEV) if rot else None
        site = Site(ops, dtype, kv, size)
        ref = Site(ops, dtype, kv, size)
        q, q_ref = (torch.full((b.n_tokens, heads * 2 * size), 5.0, dtype=dtype, device=DEV) for _ in range(2))
        err = ints([0])
        ops.rope_maps_cache_write(qkv, b.tok_seq, b.tok_pos, b.slots, freq, rot, 1.13, heads, 2, dim, vdim, q, site.args, True, err)
        refs.rope_maps_cache_write(qkv, b.tok_seq, b.tok_pos, b.slots, freq, rot, 1.13, heads, 2, dim, vdim, q_ref, ref.args, True, None)
        close(q, q_ref, dtype, "queries")
        close(site.storage, ref.storage, dtype, "cache")
        assert int(err) == 0
        again = torch.empty_like(q)
        kept = site.storage.clone()
        ops.rope_maps_cache_write(qkv, b.tok_seq, b.tok_pos, b.slots, freq, rot, 1.13, heads, 2, dim, vdim, again, site.args, False, err)
        assert torch.equal(again, q) and torch.equal(site.storage, kept)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,vdim,pitch", [(3, 14, 32), (5, 64, 64), (2, 13, 31), (4, 128, 128), (1, 256, 256), (7, 80, 96)])
def test_two_maps_brought_together(dtype, heads, vdim, pitch):
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(vdim)
    for n in (3, 900):
        x = rand(g, n, heads * 2 * pitch, dtype=dtype)
        out, want = torch.empty(n, heads * vdim, dtype=dtype, device=DEV), torch.empty(n, heads * vdim, dtype=dtype, device=DEV)
        ops.map_difference(x, pitch, 0.7, 1e-3, 0.65, out, heads, vdim)
        refs.map_difference(x, pitch, 0.7, 1e-3, 0.65, want, heads, vdim)
        close(out, want, dtype, f"{n} tokens", f32=2e-6)


@pytest.mark.parametrize("kv,pairs,size,vdim", [(2, 7, 64, 64), (1, 20, 32, 30), (2, 2, 96, 80), (4, 4, 128, 128), (1, 3, 128, 70)])
def test_single_tokens_with_the_maps_brought_together(kv, pairs, size, vdim):
    """The decode kernel's own combination (one run per sequence and several, groups beyond one tile of heads, a padding entry) against
    the plain attention and combination in float64."""
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(size + vdim)
    heads = 2 * pairs * kv
    for lengths, window, splits in (([130, 5, 640], 0, 4), ([700, 64, 65], 0, 1), ([700, 300, 1], 200, 3)):
        site = Site(ops, torch.bfloat16, kv, size, slots=4, pages=48, per_slot=12)
        site.storage.copy_(rand(g, *site.storage.shape, dtype=torch.bfloat16))
        site.storage[:, 1, :, :, vdim:] = 0
        table = torch.randperm(48, generator=g).to(torch.int32).view(4, 12).to(DEV)
        args = ops.KvSiteArgs(site.storage, table, kv, size)
        b = Batch([2, 0, 3, -1], [(n - 1, 1) for n in lengths] + [(0, 1)])
        q = rand(g, 4, heads * size, dtype=torch.bfloat16)
        scratch, err = ops.DecodeScratch(torch.device(DEV)), ints([0])
        out = torch.full((4, heads // 2 * vdim), 9.0, dtype=torch.bfloat16, device=DEV)
        for _ in range(2):   # (the second call meets the ticket counters as the first left them)
            ops.attention_decode(q, out, b.cu_q, b.tok_pos, b.slots, args, heads, 4, 0.2, window, splits, scratch, err, pairs=(0.6, 1e-4, 0.7, vdim))
        wide = torch.empty(4, heads * size, dtype=torch.float64, device=DEV)
        refs.attention_generic(q, wide, b.cu_q, b.tok_pos, b.slots, args, heads, 4, 1, 0.2, window, None)
        want = torch.empty(4, heads // 2 * vdim, dtype=torch.float64, device=DEV)
        refs.map_difference(wide, size, 0.6, 1e-4, 0.7, want, heads // 2, vdim)
        close(out[:3], want[:3], torch.bfloat16, f"{lengths} {splits}", bf16=1.5e-2)
        assert int(err) == 0 and float(out[3].abs().max()) == 0


def retention_case(g, n, heads, dim, vdim, dtype):
    width = heads * (2 * dim + 2 * vdim)
    proj = rand(g, n, width + (-width) % 8, dtype=dtype)
    cut = [0, heads * dim, 2 * heads * dim, 2 * heads * dim + heads * vdim, 2 * heads * (dim + vdim)]
    return [proj[:, cut[i]:cut[i + 1]] for i in range(4)]   # q, k, v, gate


@pytest.mark.parametrize("heads,dim,vdim,rot", [(3, 32, 64, 32), (2, 64, 64, 32), (1, 128, 128, 128), (2, 8, 8, 0), (2, 24, 40, 16), (1, 64, 128, 64),
                                                (4, 16, 32, 16)])
def test_retention_in_chunks(heads, dim, vdim, rot):
    """Unequal sequences with and without a slot, lengths around the chunk; states used before; far tokens that only the state still
    holds; decays from fast to none. The products are float32 to rounding: the reference is float64 on the same bfloat16 inputs."""
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(dim + vdim)
    decay = torch.tensor([1.0, 0.9990234375, 0.5, 0.05][:heads], dtype=torch.float64)
    powers = (decay[:, None] ** torch.arange(ops.RETENTION_CHUNK + 1)).float().to(DEV)
    freq = (torch.rand(rot // 2, generator=g) * 0.9).to(DEV) if rot else None
    size = heads * dim * vdim
    for spans, slots in (([(0, 200), (17, 64), (5, 1), (0, 65)], [2, 0, 1, -1]), ([(3, 2)], [1]), ([(0, 63), (0, 129), (400, 128)], [0, 1, 2])):
        b = Batch(slots, spans)
        q, k, v, gate = retention_case(g, b.n_tokens, heads, dim, vdim, torch.bfloat16)
        angles = ops.rope_table(b.tok_pos, freq, 1.1) if rot else None
        state = rand(g, 3, size + (-size) % 4 + 8)
        state_ref = state.clone()
        out, want = (torch.zeros(b.n_tokens, heads * vdim, dtype=torch.bfloat16, device=DEV) for _ in range(2))
        assert ops.retention_chunks_take(q, k, v, gate, state, 4, dim, vdim, rot)
        ops.retention_chunks(q, k, v, gate, angles, rot, powers, dim ** -0.5, 1e-5, b.cu_q, b.slots, b.max_q_len, state, 4, heads, dim, vdim, out)
        wide = torch.zeros(b.n_tokens, heads * vdim, dtype=torch.float64, device=DEV)
        refs._retention(q, k, v, gate, *((angles[..., 0].double(), angles[..., 1].double()) if rot else (None, None)), decay.to(DEV),
                        dim ** -0.5, 1e-5, b.cu_q, b.slots, state_ref, 4, heads, dim, vdim, wide)
        close(state, state_ref, torch.float32, f"states {spans}", f32=4e-6)
        close(out, wide, torch.bfloat16, f"outputs {spans}", bf16=5e-3)
        assert torch.equal(state[:, :4], state_ref[:, :4]) and torch.equal(state[:, 4 + size:], state_ref[:, 4 + size:])


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,dim,vdim,rot", [(3, 10, 6, 4), (2, 32, 64, 32), (1, 130, 20, 2), (1, 64, 300, 64), (4, 128, 128, 96), (1, 256, 1024, 0)])
def test_retention_of_single_tokens_and_the_scan(dtype, heads, dim, vdim, rot):
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(dim + vdim)
    decay = torch.tensor([0.96875, 1.0, 0.5, 0.99][:heads], dtype=torch.float32, device=DEV)
    freq = torch.rand(rot // 2, generator=g).to(DEV) if rot else None
    size = heads * dim * vdim
    pad = size + (-size) % 4
    b = Batch([2, -1, 0], [(9, 1), (0, 1), (700, 1)])
    q, k, v, gate = retention_case(g, 3, heads, dim, vdim, dtype)
    state = rand(g, 3, pad)
    state_ref, out = state.clone(), torch.empty(3, heads * vdim, dtype=dtype, device=DEV)
    want = torch.empty(3, heads * vdim, dtype=torch.float64, device=DEV)
    ops.retention_token(q, k, v, gate, b.tok_pos, freq, rot, 1.07, decay, dim ** -0.5, 1e-5, b.cu_q, b.slots, state, 0, heads, dim, vdim, out)
    refs.retention_token(q, k, v, gate, b.tok_pos, freq, rot, 1.07, decay, dim ** -0.5, 1e-5, b.cu_q, b.slots, state_ref, 0, heads, dim, vdim, want)
    close(out, want, dtype, "single tokens", bf16=5e-3)
    close(state, state_ref, torch.float32, "states", f32=2e-6)
    # a step of portions by rows and scan
    b = Batch([1, -1, 0], [(9, 40), (0, 3), (700, 2)])
    q, k, v, gate = retention_case(g, 45, heads, dim, vdim, dtype)
    angles = ops.rope_table(b.tok_pos, freq, 1.07) if rot else None
    rows, y = torch.empty(45, heads * (2 * dim + vdim), device=DEV), torch.empty(45, heads * vdim, device=DEV)
    ops.retention_rows(q, k, v, angles, rot, dim ** -0.5, heads, dim, vdim, rows)
    rows_ref = torch.empty_like(rows)
    refs.retention_rows(q, k, v, angles, rot, dim ** -0.5, heads, dim, vdim, rows_ref)
    close(rows, rows_ref, torch.float32, "rows", f32=1e-6)
    hd = heads * dim
    state_ref = state.clone()
    ops.outer_state_scan(rows[:, :hd], rows[:, hd:2 * hd], rows[:, 2 * hd:], decay, None, b.cu_q, b.slots, state, 0, -1, heads, heads, dim, vdim, 1.0, y, None)
    out, unit = torch.empty(45, heads * vdim, dtype=dtype, device=DEV), torch.ones(heads * vdim, dtype=dtype, device=DEV)
    ops.gated_group_norm(y, gate, unit, 1e-5, out, heads, heads, "silu", False)
    want = torch.empty(45, heads * vdim, dtype=torch.float64, device=DEV)
    refs._retention(q, k, v, gate, *((angles[..., 0].double(), angles[..., 1].double()) if rot else (None, None)), decay, dim ** -0.5, 1e-5,
                    b.cu_q, b.slots, state_ref, 0, heads, dim, vdim, want)
    close(out, want, dtype, "portions", bf16=5e-3)
    close(state, state_ref, torch.float32, "states after portions", f32=4e-6)


@pytest.mark.parametrize("dtype", BOTH)
def test_choice_among_groups_by_their_largest_softmax_score(dtype):
    """A group with one very good expert wins over one with two good ones; the weights are the softmax over the chosen."""
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(8)
    n, experts, top, width = 40, 12, 3, 32
    x, router = rand(g, n, width, dtype=dtype), rand(g, experts, width, dtype=dtype, spread=0.5)
    x_long = rand(g, 1500, width, dtype=dtype)
    for groups in ((3, 2), (4, 1), (1, 1), (12, 3), (2, 2)):
        for rows, best in ((x, 1), (x, 2), (x_long, 1)):
            logits = rows.float() @ router.float().T
            want = refs.moe_plan(logits.cpu(), top, True, True, groups=groups, group_best=best)
            for fused in (True, False) if rows is x else (False,):
                plan = ops.moe_plan(None if fused else logits, top, True, True, x=rows if fused else None, router=router if fused else None,
                                    groups=groups, group_best=best)
                at, rw = plan.dest.long().cpu().view(-1, top), want.dest.long().view(-1, top)
                offsets = plan.offsets.cpu()
                mine = (torch.searchsorted(offsets, at.flatten(), right=True) - 1).view(-1, top)
                assert torch.equal(mine.sort(-1).values, want.row_expert[rw].sort(-1).values), (groups, fused, best)
                assert max_err(plan.sorted_weight.cpu()[at].sort(-1).values, want.sorted_weight[rw].sort(-1).values) < 1e-5
    logits = torch.full((1, experts), -2.0)
    logits[0, 5], logits[0, 8], logits[0, 9] = 1.1, 1.0, 1.0
    pick = lambda best: ops.moe_plan(logits.to(DEV), 2, True, True, groups=(3, 1), group_best=best).offsets.cpu()
    assert int(pick(1)[8] - pick(1)[4]) == 2 and int(pick(2)[12] - pick(2)[8]) == 2


# ------------------------------------------------------------------ the model
def build(cfg, folder, dtype, seed=0, weights=None):
    """The model on the GPU and the weights it holds: in bfloat16 the plain implementation gets the rounded weights, and routers that
    choose by clear margins."""
    from qwenforge_b200.engine import Model
    weights = plain.random_weights(cfg, seed) if weights is None else weights
    if dtype == torch.bfloat16:
        weights = {k: v.to(torch.bfloat16).float() for k, v in steady(cfg, weights, seed).items()}
    folder, weights = make_model_dir(cfg, seed, folder, weights=weights)
    return Model.from_dir(folder, dtype, DEV), weights, folder


def run(model, cache, tokens, cuts):
    """One sequence fed in portions of the given sizes (the rest one by one); the logits of every position."""
    slot, at, got = cache.open(), 0, []
    for size in list(cuts) + [1] * (len(tokens) - sum(cuts)):
        got.append(model.step(cache, [(slot, tokens[at:at + size])], want=[list(range(size))]))
        at += size
    cache.close(slot)
    model.raise_on_kernel_error()
    return torch.cat(got)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_decoding_and_portions_agree_with_the_plain_implementation(dtype, name, tmp_path):
    cfg = CONFIGS[name]
    model, weights, _ = build(cfg, tmp_path, dtype)
    cache = model.new_cache(64 * 12, 3)
    tokens = random_tokens(cfg["vocab"], 300, 7)
    want = expect(cfg, weights, tokens)
    for cuts in ([300], [240], [2, 61, 2, 130, 65, 3, 2], [129, 128]):
        logits_close(run(model, cache, tokens, cuts), want, dtype, f"{name} cuts {cuts[:3]}")
    assert all(g.pages.n_free == g.pages.n_pages for g in cache.kv_groups)


LAS_LONG = config(1000, 320, 1e-6, 17.0, [
    layer(attention(10, 2, 32, 64, 300, 32, base=300000.0, scaling=STRETCH), dense(640)),
    layer(retention(5, 64, 128, 64), moe(12, 3, 96, groups=(4, 2))),
    layer(attention(4, 2, 64, 128, 520, 48, diff=0.7, base=1000.0), moe(20, 4, 48, groups=(5, 3))),
    layer(retention(3, 128, 64, 32), None),
    layer(attention(6, 3, 48, 96, 1100, 48, base=50000.0), moe(12, 3, 96)),
])


@pytest.mark.parametrize("dtype", BOTH)
def test_long_prompts_at_larger_sizes(dtype, tmp_path):
    """Steps of more than a thousand tokens: whole, with the last tokens decoded, and cut where the later portions reach back over
    many pages and chunks; and the kernels that are not the fast ones on the same prompt."""
    cfg, n = LAS_LONG, 1400
    model, weights, _ = build(cfg, tmp_path, dtype, seed=11)
    cache = model.new_cache(64 * 40, 3)
    tokens = random_tokens(cfg["vocab"], n, 5)
    want = expect(cfg, weights, tokens)
    for cuts in ([n], [n - 40], [1100, 200, 33]):
        logits_close(run(model, cache, tokens, cuts), want, dtype, f"cuts {cuts}")
    if dtype == torch.bfloat16:
        model.attention = "generic"
        logits_close(run(model, cache, tokens, [n - 3]), want, dtype, "plain attention kernel")
    assert all(g.pages.n_free == g.pages.n_pages for g in cache.kv_groups)


def test_the_residual_stream_after_every_layer(tmp_path):
    for name, cfg in (("odd", LAS_ODD), ("fast", LAS_FAST)):
        model, weights, _ = build(cfg, tmp_path / name, torch.float32)
        cache = model.new_cache(256, 2)
        tokens = random_tokens(cfg["vocab"], 50, 1)
        seen = {}
        model.observer = lambda i, hidden, delta: seen.__setitem__(i, (hidden if delta is None else hidden + delta.float()).clone())
        run(model, cache, tokens, [50])
        streams = []
        plain.forward(cfg, weights, tokens, streams)
        assert len(streams) == len(cfg["layers"])
        for i, stream in enumerate(streams):
            assert max_err(seen[i + 1], stream) < 5e-5 * (1 + float(stream.abs().max())), f"{name} after layer {i}"


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["odd", "fast"])
def test_unequal_batches_in_slots_used_before(dtype, name, tmp_path):
    """Requests of unequal lengths start together, are decoded together and end one by one; the second round runs in slots, pages and
    state rows that the first has used. Each request's logits equal those of the plain implementation alone."""
    cfg = CONFIGS[name]
    model, weights, _ = build(cfg, tmp_path, dtype, seed=2)
    cache = model.new_cache(64 * 10, 3)
    seqs = [random_tokens(cfg["vocab"], n, 30 + n) for n in (150, 3, 66, 1, 91)]
    want = [expect(cfg, weights, s) for s in seqs]
    for round_ in range(2):
        for batch in ([0, 1, 2], [3, 4]):
            slots = {i: cache.open() for i in batch}
            heads = {i: max(1, len(seqs[i]) - 20) for i in batch}
            logits = model.step(cache, [(slots[i], seqs[i][:heads[i]]) for i in batch], want=[list(range(heads[i])) for i in batch])
            got, o = {i: [] for i in batch}, 0
            for i in batch:
                got[i].append(logits[o:o + heads[i]])
                o += heads[i]
            fed = dict(heads)
            live = [i for i in batch if fed[i] < len(seqs[i])]
            while live:
                logits = model.step(cache, [(slots[i], [seqs[i][fed[i]]]) for i in live])
                for row, i in enumerate(live):
                    got[i].append(logits[row:row + 1])
                    fed[i] += 1
                live = [i for i in live if fed[i] < len(seqs[i])]
            for i in batch:
                cache.close(slots[i])
                logits_close(torch.cat(got[i]), want[i], dtype, f"round {round_} request {i}")
    model.raise_on_kernel_error()


@pytest.mark.parametrize("dtype", BOTH)
def test_keys_at_the_edges_of_windows_and_pages_and_tokens_far_back(dtype, tmp_path):
    """Windows of 65, 64 and 1 positions over pages of 64 with sharp scores (a scale that lets one key take the weight of its map), and
    decays that keep a token for hundreds of positions: prompts that end just inside and just outside a window, a page or a chunk,
    decoding across the edges, against the plain implementation. A window one position longer, a second map left out or a decay
    that is slightly off must show."""
    cfg = config(120, 48, 1e-6, 5.0, [
        layer(attention(4, 2, 16, 24, 65, 8, base=40000.0, scale=1.2, diff=0.3), dense(64)),
        layer(retention(2, 16, 24, 16, decay=[0.998046875, 1.0]), None),
        layer(attention(2, 2, 16, 32, 64, 16, base=900.0, scale=1.5, diff=0.5), moe(4, 2, 16, groups=(2, 1))),
        layer(attention(2, 1, 16, 16, 1, 0, scale=1.0), None),
        layer(retention(3, 8, 16, 0, decay=[0.9, 0.99, 0.9990234375]), dense(32))])
    tokens = random_tokens(cfg["vocab"], 460, 5)
    model, used, _ = build(cfg, tmp_path, dtype, seed=11)
    cache = model.new_cache(64 * 16, 2)
    want = expect(cfg, used, tokens)
    for cuts in ([460], [64], [65, 1, 1, 62, 1, 1, 100, 9], [129, 2], [63, 1, 1, 62, 2]):
        logits_close(run(model, cache, tokens, cuts), want, dtype, f"cuts {cuts}")
    # the mechanisms matter here: the same weights under a slightly different design give other logits
    def altered(change):
        layers = json.loads(json.dumps(cfg["layers"]))
        for e in layers:
            change(e["mixer"])
        return float(row_errors(plain.forward_logits({**cfg, "layers": layers}, used, tokens), want[0])[100:].median())
    longer = altered(lambda m: m["mask"].__setitem__("size", m["mask"]["size"] + 1) if "mask" in m else None)
    single = altered(lambda m: m.__setitem__("diff", m["diff"] - 0.3) if "diff" in m else None)
    faster = altered(lambda m: m.__setitem__("decay", [d * 0.99 for d in m["decay"]]) if "decay" in m else None)
    assert longer > 0.2 and single > 0.1 and faster > 0.1, (longer, single, faster)


@pytest.mark.parametrize("dtype", BOTH)
def test_long_decoding_passes_windows(dtype, tmp_path):
    cfg = config(90, 32, 1e-6, 4.0, [layer(attention(2, 1, 16, 16, 30, 16), moe(4, 2, 8, groups=(2, 1))),
                                     layer(retention(2, 8, 8, 8, decay=[0.9, 0.999]), dense(40)),
                                     layer(attention(4, 2, 32, 64, 100, 32, scaling=STRETCH), None)])
    model, weights, _ = build(cfg, tmp_path, dtype, seed=4)
    cache = model.new_cache(64 * 12, 2)
    tokens = random_tokens(cfg["vocab"], 420, 9)
    logits_close(run(model, cache, tokens, [3]), expect(cfg, weights, tokens), dtype)
    assert all(g.pages.n_free == g.pages.n_pages for g in cache.kv_groups)


def test_greedy_generation_through_the_engine(tmp_path):
    """StudentEngine.generate_ids (the scheduler's batches, CUDA-graph decoding with padding rows, prompt graphs) against greedy
    decoding of the plain implementation, in float32 where ties are the only way to differ."""
    from qwenforge_b200.engine import StudentEngine
    for name, cfg in (("odd", LAS_ODD), ("ones", LAS_ONES)):
        folder, weights = make_model_dir(cfg, 6, tmp_path / name)
        prompts = [random_tokens(cfg["vocab"], n, n) for n in (5, 70, 1, 33, 12)]
        want = [plain.greedy_generate(cfg, weights, p, 12) for p in prompts]
        for graphs in (True, False):
            engine = StudentEngine(str(folder), device=DEV, dtype="float32", cuda_graphs=graphs)
            got = engine.generate_ids(prompts, max_new_tokens=12, batch_size=3, ignore_eos=True)
            assert got == want, (name, graphs)
    # bfloat16: what the graphs replay is what the same kernels give launch by launch, and what the plain implementation would say
    weights = steady(LAS_FAST, plain.random_weights(LAS_FAST, 6))
    folder, _ = make_model_dir(LAS_FAST, 6, tmp_path / "fast", weights=weights)
    prompts = [random_tokens(LAS_FAST["vocab"], n, n) for n in (5, 170, 1, 33, 12)]
    made = [StudentEngine(str(folder), device=DEV, dtype="bfloat16", cuda_graphs=graphs).generate_ids(prompts, max_new_tokens=12, batch_size=5, ignore_eos=True)
            for graphs in (True, False)]
    assert all(len(t) == 12 for t in made[0])
    for prompt, tokens in zip(prompts, made[0]):
        logits = plain.forward_logits(LAS_FAST, weights, prompt + tokens)[len(prompt) - 1:-1]
        gap = logits.max(-1).values - logits.gather(1, torch.tensor(tokens)[:, None])[:, 0]
        assert float((gap / logits.std(-1)).max()) < 0.5   # every token is the plain implementation's best or next to it


def test_trace_replay_as_a_subprocess(tmp_path):
    cfg = LAS_ODD
    folder, weights = make_model_dir(cfg, 8, tmp_path / "m", store_dtype=torch.bfloat16)
    weights = {k: v.to(torch.bfloat16).float() for k, v in weights.items()}
    a, b = random_tokens(cfg["vocab"], 80, 1), random_tokens(cfg["vocab"], 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": [0, 69]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[70:71], "want": [0]}, {"id": "b", "tokens": b[8:], "want": [0]}], "end": ["b"]}]
    steps += [{"step": 2 + i, "entries": [{"id": "a", "tokens": [a[71 + i]], "want": [0]}], "end": ["a"] if i == 8 else []} for i in range(9)]
    root = Path(__file__).resolve().parent.parent
    out = tmp_path / "out"
    done = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                           "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                          timeout=900)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [l for l in done.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(11)]
    wa, wb = plain.forward_logits(cfg, weights, a), plain.forward_logits(cfg, weights, b)
    first = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(3, cfg["vocab"]))
    logits_close(first, torch.stack((wa[0], wa[69], wb[7])), torch.float32)
    second = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(2, cfg["vocab"]))
    logits_close(second, torch.stack((wa[70], wb[8])), torch.float32)
    last = torch.from_numpy(np.fromfile(out / "10.f32", dtype="<f4").reshape(1, cfg["vocab"]))
    logits_close(last, wa[79:80], torch.float32)
