"""The Dapupel design on a GPU: each new kernel and kernel option against its plain reference, the model against the plain
implementation (tests/plain_dapupel.py) whole, decoded, cut into portions, in unequal batches, in slots, pages and state
rows used before, and through the engine's own entry point with greedy generation. The tests make their own small
configurations (tests/helpers_dapupel.py) and weights; where random weights would hide a fault (a key at the window's edge,
a key far back), weights or inputs are made so that it shows."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests import kernel_refs as refs
from tests import plain_dapupel as plain
from tests.helpers import max_err, random_tokens
from tests.helpers_dapupel import CONFIGS, DAP_FAST, DAP_ODD, DAP_ONES, attention, config, delta, latent, layer, make_model_dir, moe, steady

pytestmark = pytest.mark.gpu
DEV = "cuda"
BOTH = [torch.float32, torch.bfloat16]


def close(got, want, dtype, what="", f32=3e-5, bf16=3e-2):
    got, want = got.double().cpu(), want.double().cpu()
    scale = float(want.abs().max()) + 1e-9
    bound = (f32 if dtype == torch.float32 else bf16) * scale
    err = float((got - want).abs().max())
    assert err <= bound, f"{what}: max |diff| {err:.3e} exceeds {bound:.3e}"


def expect(cfg, weights, tokens, margin=0.1):
    """The plain implementation's logits, and which rows' routers chose by a clear margin (of their logits) in every layer: in
    bfloat16 a router whose two candidates are closer than the rounding of its input may choose the other one, and such a
    row says nothing about the kernels."""
    margins = []
    logits = plain.forward(cfg, weights, tokens, margins=margins)
    sure = torch.ones(len(tokens), dtype=torch.bool)
    for m in margins:
        sure &= m >= margin
    return logits, sure


def logits_close(got, want, dtype, what=""):
    """The difference with its mean taken off, root mean square over the vocabulary, against the spread of the logits.
    `want`: logits, or (logits, rows whose routers chose by a clear margin)."""
    want, sure = want if isinstance(want, tuple) else (want, torch.ones(want.shape[0], dtype=torch.bool))
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    err = d.square().mean(-1).sqrt() / want.std(-1)
    if dtype == torch.float32:
        assert float(err.max()) <= 1e-4, f"{what}: worst row {float(err.max()):.3e} exceeds 1e-4"
    else:   # the typical row within rounding, and no row lost: a wrong key, a mask one position off or a lost state moves
        # every later row by about its whole spread, which the median sees; among the rows whose routers were sure hardly
        # one may stand out (a token before it whose router was not sure reaches it through keys and states)
        assert int(sure.sum()) >= max(1, len(sure) // 2), f"{what}: too few rows with a sure router to judge by"
        far = float((err[sure] > 0.4).double().mean())
        assert float(err[sure].median()) <= 0.06 and far <= 0.03 and float(err.max()) <= 1.6, \
            f"{what}: median {float(err[sure].median()):.3e}, {far:.1%} of the sure rows over 0.4, worst {float(err.max()):.3e}"


def rand(g, *shape, dtype=torch.float32, spread=1.0):
    return (spread * torch.randn(*shape, generator=g)).to(dtype).to(DEV)


def ints(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def cpu(t):
    return t.cpu() if isinstance(t, torch.Tensor) else tuple(cpu(x) for x in t) if isinstance(t, tuple) else t


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
        self.longest = max(length for _, length in spans)


def paged(n_slots, pages_per_slot, kv_heads, head_dim, planes, dtype, seed=0):
    """A paged cache whose slots hold pages in no particular order: the site on the GPU and its copy on the CPU."""
    from qwenforge_b200 import ops
    order = torch.randperm(n_slots * pages_per_slot + 3, generator=torch.Generator().manual_seed(seed))[:n_slots * pages_per_slot]
    table = order.to(torch.int32).view(n_slots, pages_per_slot).contiguous()
    storage = torch.zeros(n_slots * pages_per_slot + 3, planes, kv_heads, 64, head_dim, dtype=dtype)
    return (ops.KvSiteArgs(storage.to(DEV), table.to(DEV), kv_heads, head_dim), ops.KvSiteArgs(storage.clone(), table, kv_heads, head_dim))


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("width,n,taps", [(44, 3, 3), (128, 4, 4), (36, 7, 6), (256, 2, 2), (64, 1, 1), (896, 4, 4), (20, 8, 16)])
def test_streams_between_two_sublayers(dtype, width, n, taps):
    """Portions of unequal lengths, single tokens, a sequence without a slot; first from one row that stands for every stream, then
    from streams with a pending output (plain, or rows to be summed); the cut changes no bit."""
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(width)
    coefficients = (rand(g, n, n), rand(g, n))
    in_w, filt = rand(g, n), rand(g, width, taps, spread=0.5)
    norm = (rand(g, width, dtype=dtype), rand(g, width, dtype=dtype), 0.7)
    total, top = 83, 3
    X, y = rand(g, total, n, width, spread=2.0), rand(g, total, width, dtype=dtype)
    rows, dest, by = rand(g, total * top, width, dtype=dtype), torch.randperm(total * top, generator=g).to(torch.int32).to(DEV), rand(g, total * top).abs()
    keep = (taps - 1) * width

    def step(batch, pick, state, kind, on_gpu):
        move = (lambda t: t) if on_gpu else cpu
        source = X[pick] if kind != "start" else X[pick][:, 0].contiguous()
        yy = None if kind == "start" else y[pick]
        y_rows = None
        if kind == "rows":   # token t's rows stay where they are
            at = torch.arange(len(pick), device=DEV)
            yy, chosen = rows, dest.view(total, top)[pick].reshape(-1).contiguous()
            y_rows = (chosen, top, by)
        new = torch.full((len(pick), n, width), 7.0, device=DEV) if kind != "start" else None
        out = torch.empty(len(pick), width, dtype=dtype, device=DEV)
        new, out = move(new), move(out)
        conv = (move(filt), move(batch.cu_q), move(batch.slots), batch.longest, state, 4)
        fn = ops.streams_norm if on_gpu else refs.streams_norm
        fn(move(source), n, None if kind == "start" else move(coefficients), move(yy), move(in_w), new, move(norm), out, conv=conv,
           y_rows=move(y_rows))
        return new, out

    for kind in ("start", "plain", "rows"):
        state, state_ref = torch.zeros(4, 4 + keep + 4, device=DEV), torch.zeros(4, 4 + keep + 4)
        state[2, 4:4 + keep] = state_ref[2, 4:4 + keep] = 0.5      # a slot that its sequence has used before this step
        pick = list(range(total))
        batch = Batch([1, -1, 2], [(0, 60), (0, 20), (9, 3)])
        new, out = step(batch, pick, state, kind, True)
        new_ref, out_ref = step(batch, pick, state_ref, kind, False)
        close(out, out_ref, dtype, f"{kind} out", f32=1e-5, bf16=1e-2)
        close(state, state_ref, torch.float32, f"{kind} state", f32=1e-5)
        if new is not None:
            close(new, new_ref, torch.float32, f"{kind} streams", f32=1e-5)
        # the first sequence again in portions and single tokens, beside the third
        state2 = torch.zeros(4, 4 + keep + 4, device=DEV)
        at, pieces = 0, []
        for length in (1, 2, 17, 8, 1, 31):
            both = Batch([3, -1], [(at, length), (0, 1)])
            piece = step(both, list(range(at, at + length)) + [70], state2, kind, True)[1]
            pieces.append(piece[:length])
            at += length
        assert torch.equal(torch.cat(pieces), out[:60]), kind
        assert torch.equal(state2[3], state[1])


@pytest.mark.parametrize("dtype", BOTH)
def test_sum_of_the_streams_and_rows_of_it(dtype):
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(2)
    for width, n in ((44, 3), (128, 4)):
        X, y, coefficients = rand(g, 30, n, width), rand(g, 30, width, dtype=dtype), (rand(g, n, n), rand(g, n))
        norm = (rand(g, width, dtype=dtype), rand(g, width, dtype=dtype), 1.3)
        total, want = torch.empty(30, width, device=DEV), torch.empty(30, width)
        ops.streams_norm(X, n, coefficients, y, None, None, None, total)
        refs.streams_norm(cpu(X), n, cpu(coefficients), cpu(y), None, None, None, want)
        close(total, want, torch.float32, "total", f32=1e-5)
        rows, err = ints([29, 0, 7, 7]), torch.zeros(1, dtype=torch.int32, device=DEV)
        out, want = torch.empty(4, width, dtype=dtype, device=DEV), torch.empty(4, width, dtype=dtype)
        ops.streams_norm(X, n, coefficients, y, None, None, norm, out, rows=rows, err=err)
        refs.streams_norm(cpu(X), n, cpu(coefficients), cpu(y), None, None, cpu(norm), want, rows=rows.cpu())
        close(out, want, dtype, "rows", f32=1e-5, bf16=1e-2)
        assert int(err) == 0
        ops.streams_norm(X, n, coefficients, y, None, None, norm, out, rows=ints([29, 30, 7, -1]), err=err)
        assert int(err) == ops.ERR_ROW_RANGE


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,groups,dim,vdim", [(6, 3, 10, 7), (2, 2, 32, 64), (3, 1, 64, 64), (2, 2, 130, 20), (1, 1, 8, 8), (2, 1, 128, 128),
                                                   (2, 2, 20, 140), (4, 4, 256, 36)])
def test_delta_rule(dtype, heads, groups, dim, vdim):
    """The scan against the reference, whole and in portions of any remainder by four; single tokens' own kernel; a sequence without
    a slot and sequences that start anywhere in the batch; what lies beside the state in a slot's row stays as it was."""
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(dim + vdim)
    size, n = heads * dim * vdim, 75
    q, k, v = rand(g, n, groups * dim, dtype=dtype), rand(g, n, groups * dim, dtype=dtype), rand(g, n, heads * vdim, dtype=dtype)
    z, bias, rate = rand(g, n, heads * dim), rand(g, heads * dim), rand(g, heads)
    logit = rand(g, n, heads + 2, spread=2.0)[:, :heads]
    wide = torch.cat((q, k, v), dim=1)     # (rows of a wider product)
    q, k, v = wide[:, :groups * dim], wide[:, groups * dim:2 * groups * dim], wide[:, 2 * groups * dim:]

    def args(batch, rows, state, on_gpu):
        move = (lambda t: t) if on_gpu else cpu
        return tuple(move(t) for t in (q[rows], k[rows], v[rows], z[rows], bias, rate, logit[rows], batch.cu_q, batch.slots, state)) \
            + (5, heads, groups, dim, vdim, dim ** -0.5)

    def scan(batch, rows, state, on_gpu=True):
        y = torch.empty(len(rows), heads * vdim, device=DEV if on_gpu else "cpu")
        (ops if on_gpu else refs).delta_scan(*args(batch, rows, state, on_gpu), y)
        return y

    state, state_ref = torch.zeros(4, 5 + size + 3, device=DEV), torch.zeros(4, 5 + size + 3)
    whole = Batch([1], [(0, n)])
    y, y_ref = scan(whole, list(range(n)), state), scan(whole, list(range(n)), state_ref, False)
    close(y, y_ref, torch.float32, "whole", f32=2e-5)
    close(state, state_ref, torch.float32, "state", f32=2e-5)
    assert float(state[:, :5].abs().max()) == 0 and float(state[:, 5 + size:].abs().max()) == 0
    at, pieces = 0, []
    for length in (33, 1, 1, 38, 2):
        both = Batch([2, -1], [(at, length), (0, 3)])
        pieces.append(scan(both, list(range(at, at + length)) + [0, 1, 2], state)[:length])
        at += length
    close(torch.cat(pieces), y_ref, torch.float32, "portions", f32=3e-5)
    close(state[2], state_ref[1], torch.float32, "state of the portions", f32=3e-5)
    # unequal sequences side by side, in slots of their own
    spans = [(0, 7), (0, 1), (0, 30), (0, 2)]
    several, several_ref = torch.zeros(4, 5 + size + 3, device=DEV), torch.zeros(4, 5 + size + 3)
    rows = list(range(7)) + [9] + list(range(20, 50)) + [60, 61]
    y4, y4_ref = scan(Batch([2, 0, 1, 3], spans), rows, several), scan(Batch([2, 0, 1, 3], spans), rows, several_ref, False)
    close(y4, y4_ref, torch.float32, "several", f32=2e-5)
    close(several, several_ref, torch.float32, "their states", f32=2e-5)
    # single tokens: the state of the first 60 from the scan, then one by one, in the kernel that also norms and gates
    norm, gate = rand(g, vdim, dtype=dtype), rand(g, n, heads * vdim, dtype=dtype)
    scan(Batch([3], [(0, 60)]), list(range(60)), state)
    fused = vdim <= ops.DELTA_FUSED_MAX_VDIM
    for t in range(60, n):
        batch, rows = Batch([3, -1], [(t, 1), (0, 1)]), [t, 0]
        single, out = torch.empty(2, heads * vdim, device=DEV), torch.empty(2, heads * vdim, dtype=dtype, device=DEV)
        ops.delta_token(*args(batch, rows, state, True), y=single, **(dict(norm=norm, eps=1e-5, gate=gate[rows], out=out) if fused else {}))
        close(single[0], y_ref[t], torch.float32, f"token {t}", f32=5e-5)
        if fused:
            r = y_ref[t].double().view(heads, vdim)
            r = r / torch.sqrt(r.square().mean(-1, keepdim=True) + 1e-5) * norm.double().cpu()
            close(out[0], r.reshape(-1) * torch.sigmoid(gate[t].double().cpu()), dtype, f"normed token {t}", f32=2e-4, bf16=2e-2)
    close(state[3], state_ref[1], torch.float32, "state of single tokens", f32=5e-5)


@pytest.mark.parametrize("dtype", BOTH)
def test_latents_and_a_rotated_key_part_into_the_cache(dtype):
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(1)
    for q_rank, kv_rank, rot, row in ((11, 14, 6, 20), (64, 80, 16, 96), (200, 600, 8, 640), (0, 40, 8, 64)):
        batch = Batch([1, 0, -1], [(60, 9), (3, 1), (0, 4)])
        down = rand(g, batch.n_tokens, q_rank + kv_rank + rot)
        wq, wk = rand(g, max(q_rank, 1), dtype=dtype), rand(g, kv_rank, dtype=dtype)
        freq = torch.rand(rot // 2, generator=g).to(DEV)
        site, site_ref = paged(2, 2, 1, row, 1, dtype)
        lat, lat_ref = torch.empty(batch.n_tokens, max(q_rank, 1), dtype=dtype, device=DEV), torch.empty(batch.n_tokens, max(q_rank, 1), dtype=dtype)
        err = torch.zeros(1, dtype=torch.int32, device=DEV)
        some = q_rank > 0
        ops.latent_norm_cache(down, q_rank, wq if some else None, wk, 1e-6, batch.tok_seq, batch.tok_pos, batch.slots, lat if some else None,
                              site, True, err, rotated=(freq, 1.2))
        refs.latent_norm_cache(down.cpu(), q_rank, wq.cpu(), wk.cpu(), 1e-6, batch.tok_seq.cpu(), batch.tok_pos.cpu(), batch.slots.cpu(),
                               lat_ref, site_ref, True, None, rotated=(freq.cpu(), 1.2))
        assert int(err) == 0
        if some:
            close(lat, lat_ref, dtype, "query latent", bf16=1e-2)
        close(site.storage, site_ref.storage, dtype, "cache", bf16=1e-2)
        assert float(site.storage[..., kv_rank + rot:].abs().max()) == 0 if row > kv_rank + rot else True
        heads, dim = 3, 10
        x = rand(g, batch.n_tokens, heads * (dim + rot), dtype=dtype)
        out, want = torch.full((batch.n_tokens, heads * row), 9.0, dtype=dtype, device=DEV), torch.full((batch.n_tokens, heads * row), 9.0, dtype=dtype)
        ops.rotate_heads(x, dim + rot, dim, out, row, kv_rank, freq, 1.2, batch.tok_pos, heads)
        refs.rotate_heads(x.cpu(), dim + rot, dim, want, row, kv_rank, freq.cpu(), 1.2, batch.tok_pos.cpu(), heads)
        close(out, want, dtype, "queries", bf16=1e-2)
        # the maps into and out of rows that are wider than the latent
        weight = rand(g, heads, kv_rank, dim, dtype=dtype, spread=0.3)
        ops.head_linear(x, weight, out, x_pitch=dim + rot, out_pitch=row)
        refs.head_linear(x.cpu(), weight.cpu(), want, x_pitch=dim + rot, out_pitch=row)
        close(out, want, dtype, "into the latent space", bf16=1e-2)
        back = rand(g, heads, 7, kv_rank, dtype=dtype, spread=0.1)
        small, want2 = torch.empty(batch.n_tokens, heads * 7, dtype=dtype, device=DEV), torch.empty(batch.n_tokens, heads * 7, dtype=dtype)
        ops.head_linear(out, back, small, x_pitch=row)
        refs.head_linear(out.cpu(), back.cpu(), want2, x_pitch=row)
        close(small, want2, dtype, "out of the latent space", bf16=1e-2)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,kv_heads,dim,taps,planes", [(4, 2, 6, 3, 1), (4, 2, 64, 4, 1), (2, 1, 32, 1, 1), (3, 3, 16, 2, 2), (2, 2, 20, 7, 2)])
def test_convolution_whose_keys_go_to_the_cache(dtype, heads, kv_heads, dim, taps, planes):
    """Against the convolution and a plain write; long portions, short ones and single tokens; the same bits whatever the cut."""
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(dim)
    width, c = heads * dim, (heads + planes * kv_heads) * dim
    x, w = rand(g, 120, c + 8, dtype=dtype), rand(g, c, taps, spread=0.5)
    keep = max(taps - 1, 1) * c

    def step(batch, rows, state, site, on_gpu):
        move = (lambda t: t) if on_gpu else cpu
        out = move(torch.empty(len(rows), width, dtype=dtype, device=DEV))
        err = move(torch.zeros(1, dtype=torch.int32, device=DEV))
        (ops if on_gpu else refs).causal_conv_cached(move(x[rows])[:, :c], move(w), move(batch.cu_q), move(batch.tok_seq), move(batch.tok_pos),
                                                     move(batch.slots), state, 0, out, site, err, single=batch.longest == 1)
        assert int(err) == 0
        return out

    site, site_ref = paged(3, 2, kv_heads, dim, planes, dtype)
    state, state_ref = torch.zeros(3, keep, device=DEV), torch.zeros(3, keep)
    batch = Batch([1, -1], [(0, 100), (0, 20)])
    out, want = step(batch, list(range(120)), state, site, True), step(batch, list(range(120)), state_ref, site_ref, False)
    close(out, want, dtype, "queries", bf16=1e-2)
    close(site.storage, site_ref.storage, dtype, "cache", bf16=1e-2)
    assert torch.equal(state.cpu(), state_ref)
    at, pieces = 0, []
    for length in (2, 40, 1, 1, 56):
        pieces.append(step(Batch([2], [(at, length)]), list(range(at, at + length)), state, site, True))
        at += length
    assert torch.equal(torch.cat(pieces), out[:100]) and torch.equal(state[2], state[1])
    for page in range(2):
        assert torch.equal(site.storage[int(site.table[2, page])], site.storage[int(site.table[1, page])])


@pytest.mark.parametrize("dtype", BOTH)
def test_element_gate_and_scaled_clamped_gate(dtype):
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(3)
    for rows, width, extra in ((7, 30, 5), (33, 128, 64)):
        x, wide = rand(g, rows, width, dtype=dtype), rand(g, rows, width + extra, dtype=dtype, spread=3.0)
        want = x.clone().cpu()
        ops.sigmoid_gate(x, wide[:, extra:])
        refs.sigmoid_gate(want, wide[:, extra:].cpu())
        close(x, want, dtype, "gate", bf16=1e-2)
        gu, scale = rand(g, rows, 2 * width, dtype=dtype, spread=4.0), rand(g, rows).abs()
        out, want = torch.empty(rows, width, dtype=dtype, device=DEV), torch.empty(rows, width, dtype=dtype)
        ops.clamped_glu(gu, 1.5, 1.702, out, row_scale=scale)
        refs.clamped_glu(gu.cpu(), 1.5, 1.702, want, row_scale=scale.cpu())
        close(out, want, dtype, "clamped", bf16=1e-2)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,kv_heads,dim,window,cap,shared", [(4, 2, 64, 70, 5.0, True), (8, 1, 32, 0, 0.0, True), (4, 4, 128, 130, 3.0, False),
                                                                 (20, 1, 96, 65, 20.0, True), (3, 3, 48, 33, 4.0, True)])
def test_attention_with_a_distance_bias(dtype, heads, kv_heads, dim, window, cap, shared):
    """Whole prompts, portions far into a sequence and single tokens of every attention kernel that takes the head size."""
    from qwenforge_b200 import ops
    g = torch.Generator().manual_seed(dim)
    planes = 1 if shared else 2
    site, site_ref = paged(3, 12, kv_heads, dim, planes, dtype)
    site.storage.copy_(rand(g, *site.storage.shape, dtype=dtype))
    site_ref.storage.copy_(site.storage.cpu())
    bias = (torch.rand(heads, generator=g).add(0.5).to(DEV), torch.rand(heads, generator=g).add(0.1).to(DEV))
    scale = 2.0 * dim ** -0.5
    fast = dtype == torch.bfloat16 and dim in ops.FAST_ATTENTION_HEAD_DIMS
    for spans, slots in (([(0, 150), (0, 3)], [1, 0]), ([(600, 70), (64, 2)], [2, 1]), ([(700, 1), (5, 1), (129, 1), (0, 1)], [0, 1, 2, -1])):
        batch = Batch(slots, spans)
        q = rand(g, batch.n_tokens, heads * dim, dtype=dtype)
        want, err = torch.empty(batch.n_tokens, heads * dim, dtype=dtype), torch.zeros(1, dtype=torch.int32, device=DEV)
        refs.attention_generic(q.cpu(), want, batch.cu_q.cpu(), batch.tok_pos.cpu(), batch.slots.cpu(), site_ref, heads, batch.n_seqs,
                               batch.longest, scale, window, None, shared_values=shared, softcap=cap, distance_bias=cpu(bias))
        longest_kv = max(s + n for s, n in spans)
        scratch = ops.DecodeScratch(DEV)
        common = dict(shared_values=shared, softcap=cap, distance_bias=bias)
        single = batch.longest == 1
        for split in ((False, True) if single else (False,)):
            out = torch.empty_like(q)
            ops.attention_generic(q, out, batch.cu_q, batch.tok_pos, batch.slots, site, heads, batch.n_seqs, batch.longest, scale, window, err,
                                  scratch=scratch if split else None, max_kv_len=longest_kv, **common)
            close(out, want, dtype, f"generic {spans} split {split}", bf16=1e-2)
        if fast:
            out = torch.empty_like(q)
            ops.attention_prefill(q, out, batch.cu_q, batch.tok_pos, batch.slots, site, heads, batch.n_seqs, batch.longest, scale, window, err,
                                  max_kv_len=longest_kv, **common)
            close(out, want, dtype, f"prefill {spans}", bf16=2e-2)
        if fast and single:
            for splits in (1, 3):
                out = torch.empty_like(q)
                ops.attention_decode(q, out, batch.cu_q, batch.tok_pos, batch.slots, site, heads, batch.n_seqs, scale, window, splits, scratch,
                                     err, **common)
                close(out, want, dtype, f"decode {splits}", bf16=2e-2)
        assert int(err) == 0


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("tokens,width,ff,experts,top", [(9, 44, 14, 6, 2), (40, 128, 64, 8, 3), (600, 128, 64, 2, 1), (1100, 64, 32, 4, 4)])
def test_experts_whose_weight_multiplies_their_input(dtype, tokens, width, ff, experts, top):
    """The clamped gate with the router's score on the expert's input, in every form of the experts' products (the clamp bites: a
    weight on the output instead would give other numbers)."""
    from qwenforge_b200 import ops
    from qwenforge_b200.config import PartSpec
    from qwenforge_b200.csrc import prepare
    from qwenforge_b200.engine.step import build_context
    from qwenforge_b200.parts import build_part
    g = torch.Generator().manual_seed(tokens)
    names = {"router": "r.router"}
    weights = {"r.router": torch.randn(experts, width, generator=g) * 2 * width ** -0.5}
    for e in range(experts):
        for which, shape in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))):
            names[f"{which}.{e}"] = f"r.e{e}.{which}"
            weights[f"r.e{e}.{which}"] = torch.randn(*shape, generator=g) * 3 * shape[1] ** -0.5
    weights = {k: v.to(dtype) for k, v in weights.items()}
    part = build_part("feed_forward", PartSpec("routed_experts", dict(hidden_size=width, expert_size=ff, experts=experts, top=top, score="sigmoid",
                                                                      weight_on="input", gate="clamped", limit=0.9, alpha=1.702), names))
    prepare(part.kernel_libraries(dtype))
    part.bind({k: v.to(DEV) for k, v in weights.items()}, dtype, DEV)
    x = rand(g, tokens, width, dtype=dtype)
    ctx = build_context([(-1, 0, [0] * tokens)], None, torch.zeros(1, dtype=torch.int32, device=DEV), dtype, DEV)
    got = part.forward(x, ctx)
    margins = []
    mlp = dict(router=dict(experts=experts, top=top), expert=dict(limit=0.9))
    want = plain.moe_ff({k: v.float() for k, v in weights.items()}, "r.", mlp, x.double().cpu(), margins)
    sure = margins[0] > 1e-3
    close(got.cpu()[sure], want[sure], dtype, "experts", f32=2e-5, bf16=2e-2)


# ------------------------------------------------------------------ the model
def build(cfg, folder, dtype, seed=0, weights=None):
    """The model on the GPU and the weights it holds (the tests' weights are exact in both storage precisions). In bfloat16 the routers
    get weights that choose by clear margins: a flipped choice would reach every later token through keys and states."""
    from qwenforge_b200.engine import Model
    if dtype == torch.bfloat16:
        weights = steady(cfg, plain.random_weights(cfg, seed) if weights is None else weights, seed)
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
    for cuts in ([300], [260], [2, 61, 2, 130, 65, 3, 2], [129, 128]):
        logits_close(run(model, cache, tokens, cuts), want, dtype, f"{name} cuts {cuts[:3]}")
    assert all(g.pages.n_free == g.pages.n_pages for g in cache.kv_groups)


DAP_LONG = config(1000, 320, 4, 4, 1e-6, [
    layer(latent(5, 64, 32, 64, 96, 160, base=150000.0), moe(12, 3, 96)),
    layer(attention(10, 2, 64, 300), moe(20, 4, 48)),
    layer(delta(5, 5, 64, 64, ranks=(32, 32)), moe(12, 2, 96)),
    layer(latent(4, 48, 16, 48, 48, 96, base=10000.0), None),
    layer(attention(4, 4, 128, 520, conv=3), moe(12, 3, 96)),
    layer(delta(4, 2, 128, 128, ranks=(32, 16)), moe(12, 3, 96)),
])


@pytest.mark.parametrize("dtype", BOTH)
def test_long_prompts_at_larger_sizes(dtype, tmp_path):
    """Steps of more than a thousand tokens: whole, with the last tokens decoded, and cut where the later portions reach back
    over many pages."""
    cfg, n = DAP_LONG, 1400
    model, weights, _ = build(cfg, tmp_path, dtype, seed=11)
    cache = model.new_cache(64 * 40, 3)
    tokens = random_tokens(cfg["vocab"], n, 5)
    want = expect(cfg, weights, tokens)
    for cuts in ([n], [n - 40], [1100, 200, 33]):
        logits_close(run(model, cache, tokens, cuts), want, dtype, f"cuts {cuts}")
    assert all(g.pages.n_free == g.pages.n_pages for g in cache.kv_groups)


def test_the_streams_after_every_layer(tmp_path):
    model, weights, _ = build(DAP_ODD, tmp_path, torch.float32)
    cache = model.new_cache(256, 2)
    tokens = random_tokens(DAP_ODD["vocab"], 50, 1)
    seen = {}
    model.observer = lambda i, hidden, delta: seen.__setitem__(i, (hidden if delta is None else hidden + delta.float()).clone())
    run(model, cache, tokens, [50])
    model.observer = None
    streams = []
    plain.forward(DAP_ODD, weights, tokens, streams)
    assert len(streams) == 5
    for i, stream in enumerate(streams):
        assert max_err(seen[i + 1], stream) < 2e-4 * (1 + float(stream.abs().max())), f"after layer {i}"


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["odd", "fast", "wide"])
def test_unequal_batches_in_slots_used_before(dtype, name, tmp_path):
    """Requests of unequal lengths start together, are decoded together and end one by one; the second round runs in slots,
    pages and state rows that the first has used. Each request's logits equal those of the plain implementation alone."""
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
            # (in bfloat16 a request of a few tokens is too short to judge by its middle: the long ones carry it)
            for i in batch:
                cache.close(slots[i])
                if dtype == torch.float32 or len(seqs[i]) > 60:
                    logits_close(torch.cat(got[i]), want[i], dtype, f"round {round_} request {i}")
    model.raise_on_kernel_error()


def peaked(cfg, weights, factor=5.0):
    """Weights under which one score stands out: the queries of every attention grown, the distance bias small beside them, and what
    the mixers write large beside the embedding."""
    w = {k: v.clone() for k, v in weights.items()}
    w["embed"] *= 0.4
    for name in w:
        if name.endswith("hc1.out"):
            w[name] = 2.5 * w[name].abs()
    for i, entry in enumerate(cfg["layers"]):
        if entry["type"] == "attention":
            w[f"l{i}.mix.q"] *= factor
            w[f"l{i}.mix.r1"] *= 0.1
        elif entry["type"] == "latent_attention":
            w[f"l{i}.mix.uq"] *= factor
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}


@pytest.mark.parametrize("dtype", BOTH)
def test_keys_at_the_edges_of_windows_and_pages_and_keys_far_back(dtype, tmp_path):
    """Windows of 65, 64 and 1 positions over pages of 64 with sharp scores, and latent attention with sharp scores over 460
    positions: prompts that end just inside and just outside a window or a page, decoding across the edges, against the plain
    implementation. A window one position off moves a sharp row by its whole spread."""
    cfg = config(120, 48, 2, 3, 1e-6, [
        layer(attention(4, 2, 16, 65, softcap=40.0), None),
        layer(latent(4, 16, 8, 16, 24, 24, base=4000.0), None),
        layer(attention(2, 2, 32, 64, conv=2, softcap=40.0), moe(2, 1, 16)),
        layer(attention(2, 1, 16, 1), None),
        layer(latent(2, 16, 16, 16, 16, 24, base=900.0, scaling=None), None)])
    weights = peaked(cfg, plain.random_weights(cfg, 11))
    tokens = random_tokens(cfg["vocab"], 460, 5)
    model, used, _ = build(cfg, tmp_path, dtype, weights=weights)
    cache = model.new_cache(64 * 16, 2)
    want = expect(cfg, used, tokens)
    for cuts in ([460], [64], [65, 1, 1, 62, 1, 1, 100, 9], [129, 2], [63, 1, 1, 62, 2]):
        logits_close(run(model, cache, tokens, cuts), want, dtype, f"cuts {cuts}")
    # the mask and the positions matter here: every window one position longer, or no keys beyond 300 back, give other logits
    longer = {**cfg, "layers": [dict(e, mixer={**e["mixer"], "mask": {"size": e["mixer"]["mask"]["size"] + 1}}) if e["type"] == "attention" else e
                                for e in cfg["layers"]]}
    moved = lambda d: float((d - d.mean(-1, keepdim=True)).square().mean(-1).sqrt().median() / want[0].std())
    assert moved((plain.forward_logits(longer, used, tokens) - want[0])[100:]) > (0.03 if dtype == torch.float32 else 0.1)
    assert moved(plain.forward_logits(cfg, used, tokens[300:])[100:] - want[0][400:]) > 0.3


@pytest.mark.parametrize("dtype", BOTH)
def test_long_decoding_passes_windows(dtype, tmp_path):
    cfg = config(90, 32, 2, 4, 1e-6, [layer(attention(2, 1, 16, 30), moe(4, 2, 8)), layer(delta(2, 2, 8, 8, ranks=(2, 2)), moe(4, 2, 16)),
                                      layer(latent(4, 8, 4, 8, 12, 12), None)])
    model, weights, _ = build(cfg, tmp_path, dtype, seed=4)
    cache = model.new_cache(64 * 12, 2)
    tokens = random_tokens(cfg["vocab"], 420, 9)
    logits_close(run(model, cache, tokens, [3]), expect(cfg, weights, tokens), dtype)
    assert all(g.pages.n_free == g.pages.n_pages for g in cache.kv_groups)


def test_greedy_generation_through_the_engine(tmp_path):
    """StudentEngine.generate_ids (the scheduler's batches, CUDA-graph decoding with padding rows, prompt graphs) against
    greedy decoding of the plain implementation, in float32 where ties are the only way to differ."""
    from qwenforge_b200.engine import StudentEngine
    for name in ("odd", "ones", "wide"):
        cfg = CONFIGS[name]
        folder, weights = make_model_dir(cfg, 6, tmp_path / name)
        prompts = [random_tokens(cfg["vocab"], n, n) for n in (5, 70, 1, 33, 12)]
        want = [plain.greedy_generate(cfg, weights, p, 12) for p in prompts]
        for graphs in (True, False):
            engine = StudentEngine(str(folder), device=DEV, dtype="float32", cuda_graphs=graphs)
            got = engine.generate_ids(prompts, max_new_tokens=12, batch_size=3, ignore_eos=True)
            assert got == want, (name, graphs)
    folder, _ = make_model_dir(DAP_FAST, 6, tmp_path / "fast")
    prompts = [random_tokens(DAP_FAST["vocab"], n, n) for n in (5, 170, 1, 33, 12)]
    made = []
    for graphs in (True, False):
        engine = StudentEngine(str(folder), device=DEV, dtype="bfloat16", cuda_graphs=graphs)
        made.append([engine.generate_ids(prompts, max_new_tokens=12, batch_size=5, ignore_eos=True) for _ in range(2)])
    assert made[0][0] == made[0][1] and all(len(t) == 12 for t in made[0][0])   # a replay gives what the first run gave
    same = sum(a == b for x, y in zip(made[0][0], made[1][0]) for a, b in zip(x[:3], y[:3]))
    assert same >= 12    # first tokens with and without graphs (padding shapes may round a close call the other way)


def test_trace_replay_as_a_subprocess(tmp_path):
    cfg = DAP_ODD
    folder, weights = make_model_dir(cfg, 8, tmp_path / "m", store_dtype=torch.bfloat16)
    a, b = random_tokens(cfg["vocab"], 80, 1), random_tokens(cfg["vocab"], 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": [0, 69]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[70:71], "want": [0]}, {"id": "b", "tokens": b[8:], "want": [0]}], "end": ["b"]}]
    steps += [{"step": 2 + i, "entries": [{"id": "a", "tokens": [a[71 + i]], "want": [0]}], "end": ["a"] if i == 8 else []} for i in range(9)]
    root = Path(__file__).resolve().parent.parent
    out = tmp_path / "out"
    done = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                           "--max-tokens", "128", "--dump-layers", str(tmp_path / "layers")],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [l for l in done.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(11)]
    streams = []
    wa, wb = plain.forward(cfg, weights, a, streams), plain.forward_logits(cfg, weights, b)
    read = lambda path, rows: torch.from_numpy(np.fromfile(path, dtype="<f4").reshape(rows, -1))
    logits_close(read(out / "0.f32", 3), torch.stack((wa[0], wa[69], wb[7])), torch.float32)
    logits_close(read(out / "1.f32", 2), torch.stack((wa[70], wb[8])), torch.float32)
    logits_close(read(out / "10.f32", 1), wa[79:80], torch.float32)
    last = read(tmp_path / "layers" / "0.layer5.f32", 78)
    assert max_err(last[:70], streams[-1][:70]) < 2e-4 * (1 + float(streams[-1].abs().max()))
