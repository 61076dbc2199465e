"""Plain PyTorch references of every CUDA kernel, with the kernels' own signatures.

Each function states in tensor operations what its kernel computes; the `-m gpu` tests compare the
two on the same inputs. The functions work on any device, so the CPU tests can also put them in
the kernels' place (`conftest.reference_kernels`) to exercise the step function, the cache and the
generation loop without a GPU. They are test code: the package never imports them.
"""
from __future__ import annotations

import torch

from tests import plain_qwen2 as plain

PAGE = 64


def _f(t):
    return t.to(torch.float64)


def embed_gather(ids, table, out, err, scale=1.0):
    out.copy_(table[ids.long()].to(torch.float32) * scale)


def gather_rows(hidden, delta, rows, out, err):
    picked = hidden[rows.long()]
    if delta is not None:
        picked = picked + delta[rows.long()].to(torch.float32)
    out.copy_(picked)


def gather_rows_norm(hidden, delta, rows, weight, eps, out, err):
    picked = hidden[rows.long()]
    if delta is not None:
        picked = picked + delta[rows.long()].to(torch.float32)
    x = _f(picked)
    out.copy_((x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * _f(weight)).to(out.dtype))


def add_rms_norm(hidden, delta, weight, eps, out):
    if delta is not None:
        hidden += delta.to(torch.float32)
    x = _f(hidden)
    normed = x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * _f(weight)
    out.copy_(normed.to(out.dtype))


def gemm_f32(x, weight, bias, out):
    y = _f(x) @ _f(weight).T
    if bias is not None:
        y = y + _f(bias)
    out.copy_(y.to(out.dtype))


def linear(x, weight, bias=None, out=None, out_dtype=None):
    y = _f(x) @ _f(weight).T
    if bias is not None:
        y = y + _f(bias)
    y = y.to(out_dtype or x.dtype)
    if out is not None:
        out.copy_(y)
        return out
    return y


def _kv_rows(site, slot, positions, head, which):
    """storage rows of `positions` (list) for one head: returns (page ids, offsets)."""
    pages = site.table[slot, torch.as_tensor(positions, device=site.table.device) // PAGE].long()
    offs = torch.as_tensor(positions, device=site.table.device) % PAGE
    return pages, offs


def rope_cache_write(qkv, tok_seq, tok_pos, slots, inv_freq, rot_dim, n_heads, q_out, site, write_cache, err, bias=None,
                     unit_norm_eps=None, norm_dim=0, has_kv=True, interleaved=False, norm_first=False, q_norm=None, k_norm=None):
    n = qkv.shape[0]
    d, kvh = site.head_dim, site.kv_heads
    x = _f(qkv)[:, :(n_heads + (2 * kvh if has_kv else 0)) * d]
    if bias is not None:
        x = x + _f(bias)
    q = x[:, :n_heads * d].reshape(n, n_heads, d).clone()
    if has_kv:
        k = x[:, n_heads * d:(n_heads + kvh) * d].reshape(n, kvh, d).clone()
        v = x[:, (n_heads + kvh) * d:].reshape(n, kvh, d)
    else:
        k, v = q[:, :0].clone(), None
    if unit_norm_eps is not None and norm_first:
        over = norm_dim or d
        for t, w in ((q, q_norm), (k, k_norm)):
            t[..., :over] = t[..., :over] / torch.sqrt(t[..., :over].square().mean(-1, keepdim=True) + unit_norm_eps) \
                * (1.0 if w is None else _f(w))
    if inv_freq is not None and rot_dim > 0 and interleaved:
        angle = (tok_pos.to(torch.float32).unsqueeze(-1) * inv_freq.to(torch.float32)).to(torch.float64)
        cos, sin = angle.cos().unsqueeze(1), angle.sin().unsqueeze(1)
        for t in (q, k):
            x1, x2 = t[..., 0:rot_dim:2].clone(), t[..., 1:rot_dim:2].clone()
            t[..., 0:rot_dim:2] = x1 * cos - x2 * sin
            t[..., 1:rot_dim:2] = x2 * cos + x1 * sin
    elif inv_freq is not None and rot_dim > 0:
        angle = (tok_pos.to(torch.float32).unsqueeze(-1) * inv_freq.to(torch.float32)).to(torch.float64)
        cos, sin = angle.cos().unsqueeze(1), angle.sin().unsqueeze(1)
        half = rot_dim // 2
        for t in (q, k):
            x1, x2 = t[..., :half].clone(), t[..., half:rot_dim].clone()
            t[..., :half] = x1 * cos - x2 * sin
            t[..., half:rot_dim] = x2 * cos + x1 * sin
    if unit_norm_eps is not None and not norm_first:
        over = norm_dim or d
        for t in (q, k):
            t /= torch.sqrt(t[..., :over].square().mean(-1, keepdim=True) + unit_norm_eps)
    q_out.copy_(q.reshape(n, n_heads * d).to(q_out.dtype))
    if not write_cache:
        return
    for t in range(n):
        slot = int(slots[int(tok_seq[t])])
        if slot < 0:
            continue
        pos = int(tok_pos[t])
        page = int(site.table[slot, pos // PAGE])
        assert page >= 0, "reference: write to a page that is not held"
        site.storage[page, 0, :, pos % PAGE, :] = k[t].to(site.storage.dtype)
        site.storage[page, 1, :, pos % PAGE, :] = v[t].to(site.storage.dtype)


def gather_kv(site, slot, lo, hi):
    """Keys and values of positions lo..hi-1 of `slot`: two [kv_heads, hi-lo, head_dim] float64 tensors."""
    pos = torch.arange(lo, hi, device=site.table.device)
    pages = site.table[slot, pos // PAGE].long()
    assert bool((pages >= 0).all()), "reference: read of a page that is not held"
    k = site.storage[pages, 0, :, pos % PAGE, :]  # [n, kvh, d]
    v = site.storage[pages, 1, :, pos % PAGE, :]
    return _f(k).transpose(0, 1), _f(v).transpose(0, 1)


def gather_keys(site, slot, lo, hi):
    """Rows lo..hi-1 of a one-plane cache: [kv_heads, hi-lo, head_dim] float64."""
    pos = torch.arange(lo, hi, device=site.table.device)
    pages = site.table[slot, pos // PAGE].long()
    assert bool((pages >= 0).all()), "reference: read of a page that is not held"
    return _f(site.storage[pages, 0, :, pos % PAGE, :]).transpose(0, 1)


def attention_generic(q, out, cu_q, tok_pos, slots, site, n_heads, n_seqs, max_q_len, scale, window, err, scratch=None, max_kv_len=None,
                      sinks=None, shared_values=False, chunk=0, softcap=0.0, blocks=None, pool=0, distance_bias=None):
    d, kvh = site.head_dim, site.kv_heads
    groups = n_heads // kvh
    for s in range(n_seqs):
        b, e = int(cu_q[s]), int(cu_q[s + 1])
        slot = int(slots[s])
        if slot < 0:
            out[b:e] = 0
            continue
        for t in range(b, e):
            p = int(tok_pos[t])
            lo = max(0, p - window + 1) if window > 0 else 0
            if chunk > 0:
                lo = max(lo, p // chunk * chunk)
            if shared_values:
                k = v = gather_keys(site, slot, lo, p + 1)
            else:
                k, v = gather_kv(site, slot, lo, p + 1)
            if pool > 0 and p - window + 1 >= pool:   # the rows of the blocks that lie wholly before the window
                bk, bv = gather_kv(blocks, slot, 0, (p - window + 1) // pool)
                k, v = torch.cat((bk, k), dim=1), torch.cat((bv, v), dim=1)
            qt = _f(q[t]).view(n_heads, d)
            k = k.repeat_interleave(groups, dim=0)
            v = v.repeat_interleave(groups, dim=0)
            scores = torch.einsum("hd,hjd->hj", qt, k) * scale
            if softcap > 0:
                scores = softcap * torch.tanh(scores / softcap)
            if distance_bias is not None:
                far = torch.arange(p - lo, -1, -1, device=q.device, dtype=torch.float64)
                scores = scores - _f(distance_bias[0])[:, None] * torch.log1p(_f(distance_bias[1])[:, None] * far[None, :])
            if sinks is not None:   # one more term in the denominator, with no value
                weights = torch.softmax(torch.cat((scores, _f(sinks)[:, None]), dim=-1), -1)[:, :-1]
            else:
                weights = torch.softmax(scores, -1)
            ctx = torch.einsum("hj,hjd->hd", weights, v)
            out[t] = ctx.reshape(-1).to(out.dtype)


def swiglu(gate_up, out):
    inter = gate_up.shape[1] // 2
    g, u = _f(gate_up[:, :inter]), _f(gate_up[:, inter:])
    out.copy_((g * torch.sigmoid(g) * u).to(out.dtype))


def sample(logits, temperature, seed, seq_ids, steps, out, scratch=None):
    for r in range(logits.shape[0]):
        token, _ = plain.sample_token(logits[r].cpu(), temperature, seed,
                                      int(seq_ids[r]) if seq_ids is not None else 0,
                                      int(steps[r]) if steps is not None else 0)
        out[r] = token


def _rms(x, weight, eps):
    x = _f(x)
    return x * torch.rsqrt(x.square().mean(-1, keepdim=True) + eps) * _f(weight)


def embed_positions(ids, tok_pos, table, positions, out, err):
    out.copy_((_f(table[ids.long()]) + _f(positions[tok_pos.long()])).to(torch.float32))


def sandwich_norm(hidden, y, post_weight, post_eps, next_weight=None, next_eps=0.0, out=None, dest=None, top=1, row_weight=None):
    if dest is not None:
        y = _f(y) if row_weight is None else _f(y) * _f(row_weight)[:, None]
        y = y[dest.long()].view(-1, top, y.shape[1]).sum(1)
    hidden += _rms(y, post_weight, post_eps).to(torch.float32)
    if next_weight is not None:
        out.copy_(_rms(hidden, next_weight, next_eps).to(out.dtype))


def clamped_glu(gate_up, limit, alpha, out, row_scale=None):
    inter = gate_up.shape[1] // 2
    s = 1.0 if row_scale is None else _f(row_scale)[:, None]
    g = (s * _f(gate_up[:, :inter])).clamp(max=limit)
    u = (s * _f(gate_up[:, inter:])).clamp(min=-limit, max=limit)
    out.copy_((g * torch.sigmoid(alpha * g) * (u + 1)).to(out.dtype))


def latent_norm_cache(down, q_rank, q_norm, kv_norm, eps, tok_seq, tok_pos, slots, q_latent, site, write_cache, err, latent_out=None, rotated=None):
    if q_rank:
        q_latent.copy_(_rms(down[:, :q_rank], q_norm, eps).to(q_latent.dtype))
    r = kv_norm.numel()
    c = _rms(down[:, q_rank:q_rank + r], kv_norm, eps)
    if rotated is not None:
        turned = _turn_pairs(_f(down[:, q_rank + r:]), tok_pos, *rotated)
    if latent_out is not None:
        latent_out.copy_(c.to(latent_out.dtype))
    if not write_cache:
        return
    for t in range(down.shape[0]):
        slot = int(slots[int(tok_seq[t])])
        if slot < 0:
            continue
        pos = int(tok_pos[t])
        page = int(site.table[slot, pos // PAGE])
        assert page >= 0, "reference: write to a page that is not held"
        site.storage[page, 0, 0, pos % PAGE, :r] = c[t].to(site.storage.dtype)
        if rotated is not None:
            site.storage[page, 0, 0, pos % PAGE, r:r + turned.shape[1]] = turned[t].to(site.storage.dtype)


def _turn_pairs(x, tok_pos, inv_freq, amplitude):
    """x [T, ..., R]: neighbours turned by position * inv_freq, cosine and sine times the amplitude."""
    angle = (tok_pos.to(torch.float32).unsqueeze(-1) * inv_freq.to(torch.float32)).to(torch.float64)
    angle = angle.view((x.shape[0],) + (1,) * (x.dim() - 2) + (inv_freq.numel(),))
    cos, sin = angle.cos() * amplitude, angle.sin() * amplitude
    a, b = x[..., 0::2], x[..., 1::2]
    return torch.stack((a * cos - b * sin, b * cos + a * sin), dim=-1).reshape(x.shape)


def rotate_heads(x, x_pitch, x_first, out, out_pitch, out_first, inv_freq, amplitude, tok_pos, n_heads):
    rot, n = 2 * inv_freq.numel(), x.shape[0]
    part = _f(x).view(n, n_heads, x_pitch)[:, :, x_first:x_first + rot]
    to = out.view(n, n_heads, out_pitch)
    to[:, :, out_first:out_first + rot] = _turn_pairs(part, tok_pos, inv_freq, amplitude).to(out.dtype)
    to[:, :, out_first + rot:] = 0


def head_linear(x, weight, out, x_pitch=0, out_pitch=0):
    groups, n, k = weight.shape
    y = torch.einsum("tgk,gnk->tgn", _f(x).view(x.shape[0], groups, x_pitch or k)[:, :, :k], _f(weight))
    out.view(x.shape[0], groups, out_pitch or n)[:, :, :n] = y.to(out.dtype)


class _Routing:
    pass


def linear_rows(x, weight, out_dtype=None):
    return linear(x, weight, None, out_dtype=out_dtype)


def moe_tile_rows(n_tokens, n_experts, top, weight):
    return 64


def expert_gate_takes(x, weight, plan):
    return False


def tc_gemm_grouped(epilogue, x, weight, plan, out, row_scale=None, err=None, clamp=None):
    y = torch.einsum("rk,rnk->rn", _f(x), _f(weight)[plan.row_expert])
    if epilogue == 1:   # gate rows then up rows, a scale on both before the gate
        inter = y.shape[1] // 2
        s = _f(row_scale)[:, None] if row_scale is not None else 1.0
        g, u = y[:, :inter] * s, y[:, inter:] * s
        if clamp is not None:
            g, u = g.clamp(max=clamp[0]), u.clamp(min=-clamp[0], max=clamp[0]) + 1
            y = g * torch.sigmoid(clamp[1] * g) * u
        else:
            y = g * torch.sigmoid(g) * u
    out.copy_(y.to(out.dtype))


def scaled_swiglu(gate_up, row_scale, out):
    inter = gate_up.shape[1] // 2
    g, u = _f(gate_up[:, :inter]) * _f(row_scale)[:, None], _f(gate_up[:, inter:]) * _f(row_scale)[:, None]
    out.copy_((g * torch.sigmoid(g) * u).to(out.dtype))


def moe_plan(logits, top, softmax_scores=False, renormalize=False, tile_rows=64, x=None, router=None, bias=None, correction=None,
             groups=None, group_best=2):
    if logits is None:
        logits = (_f(x) @ _f(router).T)
    z = logits.to(torch.float32)
    if bias is not None:
        z = z + bias.to(torch.float32)
    scores = torch.softmax(z, -1) if softmax_scores else torch.sigmoid(z)
    if correction is not None or groups is not None:
        choice = scores if correction is None else scores + correction.to(torch.float32)
        count, keep = groups if groups is not None else (1, 1)
        if keep < count:
            grouped = choice.view(z.shape[0], count, -1)
            group_score = grouped.topk(min(group_best, grouped.shape[-1]), dim=-1).values.sum(-1)
            kept = torch.zeros_like(group_score, dtype=torch.bool).scatter_(1, group_score.topk(keep, dim=-1).indices, True)
            choice = grouped.masked_fill(~kept[:, :, None], float("-inf")).reshape(z.shape)
        picked = torch.topk(choice, top, dim=-1).indices
        chosen = torch.return_types.topk((scores.gather(1, picked), picked))
    else:
        chosen = torch.topk(scores, top, dim=-1)
    weights = chosen.values / chosen.values.sum(-1, keepdim=True) if renormalize else chosen.values
    plan = _Routing()
    plan.n_tokens, plan.n_experts, plan.top, plan.pairs = z.shape[0], z.shape[1], top, z.shape[0] * top
    experts = chosen.indices.reshape(-1)
    order = torch.sort(experts, stable=True).indices                    # rows: pairs sorted by expert
    plan.sorted_token = (order // top).to(torch.int32)
    plan.sorted_weight = weights.reshape(-1)[order].to(torch.float32)
    plan.row_expert = experts[order]
    plan.dest = torch.empty(plan.pairs, dtype=torch.int32)
    plan.dest[order] = torch.arange(plan.pairs, dtype=torch.int32)
    return plan


def moe_gather(x, plan, out, scale_input):
    rows = _f(x)[plan.sorted_token.long()]
    if scale_input:
        rows = rows * _f(plan.sorted_weight)[:, None]
    out.copy_(rows.to(out.dtype))


def moe_combine(y, plan, out, scale_output, extra=None, extra_gate=None, gate_input=None, gate_weight=None):
    if gate_weight is not None:
        extra_gate = _f(gate_input) @ _f(gate_weight)
    rows = _f(y)
    if scale_output:
        rows = rows * _f(plan.sorted_weight)[:, None]
    total = rows[plan.dest.long()].view(plan.n_tokens, plan.top, -1).sum(1)
    if extra is not None:
        total = total + _f(extra) * (1.0 if extra_gate is None else torch.sigmoid(_f(extra_gate)).view(-1, 1))
    out.copy_(total.to(out.dtype))


def expert_linear(x, weight, plan, out, gather=False, activation=None):
    rows = _f(x)[plan.sorted_token.long()] if gather else _f(x)
    y = torch.einsum("rk,rnk->rn", rows, _f(weight)[plan.row_expert])
    out.copy_((y if activation is None else _act(y, activation)).to(out.dtype))


def bias_act(x, bias, kind, out):
    z = _f(x) if bias is None else _f(x) + _f(bias)
    if kind == "relu2":
        y = torch.relu(z) ** 2
    elif kind == "gelu_tanh":
        y = 0.5 * z * (1 + torch.tanh(0.7978845608028654 * (z + 0.044715 * z ** 3)))
    elif kind == "silu":
        y = z * torch.sigmoid(z)
    elif kind == "gelu":
        y = 0.5 * z * (1 + torch.erf(z / 2 ** 0.5))
    elif kind == "tanh":
        y = torch.tanh(z)
    else:
        y = torch.relu(z)
    out.copy_(y.to(out.dtype))


def _act(z, kind):
    out = torch.empty_like(z)
    bias_act(z, None, kind, out)
    return out


def bias_glu(gate_up, bias, kind, out):
    inter = out.shape[1]
    z = _f(gate_up) if bias is None else _f(gate_up) + _f(bias)
    out.copy_((_act(z[:, :inter], kind) * z[:, inter:]).to(out.dtype))


def add_rms_norm_scaled(hidden, a, scale_a, b, scale_b, weight, eps, out):
    residual_add_scaled(hidden, a, scale_a, b, scale_b)
    out.copy_(_rms(hidden, weight, eps).to(out.dtype))


def residual_add_scaled(hidden, a, scale_a, b=None, scale_b=0.0):
    t = scale_a * _f(a)
    if b is not None:
        t = t + scale_b * _f(b)
    hidden.add_(t.to(torch.float32))


def rms_norm_cols(x, runs, eps):
    for col0, width, count, weight in runs:
        v = _f(x[:, col0:col0 + width])
        x[:, col0:col0 + width] = (v / torch.sqrt(v.square().sum(-1, keepdim=True) / count + eps) * _f(weight)).to(x.dtype)


def mix_rows(x, other, heads, size, x_head, other_head, weight):
    for h in range(heads):
        mine, theirs = x[:, h * x_head:h * x_head + size], other[:, h * other_head:h * other_head + size]
        mine.copy_(((1.0 - weight) * _f(mine) + weight * _f(theirs)).to(x.dtype))


def rows_prepare(x, runs, eps, mix=None):
    for index, (col0, width, count, bias, weight) in enumerate(runs):
        view = x[:, col0:col0 + width]
        if bias is not None:
            view.copy_((_f(view) + _f(bias)).to(x.dtype))
        if mix is not None and mix[0] == index:
            _, other, size, x_head, other_head, lam = mix
            mix_rows(view, other, -(-width // x_head), size, x_head, other_head, lam)
        if count > 0:
            rms_norm_cols(x, ((col0, width, count, weight),), eps)


def shift_mix(h, mu, cu_q, tok_seq, slots, state, offset, out, single=False):
    width = h.shape[1]
    for s in range(cu_q.numel() - 1):
        begin, end, slot = int(cu_q[s]), int(cu_q[s + 1]), int(slots[s])
        if end <= begin:
            continue
        first = _f(state[slot, offset:offset + width]) if slot >= 0 else torch.zeros(width, dtype=torch.float64, device=h.device)
        mine = _f(h[begin:end])
        before = torch.cat((first[None], mine[:-1]), dim=0)
        for i in range(mu.shape[0]):
            out[begin:end, i * width:(i + 1) * width] = (mine + (before - mine) * _f(mu[i])).to(out.dtype)
        if slot >= 0:
            state[slot, offset:offset + width] = mine[-1].float()


def channel_decay(pre, bias, kind, out, tau=1.0):
    z = _f(pre) if bias is None else _f(pre) + _f(bias)
    w = torch.exp(-torch.exp(z)) if kind == "double_exp" else torch.exp(torch.nn.functional.logsigmoid(z) / tau)
    out.copy_(w.float())


def outer_state_scan_rows(q, k, v, decay, cu_q, slots, state, s_offset, n_heads, dim, vdim, q_scale, y, bonus=None, decay_from=None):
    size = n_heads * dim * vdim
    if decay_from is not None:
        made = torch.empty_like(decay)
        channel_decay(decay, decay_from[1], decay_from[0], made, tau=decay_from[2])
        decay = made
    for s in range(cu_q.numel() - 1):
        slot = int(slots[s])
        S = torch.zeros(n_heads, dim, vdim, dtype=torch.float64, device=q.device)
        if slot >= 0:
            S = _f(state[slot, s_offset:s_offset + size]).view(n_heads, dim, vdim).clone()
        for t in range(int(cu_q[s]), int(cu_q[s + 1])):
            qt, kt, vt = (_f(q[t]) * q_scale).view(n_heads, dim), _f(k[t]).view(n_heads, dim), _f(v[t]).view(n_heads, vdim)
            kv = kt[:, :, None] * vt[:, None, :]
            if bonus is not None:
                y[t] = torch.einsum("hdv,hd->hv", S + _f(bonus).view(n_heads, dim)[:, :, None] * kv, qt).reshape(-1).float()
            S = _f(decay[t]).view(n_heads, dim)[:, :, None] * S + kv
            if bonus is None:
                y[t] = torch.einsum("hdv,hd->hv", S, qt).reshape(-1).float()
        if slot >= 0:
            state[slot, s_offset:s_offset + size] = S.reshape(-1).float()


def softcap_(x, cap):
    x.copy_((cap * torch.tanh(_f(x) / cap)).to(x.dtype))


def stabilized_gates(pre, bias, cap, cu_q, slots, state, m_offset, n_heads, decay, take, floor):
    z = _f(pre) + _f(bias)
    a = cap * torch.tanh(z[:, :n_heads] / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh(z[:, n_heads:] / cap))
    for s in range(cu_q.numel() - 1):
        slot = int(slots[s])
        m = _f(state[slot, m_offset:m_offset + n_heads]) if slot >= 0 else torch.zeros(n_heads, dtype=torch.float64, device=pre.device)
        for t in range(int(cu_q[s]), int(cu_q[s + 1])):
            m_new = torch.maximum(f[t] + m, a[t])
            decay[t] = torch.exp(f[t] + m - m_new).float()
            take[t] = torch.exp(a[t] - m_new).float()
            floor[t] = torch.exp(-m_new).float()
            m = m_new
        if slot >= 0:
            state[slot, m_offset:m_offset + n_heads] = m.float()


def decay_gates(dt_pre, dt_bias, rate_log, decay, take):
    dt = torch.nn.functional.softplus(_f(dt_pre) + _f(dt_bias))
    decay.copy_(torch.exp(-torch.exp(_f(rate_log)) * dt).float())
    take.copy_(dt.float())


def outer_state_scan(q, k, v, decay, take, cu_q, slots, state, s_offset, n_offset, n_heads, n_groups, dim, vdim, q_scale, y, nq):
    per = n_heads // n_groups
    for s in range(cu_q.numel() - 1):
        slot = int(slots[s])
        S = torch.zeros(n_heads, dim, vdim, dtype=torch.float64, device=q.device)
        nv = torch.zeros(n_heads, dim, dtype=torch.float64, device=q.device)
        if slot >= 0:
            S = _f(state[slot, s_offset:s_offset + n_heads * dim * vdim]).view(n_heads, dim, vdim).clone()
            if nq is not None:
                nv = _f(state[slot, n_offset:n_offset + n_heads * dim]).view(n_heads, dim).clone()
        for t in range(int(cu_q[s]), int(cu_q[s + 1])):
            qt = (_f(q[t]) * q_scale).view(n_groups, dim).repeat_interleave(per, dim=0)
            kt = _f(k[t]).view(n_groups, dim).repeat_interleave(per, dim=0)
            vt = _f(v[t]).view(n_heads, vdim)
            d, g = (_f(decay[t])[:, None], _f(take[t])[:, None]) if take is not None else (_f(decay)[:, None], torch.ones_like(_f(decay))[:, None])
            S = d[:, :, None] * S + g[:, :, None] * kt[:, :, None] * vt[:, None, :]
            y[t] = torch.einsum("hdv,hd->hv", S, qt).reshape(-1).float()
            if nq is not None:
                nv = d * nv + g * kt
                nq[t] = (nv * qt).sum(-1).float()
        if slot >= 0:
            state[slot, s_offset:s_offset + n_heads * dim * vdim] = S.reshape(-1).float()
            if nq is not None:
                state[slot, n_offset:n_offset + n_heads * dim] = nv.reshape(-1).float()


def gated_group_norm(y, gate, weight, eps, out, n_parts, n_heads, gate_kind, gate_first, nq=None, floor=None, floor_add=0.0,
                     skip=None, skip_x=None):
    n, c = y.shape
    z = _f(y).view(n, n_heads, c // n_heads)
    if nq is not None:
        z = z / (torch.maximum(_f(nq).abs(), _f(floor)) + floor_add)[:, :, None]
    if skip is not None:
        z = z + _f(skip)[None, :, None] * _f(skip_x).view(n, n_heads, -1)
    z = z.reshape(n, c)
    g = _f(gate)
    g = torch.sigmoid(g) if gate_kind == "sigmoid" else g * torch.sigmoid(g)
    if gate_first:
        z = z * g
    z = z.view(n, n_parts, c // n_parts)
    z = (z / torch.sqrt(z.square().mean(-1, keepdim=True) + eps)).reshape(n, c) * _f(weight)
    if not gate_first:
        z = z * g
    out.copy_(z.to(out.dtype))


def causal_conv_silu(x, weight, bias, cu_q, tok_seq, slots, state, offset, out, activation="silu", single=False):
    n, c = x.shape
    taps = weight.shape[1]
    for s in range(cu_q.numel() - 1):
        b, e = int(cu_q[s]), int(cu_q[s + 1])
        slot = int(slots[s])
        before = torch.zeros(taps - 1, c, dtype=torch.float64, device=x.device)
        if slot >= 0:
            before = _f(state[slot, offset:offset + (taps - 1) * c]).view(taps - 1, c)
        padded = torch.cat((before, _f(x[b:e])))
        z = sum(padded[j:j + e - b] * _f(weight)[:, j] for j in range(taps))
        if bias is not None:
            z = z + _f(bias)
        out[b:e] = (z * torch.sigmoid(z) if activation == "silu" else z).to(out.dtype)
        if slot >= 0 and taps > 1:
            state[slot, offset:offset + (taps - 1) * c] = padded[padded.shape[0] - (taps - 1):].reshape(-1).float()


def causal_conv(x, weight, bias, cu_q, tok_seq, slots, state, offset, out, single=False):
    causal_conv_silu(x, weight, bias, cu_q, tok_seq, slots, state, offset, out, activation="none")


def causal_conv_cached(x, weight, cu_q, tok_seq, tok_pos, slots, state, offset, out, site, err, single=False):
    whole = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    causal_conv(x, weight, None, cu_q, tok_seq, slots, state, offset, whole)
    width = out.shape[1]
    out.copy_(whole[:, :width])
    planes = site.storage.shape[1]
    rows = whole[:, width:].reshape(x.shape[0], planes, site.kv_heads, site.head_dim)
    for t in range(x.shape[0]):
        slot = int(slots[int(tok_seq[t])])
        if slot < 0:
            continue
        pos = int(tok_pos[t])
        page = int(site.table[slot, pos // PAGE])
        assert page >= 0, "reference: write to a page that is not held"
        site.storage[page, :, :, pos % PAGE, :] = rows[t]


def sigmoid_gate(x, gate):
    x.copy_((_f(x) * torch.sigmoid(_f(gate))).to(x.dtype))


def delta_scan(q, k, v, z, bias, rate_log, logit, cu_q, slots, state, s_offset, n_heads, n_groups, dim, vdim, q_scale, y, max_q_len=0, err=None):
    per, size = n_heads // n_groups, n_heads * dim * vdim
    unit = lambda x: x / torch.sqrt(x.square().sum(-1, keepdim=True) + 1e-6)
    spread = lambda x: unit(_f(x).view(x.shape[0], n_groups, dim)).repeat_interleave(per, dim=1)
    qs, ks, vs = spread(q) * q_scale, spread(k), _f(v).view(v.shape[0], n_heads, vdim)
    rate = torch.nn.functional.softplus(_f(z) + _f(bias)).view(-1, n_heads, dim)
    g = torch.exp(-torch.exp(_f(rate_log))[None, :, None] * rate)
    beta = torch.sigmoid(_f(logit))
    for s in range(cu_q.numel() - 1):
        slot = int(slots[s])
        S = torch.zeros(n_heads, dim, vdim, dtype=torch.float64, device=q.device)
        if slot >= 0:
            S = _f(state[slot, s_offset:s_offset + size]).view(n_heads, dim, vdim).clone()
        for t in range(int(cu_q[s]), int(cu_q[s + 1])):
            S = g[t][:, :, None] * S
            u = beta[t][:, None] * (vs[t] - torch.einsum("hdv,hd->hv", S, ks[t]))
            S = S + ks[t][:, :, None] * u[:, None, :]
            y[t] = torch.einsum("hdv,hd->hv", S, qs[t]).reshape(-1).float()
        if slot >= 0:
            state[slot, s_offset:s_offset + size] = S.reshape(-1).float()


def delta_token(q, k, v, z, bias, rate_log, logit, cu_q, slots, state, s_offset, n_heads, n_groups, dim, vdim, q_scale, y=None,
                norm=None, eps=0.0, gate=None, out=None):
    made = torch.empty(q.shape[0], n_heads * vdim, dtype=torch.float32, device=q.device)
    delta_scan(q, k, v, z, bias, rate_log, logit, cu_q, slots, state, s_offset, n_heads, n_groups, dim, vdim, q_scale, made)
    if y is not None:
        y.copy_(made)
    if out is not None:
        r = _f(made).view(-1, n_heads, vdim)
        r = r / torch.sqrt(r.square().mean(-1, keepdim=True) + eps) * _f(norm)
        out.copy_((r.reshape(made.shape) * torch.sigmoid(_f(gate))).to(out.dtype))


def streams_norm(source, n_streams, coefficients, y, in_weight, new=None, norm=None, out=None, conv=None, rows=None, err=None,
                 y_rows=None):
    X = _f(source)
    if X.dim() == 2:
        X = X[:, None, :].expand(-1, n_streams, -1)
    Y = X
    if y is not None:
        mix, out_w = coefficients
        y = _f(y)
        if y_rows is not None:
            dest, top, row_weight = y_rows
            if row_weight is not None:
                y = y * _f(row_weight)[:, None]
            y = y[dest.long()].view(-1, top, y.shape[1]).sum(1)
        Y = torch.einsum("sr,tsw->trw", _f(mix), X) + _f(out_w)[None, :, None] * y[:, None, :]
    if new is not None:
        new.copy_(Y.to(torch.float32))
    u = Y.sum(1) if in_weight is None else torch.einsum("s,tsw->tw", _f(in_weight), Y)
    if rows is not None:
        u = u[rows.long()]
    if norm is None:
        out.copy_(u.to(out.dtype))
        return
    h = torch.tanh(norm[2] * u) * _f(norm[0]) + _f(norm[1])
    if conv is not None:
        taps, cu_q, slots, _, state, offset = conv
        n, c = taps.shape[1], taps.shape[0]
        filtered = torch.empty_like(h)
        for s in range(cu_q.numel() - 1):
            b, e, slot = int(cu_q[s]), int(cu_q[s + 1]), int(slots[s])
            before = torch.zeros(n - 1, c, dtype=torch.float64, device=h.device)
            if slot >= 0:
                before = _f(state[slot, offset:offset + (n - 1) * c]).view(n - 1, c)
            padded = torch.cat((before, h[b:e]))
            filtered[b:e] = h[b:e] + sum(padded[j:j + e - b] * _f(taps)[:, j] for j in range(n))
            if slot >= 0 and n > 1 and e > b:
                state[slot, offset:offset + (n - 1) * c] = padded[padded.shape[0] - (n - 1):].reshape(-1).float()
        h = filtered
    out.copy_(h.to(out.dtype))


def add_dyt_norm(hidden, a, b, weight, bias, alpha, out):
    if a is not None or b is not None:
        hidden += ((0 if a is None else _f(a)) + (0 if b is None else _f(b))).to(hidden.dtype)
    out.copy_((torch.tanh(alpha * _f(hidden)) * _f(weight) + _f(bias)).to(out.dtype))


def add_dyt_norm_shift(hidden, a, b, weight, bias, alpha, out, taps, slots, state, shifted):
    add_dyt_norm(hidden, a, b, weight, bias, alpha, out)
    rows = out.shape[0]
    every = torch.arange(rows + 1, dtype=torch.int32, device=out.device)
    causal_conv(out, taps, None, every, every[:-1], slots, state, 0, shifted, single=True)


def gated_rows(x, weight, out, clamp=None):
    return False     # the product and the gate as two steps


def residual_add_pair(hidden, a, b):
    if a is not None or b is not None:
        hidden += ((0 if a is None else _f(a)) + (0 if b is None else _f(b))).to(hidden.dtype)


def stream_pair(hidden, a, b, other, out):
    x = _f(hidden) + (0 if a is None else _f(a)) + (0 if b is None else _f(b))
    out.copy_(torch.cat((x, _f(other)), dim=-1).to(out.dtype))


def head_gate(x, gate, n_heads):
    rows = x.shape[0]
    x.copy_((_f(x).view(rows, n_heads, -1) * torch.sigmoid(_f(gate))[:, :, None]).view(rows, -1).to(x.dtype))


def pool_cache_write(cu_q, tok_pos, slots, site, blocks, pool, max_q_len, err):
    for s in range(slots.numel()):
        slot, b, e = int(slots[s]), int(cu_q[s]), int(cu_q[s + 1])
        if slot < 0 or e <= b:
            continue
        start = int(tok_pos[b])
        for block in range(start // pool, (start + e - b) // pool):
            k, v = gather_kv(site, slot, block * pool, block * pool + pool)      # [kvh, pool, d]
            page = int(blocks.table[slot, block // PAGE])
            assert page >= 0, "reference: write to a page of block rows that is not held"
            blocks.storage[page, 0, :, block % PAGE, :] = k.mean(1).to(blocks.storage.dtype)
            blocks.storage[page, 1, :, block % PAGE, :] = v.mean(1).to(blocks.storage.dtype)


ALL = dict(causal_conv_cached=causal_conv_cached, sigmoid_gate=sigmoid_gate, delta_scan=delta_scan, delta_token=delta_token, streams_norm=streams_norm,
           rotate_heads=rotate_heads, rows_prepare=rows_prepare, bias_glu=bias_glu, add_rms_norm_scaled=add_rms_norm_scaled, residual_add_scaled=residual_add_scaled, rms_norm_cols=rms_norm_cols,
           mix_rows=mix_rows, shift_mix=shift_mix, channel_decay=channel_decay, outer_state_scan_rows=outer_state_scan_rows,
           gated_rows=gated_rows, causal_conv=causal_conv, add_dyt_norm=add_dyt_norm, add_dyt_norm_shift=add_dyt_norm_shift, residual_add_pair=residual_add_pair, stream_pair=stream_pair,
           head_gate=head_gate, pool_cache_write=pool_cache_write, bias_act=bias_act, softcap_=softcap_, stabilized_gates=stabilized_gates, decay_gates=decay_gates,
           outer_state_scan=outer_state_scan, gated_group_norm=gated_group_norm, causal_conv_silu=causal_conv_silu,
           expert_gate_takes=expert_gate_takes, linear_rows=linear_rows, moe_tile_rows=moe_tile_rows, scaled_swiglu=scaled_swiglu, embed_positions=embed_positions, sandwich_norm=sandwich_norm, clamped_glu=clamped_glu, latent_norm_cache=latent_norm_cache,
           head_linear=head_linear, moe_plan=moe_plan, moe_gather=moe_gather, moe_combine=moe_combine, expert_linear=expert_linear,
           embed_gather=embed_gather, gather_rows=gather_rows, gather_rows_norm=gather_rows_norm, add_rms_norm=add_rms_norm, gemm_f32=gemm_f32,
           linear=linear, rope_cache_write=rope_cache_write, attention_generic=attention_generic, swiglu=swiglu,
           sample=sample)


# ---------------------------------------------------------------- heads of two maps, two norms of one stream, retention
def _turn_halves(x, cos, sin):
    """x [T, ..., D]; cos, sin [T, R/2]: component j of the first R turned with j + R/2."""
    half = cos.shape[1]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    c, s = cos.view(shape), sin.view(shape)
    a, b = x[..., :half], x[..., half:2 * half]
    return torch.cat((a * c - b * s, b * c + a * s, x[..., 2 * half:]), dim=-1)


def rope_table(tok_pos, inv_freq, amplitude=1.0):
    angle = (tok_pos.to(torch.float32).unsqueeze(-1) * inv_freq.to(torch.float32)).to(torch.float64)
    return (torch.stack((angle.cos(), angle.sin()), dim=-1) * amplitude).to(torch.float32)


def _angles_of(tok_pos, inv_freq, amplitude):
    angle = (tok_pos.to(torch.float32).unsqueeze(-1) * inv_freq.to(torch.float32)).to(torch.float64)
    return angle.cos() * amplitude, angle.sin() * amplitude


def rope_maps_cache_write(qkv, tok_seq, tok_pos, slots, inv_freq, rot_dim, amplitude, n_heads, maps, dim, vdim, q_out, site, write_cache, err):
    n, d, kvh = qkv.shape[0], site.head_dim, site.kv_heads
    x = _f(qkv)
    a, b = n_heads * maps * dim, kvh * maps * dim
    q, k, v = x[:, :a].reshape(n, n_heads, maps, dim), x[:, a:a + b].reshape(n, kvh, maps, dim), x[:, a + b:a + b + kvh * vdim].reshape(n, kvh, vdim)
    if inv_freq is not None and rot_dim > 0:
        cos, sin = _angles_of(tok_pos, inv_freq, amplitude)
        q, k = _turn_halves(q, cos, sin), _turn_halves(k, cos, sin)
    wide = torch.zeros((n, n_heads, maps, d), dtype=torch.float64, device=qkv.device)
    for m in range(maps):
        wide[:, :, m, m * dim:(m + 1) * dim] = q[:, :, m]
    q_out.copy_(wide.reshape(n, -1).to(q_out.dtype))
    if not write_cache:
        return
    for t in range(n):
        slot = int(slots[int(tok_seq[t])])
        if slot < 0:
            continue
        pos = int(tok_pos[t])
        page = int(site.table[slot, pos // PAGE])
        assert page >= 0, "reference: write to a page that is not held"
        rows = site.storage[page, :, :, pos % PAGE, :]
        rows.zero_()
        rows[0, :, :maps * dim] = k[t].reshape(kvh, maps * dim).to(rows.dtype)
        rows[1, :, :vdim] = v[t].to(rows.dtype)


def map_difference(x, pitch, weight, eps, gain, out, heads, vdim):
    a = _f(x).view(x.shape[0], heads, 2, pitch)[..., :vdim]
    o = a[:, :, 0] - weight * a[:, :, 1]
    out.copy_((gain * o / torch.sqrt(o.square().mean(-1, keepdim=True) + eps)).reshape(out.shape).to(out.dtype))


def pair_rms_norm(hidden, a, b, weight1=None, eps1=0.0, out1=None, weight2=None, eps2=0.0, out2=None, b_rows=None, rows=None, err=None):
    total = torch.zeros(hidden.shape, dtype=torch.float64, device=hidden.device)
    if b is not None:
        y = _f(b)
        if b_rows is not None:
            dest, top, row_weight = b_rows
            if row_weight is not None:
                y = y * _f(row_weight)[:, None]
            y = y[dest.long()].view(-1, top, y.shape[1]).sum(1)
        total += y
    if a is not None:
        total += _f(a)
    x = _f(hidden) + total
    if rows is None:
        hidden.copy_(x.to(torch.float32))
        x = _f(hidden)
    else:
        x = x[rows.long()]
    for weight, eps, out in ((weight1, eps1, out1), (weight2, eps2, out2)):
        if weight is not None:
            out.copy_(_rms(x, weight, eps).to(out.dtype))


def retention_chunks_take(q, k, v, gate, state, s_offset, dim, vdim, rot_dim):
    return q.dtype == torch.bfloat16


def _retention(q, k, v, gate, cos, sin, decay, k_scale, eps, cu_q, slots, state, s_offset, n_heads, dim, vdim, out):
    n, size = q.shape[0], n_heads * dim * vdim
    qh, kh, vh = _f(q).reshape(n, n_heads, dim), _f(k).reshape(n, n_heads, dim), _f(v).reshape(n, n_heads, vdim)
    if cos is not None:
        qh, kh = _turn_halves(qh, cos, sin), _turn_halves(kh, cos, sin)
    kh = kh * k_scale
    for s in range(cu_q.numel() - 1):
        slot = int(slots[s])
        S = torch.zeros(n_heads, dim, vdim, dtype=torch.float64, device=q.device)
        if slot >= 0:
            S = _f(state[slot, s_offset:s_offset + size]).view(n_heads, dim, vdim).clone()
        for t in range(int(cu_q[s]), int(cu_q[s + 1])):
            S = _f(decay)[:, None, None] * S + kh[t][:, :, None] * vh[t][:, None, :]
            o = torch.einsum("hdv,hd->hv", S, qh[t])
            o = o / torch.sqrt(o.square().mean(-1, keepdim=True) + eps)
            g = _f(gate[t])
            out[t] = (o.reshape(-1) * g * torch.sigmoid(g)).to(out.dtype)
        if slot >= 0:
            state[slot, s_offset:s_offset + size] = S.reshape(-1).float()


def retention_chunks(q, k, v, gate, angles, rot_dim, powers, k_scale, eps, cu_q, slots, max_q_len, state, s_offset, n_heads, dim, vdim, out):
    cos, sin = (_f(angles[..., 0]), _f(angles[..., 1])) if rot_dim else (None, None)
    _retention(q, k, v, gate, cos, sin, powers[:, 1], k_scale, eps, cu_q, slots, state, s_offset, n_heads, dim, vdim, out)


def retention_token(q, k, v, gate, tok_pos, inv_freq, rot_dim, amplitude, decay, k_scale, eps, cu_q, slots, state, s_offset, n_heads, dim, vdim, out):
    cos, sin = _angles_of(tok_pos, inv_freq, amplitude) if rot_dim else (None, None)
    _retention(q, k, v, gate, cos, sin, decay, k_scale, eps, cu_q, slots, state, s_offset, n_heads, dim, vdim, out)


def retention_rows(q, k, v, angles, rot_dim, k_scale, n_heads, dim, vdim, rows):
    n = q.shape[0]
    qh, kh = _f(q).reshape(n, n_heads, dim), _f(k).reshape(n, n_heads, dim)
    if rot_dim:
        cos, sin = _f(angles[..., 0]), _f(angles[..., 1])
        qh, kh = _turn_halves(qh, cos, sin), _turn_halves(kh, cos, sin)
    rows.copy_(torch.cat((qh.reshape(n, -1), kh.reshape(n, -1) * k_scale, _f(v)), dim=-1).to(torch.float32))


ALL.update(rope_table=rope_table, rope_maps_cache_write=rope_maps_cache_write, map_difference=map_difference, pair_rms_norm=pair_rms_norm,
           retention_chunks_take=retention_chunks_take, retention_chunks=retention_chunks, retention_token=retention_token,
           retention_rows=retention_rows)
