"""A plain, slow implementation of the Dapupel decoder, one function per mechanism, in float64 on the CPU.

It shares no code with the package: the tests compare the package's kernels, cache, state and step function with it.
Every function works on ONE whole sequence from its position 0 (no cache, no state: earlier tokens are simply there).

The design, in this file's notation (t: a token at position p_t counted from 0; X: the n streams [n, width] of a token):

  streams     X[s] = E[token] for every s
  sublayer    u = sum_s a[s] X[s];  y = f(filter(dyt(u)));  X[r] <- sum_s M[s, r] X[s] + b[r] y   (all r from the old X)
              with a, b, M of the layer's own for its mixer and for its feed-forward (which a layer may lack)
  dyt(v)      tanh(alpha v) w + c
  filter(h)_t h_t + sum_j F[:, j] h_(t - taps + 1 + j)   per channel, zeros before the start
  latent      cq = rms(Dq h; nq), q = Uq cq in heads of [dim | rot];  [l | e] = Dkv h, c = rms(l; nkv), the last rot of q and
              e turned by the position;  s_ij = scale (q_i . Uk c_j + qr_i . e_j), j <= i;  softmax;  v_j = Uv c_j;  out = Wo .
  turn        neighbours (2i, 2i + 1) by the angle p f_i, f_i = base^(-2i/dims) stretched as YaRN does, cos and sin under its factor
  delta       q, k, v = silu(conv(W h)) in heads;  q, k over their lengths, q / sqrt(dim);  beta = sigmoid(Wb h);
              g = exp(-exp(A) softplus(A2 A1 h + z)) per head and key channel;
              S <- diag(g) S;  S <- S + k (beta (v - S^T k))^T;  o = S^T q;  out = Wo (rms(o; n) sigmoid(G2 G1 h))
  attention   q, k = conv(W h) in heads, v = k;  s_ij = cap tanh(scale q_i . k_j / cap) - r1 ln(1 + r2 (i - j)) for 0 <= i - j < size;
              softmax;  out = Wo (concat_heads * sigmoid(Wg h))
  experts     s = sigmoid(R h); the `top` largest;  out = sum over the chosen of expert(s_e h),
              expert(v) = Wd (g sigmoid(1.702 g) (u + 1)), g = min(Wg v, limit), u = clamp(Wu v, -limit, limit)
  logits      E dyt(sum_s X[s])
"""
from __future__ import annotations

import math

import torch

F = torch.float64
GATE_SLOPE = 1.702
LENGTH_EPS = 1e-6


# ------------------------------------------------------------------ small pieces
def dyt(v, weights, name):
    w = lambda n: weights[n].to(F)
    return torch.tanh(w(name + ".alpha") * v) * w(name) + w(name + ".b")


def rms(v, w, eps):
    out = v / torch.sqrt(v.square().mean(-1, keepdim=True) + eps)
    return out if w is None else out * w.to(F)


def causal_conv(x, taps):
    """x [T, C], taps [C, n]: sum_j taps[:, j] x_(t - n + 1 + j), zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat((torch.zeros((n - 1, x.shape[1]), dtype=F), x), dim=0)
    return sum(padded[j:j + x.shape[0]] * taps[:, j].to(F) for j in range(n))


def frequencies(rot):
    """The angle per position of every pair, and the factor on cos and sin."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    scaling = rot.get("scaling")
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            place = lambda turns: dims * math.log(float(scaling["original"]) / (2 * math.pi * turns)) / (2 * math.log(base))
            lo = max(math.floor(place(float(scaling["fast"]))), 0)
            hi = min(math.ceil(place(float(scaling["slow"]))), dims - 1)
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / float(scaling["factor"]) * ramp + f * (1.0 - ramp)
        out.append(f)
    return torch.tensor(out, dtype=F), (0.1 * math.log(float(scaling["factor"])) + 1.0 if scaling else 1.0)


def turn(x, positions, rot):
    """x [T, ..., dims], neighbours paired."""
    freq, factor = frequencies(rot)
    angle = positions.to(F)[:, None] * freq[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (freq.numel(),)
    cos, sin = (torch.cos(angle) * factor).view(shape), (torch.sin(angle) * factor).view(shape)
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack((u * cos - v * sin, v * cos + u * sin), dim=-1).reshape(x.shape)


# ------------------------------------------------------------------ mixers
def latent_attention(weights, p, m, h, eps):
    t = h.shape[0]
    heads, dim, rd, vdim, rank = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    w = lambda name: weights[p + name].to(F)
    positions = torch.arange(t)
    q = (rms(h @ w("dq").T, w("dq.norm"), eps) @ w("uq").T).view(t, heads, dim + rd)
    down = h @ w("dkv").T
    c, e = rms(down[:, :rank], w("dkv.norm"), eps), turn(down[:, rank:], positions, m["rot"])
    k = (c @ w("uk").T).view(t, heads, dim)
    v = (c @ w("uv").T).view(t, heads, vdim)
    qr = turn(q[..., dim:], positions, m["rot"])
    seen = torch.arange(t)[None, :] <= torch.arange(t)[:, None]
    out = torch.zeros((t, heads, vdim), dtype=F)
    for i in range(heads):
        s = (q[:, i, :dim] @ k[:, i].T + qr[:, i] @ e.T) * float(m["scale"])
        out[:, i] = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, i]
    return out.reshape(t, heads * vdim) @ w("o").T


def channel_delta(weights, p, m, h, eps):
    t = h.shape[0]
    heads, groups, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    w = lambda name: weights[p + name].to(F)
    mixed = {}
    for name in "qkv":
        z = causal_conv(h @ w(name).T, w(name + ".conv"))
        mixed[name] = z * torch.sigmoid(z)
    unit = lambda x: x / torch.sqrt(x.square().sum(-1, keepdim=True) + LENGTH_EPS)
    q = unit(mixed["q"].view(t, groups, dim)).repeat_interleave(heads // groups, dim=1) * dim ** -0.5
    k = unit(mixed["k"].view(t, groups, dim)).repeat_interleave(heads // groups, dim=1)
    v = mixed["v"].view(t, heads, vdim)
    beta = torch.sigmoid(h @ w("b").T)
    rate = torch.nn.functional.softplus((h @ w("a1").T) @ w("a2").T + w("dt_bias")).view(t, heads, dim)
    g = torch.exp(-torch.exp(w("A_log"))[None, :, None] * rate)
    state = torch.zeros((heads, dim, vdim), dtype=F)
    out = torch.zeros((t, heads, vdim), dtype=F)
    for i in range(t):
        state = g[i][:, :, None] * state
        u = beta[i][:, None] * (v[i] - torch.einsum("hkv,hk->hv", state, k[i]))
        state = state + k[i][:, :, None] * u[:, None, :]
        out[i] = torch.einsum("hkv,hk->hv", state, q[i])
    gate = torch.sigmoid((h @ w("g1").T) @ w("g2").T)
    return (rms(out, w("norm"), eps).reshape(t, heads * vdim) * gate) @ w("o").T


def windowed_attention(weights, p, m, h):
    t = h.shape[0]
    heads, groups, dim, size = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["mask"]["size"])
    w = lambda name: weights[p + name].to(F)
    q = causal_conv(h @ w("q").T, w("q.conv")).view(t, heads, dim)
    k = causal_conv(h @ w("k").T, w("k.conv")).view(t, groups, dim)
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    seen = (j <= i) & (i - j < size)
    far = (i - j).clamp(min=0).to(F)
    out = torch.zeros((t, heads, dim), dtype=F)
    for n in range(heads):
        key = k[:, n // (heads // groups)]
        s = (q[:, n] @ key.T) * float(m["scale"])
        if m.get("softcap"):
            s = float(m["softcap"]) * torch.tanh(s / float(m["softcap"]))
        s = s - w("r1")[n] * torch.log1p(w("r2")[n] * far)
        out[:, n] = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ key
    return (out.reshape(t, heads * dim) * torch.sigmoid(h @ w("g").T)) @ w("o").T


# ------------------------------------------------------------------ feed-forward
def expert(weights, p, h, limit):
    g = (h @ weights[p + "gate"].to(F).T).clamp(max=limit)
    u = (h @ weights[p + "up"].to(F).T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(GATE_SLOPE * g) * (u + 1.0)) @ weights[p + "down"].to(F).T


def router(weights, p, mlp, h):
    """Per token: the chosen experts, their scores, and the margin between the last choice and the best one left out."""
    top = int(mlp["router"]["top"])
    z = h @ weights[p + "router"].to(F).T
    s = torch.sigmoid(z)
    order = torch.argsort(s, dim=-1, descending=True, stable=True)
    margin = torch.full((h.shape[0],), float("inf"), dtype=F)
    if top < s.shape[1]:
        margin = z.gather(1, order[:, top - 1:top])[:, 0] - z.gather(1, order[:, top:top + 1])[:, 0]
    return order[:, :top], s.gather(1, order[:, :top]), margin


def moe_ff(weights, p, mlp, h, margins=None):
    chosen, weight, margin = router(weights, p, mlp, h)
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        for k in range(chosen.shape[1]):
            rows = torch.nonzero(chosen[:, k] == e)[:, 0]
            if rows.numel():
                out[rows] += expert(weights, f"{p}e{e}.", weight[rows, k][:, None] * h[rows], float(mlp["expert"]["limit"]))
    return out


# ------------------------------------------------------------------ the model
def sublayer(weights, p, which, X, f):
    """X [T, n, width]; f: what reads the filtered norm."""
    w = lambda name: weights[f"{p}hc{which}.{name}"].to(F)
    u = torch.einsum("s,tsw->tw", w("in"), X)
    h = dyt(u, weights, f"{p}norm{which}")
    h = h + causal_conv(h, weights[f"{p}canon{which}"])
    y = f(h)
    return torch.einsum("sr,tsw->trw", w("mix"), X) + w("out")[None, :, None] * y[:, None, :]


def layer_forward(cfg, weights, index, X, margins=None):
    layer = cfg["layers"][index]
    p, eps, m = f"l{index}.", float(cfg["norm"]["eps"]), layer["mixer"]
    mix = {"latent_attention": lambda h: latent_attention(weights, p + "mix.", m, h, eps),
           "channel_delta": lambda h: channel_delta(weights, p + "mix.", m, h, eps),
           "attention": lambda h: windowed_attention(weights, p + "mix.", m, h)}[layer["type"]]
    X = sublayer(weights, p, 1, X, mix)
    if layer.get("mlp") is not None:
        X = sublayer(weights, p, 2, X, lambda h: moe_ff(weights, p + "mlp.", layer["mlp"], h, margins))
    return X


def forward(cfg, weights, tokens, streams=None, margins=None):
    """Logits [T, vocab] of one whole sequence; `streams` collects the sum of the streams after every layer."""
    x = weights["embed"].to(F)[torch.as_tensor(tokens, dtype=torch.long)]
    X = x[:, None, :].repeat(1, int(cfg["streams"]), 1)
    for index in range(len(cfg["layers"])):
        X = layer_forward(cfg, weights, index, X, margins)
        if streams is not None:
            streams.append(X.sum(1))
    return dyt(X.sum(1), weights, "final.norm") @ weights["embed"].to(F).T


def forward_logits(cfg, weights, tokens):
    return forward(cfg, weights, tokens)


def greedy_generate(cfg, weights, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]


# ------------------------------------------------------------------ shapes and random weights
def tensor_shapes(cfg):
    width, vocab, n, taps = int(cfg["width"]), int(cfg["vocab"]), int(cfg["streams"]), int(cfg["canon"]["taps"])
    shapes = {"embed": (vocab, width)}

    def norm(name):
        shapes.update({name: (width,), name + ".b": (width,), name + ".alpha": ()})

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q, heads, dim = p + "mix.", m["heads"], m["dim"]
        for which in (1, 2) if layer.get("mlp") is not None else (1,):
            norm(f"{p}norm{which}")
            shapes.update({f"{p}hc{which}.in": (n,), f"{p}hc{which}.out": (n,), f"{p}hc{which}.mix": (n, n),
                           f"{p}canon{which}": (width, taps)})
        if layer["type"] == "attention":
            hd, gd = heads * dim, m["kv_heads"] * dim
            shapes.update({q + "q": (hd, width), q + "k": (gd, width), q + "q.conv": (hd, m["conv"]), q + "k.conv": (gd, m["conv"]),
                           q + "r1": (heads,), q + "r2": (heads,), q + "g": (hd, width), q + "o": (width, hd)})
        elif layer["type"] == "latent_attention":
            r, qr, rd = m["kv_rank"], m["q_rank"], m["rot_dim"]
            shapes.update({q + "dq": (qr, width), q + "dq.norm": (qr,), q + "uq": (heads * (dim + rd), qr), q + "dkv": (r + rd, width),
                           q + "dkv.norm": (r,), q + "uk": (heads * dim, r), q + "uv": (heads * m["vdim"], r),
                           q + "o": (width, heads * m["vdim"])})
        else:
            gd, hd, hv = m["kv_heads"] * dim, heads * dim, heads * m["vdim"]
            a, g = m["ranks"]     # (of this file's own configurations; the weights' shapes carry them)
            shapes.update({q + "q": (gd, width), q + "k": (gd, width), q + "v": (hv, width), q + "q.conv": (gd, m["conv"]),
                           q + "k.conv": (gd, m["conv"]), q + "v.conv": (hv, m["conv"]), q + "b": (heads, width), q + "A_log": (heads,),
                           q + "norm": (m["vdim"],), q + "a1": (a, width), q + "a2": (hd, a), q + "dt_bias": (hd,),
                           q + "g1": (g, width), q + "g2": (hv, g), q + "o": (width, hv)})
        mlp = layer.get("mlp")
        if mlp is not None:
            ff = mlp["expert"]["ff"]
            for e in range(mlp["router"]["experts"]):
                e = f"{p}mlp.e{e}."
                shapes.update({e + "gate": (ff, width), e + "up": (ff, width), e + "down": (width, ff)})
            shapes[p + "mlp.router"] = (mlp["router"]["experts"], width)
    return shapes


def random_weights(cfg, seed):
    """Weights that keep every mechanism alive: streams that differ, decays spread over (0, 1), clamps that bite."""
    gen = torch.Generator().manual_seed(seed)
    n = int(cfg["streams"])
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        normal = lambda std, mean=0.0: torch.randn(shape, generator=gen) * std + mean
        if ".hc" in name:
            t = normal(0.3, 1.0 / n) if last == "in" else normal(0.15, 0.4) if last == "out" else \
                normal(0.3 / n) + 0.9 * torch.eye(n)
        elif last == "alpha":
            t = normal(0.1, 0.7)
        elif ".norm" in name and last != "b":
            t = normal(0.1, 1.0)
        elif ".norm" in name:
            t = normal(0.1)
        elif last == "conv" or "canon" in name:
            t = (normal(0.5) + (1.0 if last == "conv" else 0.0)) * shape[-1] ** -0.5
        elif last in ("r1", "r2"):
            t = torch.rand(shape, generator=gen) + 0.25
        elif last == "A_log":
            t = normal(0.7, -1.0)
        elif last == "dt_bias":
            t = normal(1.0, -1.0)
        elif last in ("a2", "g2"):
            t = normal(0.5)
        elif last == "b":
            t = normal(2.0 * shape[-1] ** -0.5)
        elif last in ("gate", "up"):
            t = normal(2.0 * shape[-1] ** -0.5)
        elif last == "router":
            t = normal(2.0 * shape[-1] ** -0.5)
        elif name == "embed":
            t = normal(1.0)
        else:
            t = normal(shape[-1] ** -0.5)
        out[name] = t.to(torch.bfloat16).to(torch.float32)   # exact in both storage precisions
    return out
