"""A plain, slow implementation of the Lasonex decoder, one function per mechanism, in float64 on the CPU.

It shares no code with the package: the tests compare the package's kernels, cache, state and step function with it.
Every function works on ONE whole sequence from its position 0 (no cache, no state: earlier tokens are simply there).

The design, in this file's notation (t: a token at position p_t counted from 0; x: the stream; c: embedding.scale):

  stream      x_t = c * E[token_t]
  layer       x <- x + (mixer(rms(x; n1)) + ff(rms(x; n2)))   both sublayers read the same x (a layer may have no feed-forward)
  rms(v; w)   v / sqrt(mean(v^2) + eps) * w
  turn        the first `rot.dims` components of a head turn by p_t, component i with i + dims/2, angle p * f_i, f_i = base^(-2i/dims);
              with rot.scaling the frequencies are stretched (YaRN) and cosine and sine multiplied by 0.1 ln(factor) + 1
  attention   differential: every query head has two queries and every key/value head two keys (maps 1 and 2, one after the
              other in the head's rows) and one value; each map is turned by itself and is a windowed softmax attention of its
              own over the head's values, s_ij = scale q_i . k_j for 0 <= i - j < size; with a1, a2 the two results
              o = a1 - lam a2, lam = exp(lq1 . lk1) - exp(lq2 . lk2) + diff (one number per layer);
              o <- (1 - diff) o / sqrt(mean(o^2) + eps) per head; out = Wo concat_heads
  retention   q, k turned per head, k * dim^-1/2;  S <- decay_h S + k_t v_t^T,  o_t = S^T q_t (the state AFTER this token);
              o <- o / sqrt(mean(o^2) + eps) per head;  out = Wo (concat_heads * silu(Wg h))
  dense ff    g = min(Wg h, limit), u = clamp(Wu h, -limit, limit);  Wd (g sigmoid(1.702 g) (u + 1))
  moe         z = R h;  s = softmax(z) over all experts;  experts in `count` equal groups of neighbours, a group's score its
              largest s;  only experts of the `keep` best groups may be chosen;  the `top` largest s among them;
              out = sum over the chosen of s_e / (sum of the chosen s + 1e-20) * expert_e(h), every expert of the dense form
  logits      H rms(x; nf)
"""
from __future__ import annotations

import math

import torch

F = torch.float64
SLOPE = 1.702


# ------------------------------------------------------------------ small pieces
def rms(v, w, eps):
    out = v / torch.sqrt(v.square().mean(-1, keepdim=True) + eps)
    return out if w is None else out * w.to(F)


def silu(z):
    return z * torch.sigmoid(z)


def frequencies(rot):
    """The turning frequencies of the dims/2 pairs, and the factor on cosine and sine."""
    dims, base = int(rot["dims"]), float(rot["base"])
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if not scaling:
        return freq, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def place(turns):   # the (fractional) pair that turns `turns` times within the original length
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(place(float(scaling["fast"]))), 0), min(math.ceil(place(float(scaling["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def turn(x, positions, rot):
    """x [T, ..., dim]: the first rot.dims components of the last axis turned by the token's position."""
    dims = int(rot["dims"])
    if dims == 0:
        return x
    freq, amplitude = frequencies(rot)
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (dims // 2,)
    angle = (positions.to(F)[:, None] * torch.tensor(freq, dtype=F)[None, :]).view(shape)
    cos, sin = torch.cos(angle) * amplitude, torch.sin(angle) * amplitude
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat((u * cos - v * sin, v * cos + u * sin, x[..., dims:]), dim=-1)


def window_softmax(q, k, v, scale, size):
    """One head and map: q, k [T, D], v [T, V]; position i sees j with 0 <= i - j < size."""
    t = q.shape[0]
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    s = (q @ k.T) * scale
    s = s.masked_fill((j > i) | (i - j >= size), float("-inf"))
    return torch.softmax(s, dim=-1) @ v


def difference_weight(weights, p, m):
    w = lambda name: weights[p + name].to(F)
    return math.exp(float((w("lq1") * w("lk1")).sum())) - math.exp(float((w("lq2") * w("lk2")).sum())) + float(m["diff"])


def combine_maps(a1, a2, lam, diff, eps):
    """a1, a2 [..., vdim]: the two maps' results of one head."""
    return rms(a1 - lam * a2, None, eps) * (1.0 - diff)


# ------------------------------------------------------------------ mixers
def differential_attention(weights, p, m, h, eps):
    t = h.shape[0]
    heads, groups, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    w = lambda name: weights[p + name].to(F)
    positions = torch.arange(t)
    q = turn((h @ w("q").T).view(t, heads, 2, dim), positions, m["rot"])
    k = turn((h @ w("k").T).view(t, groups, 2, dim), positions, m["rot"])
    v = (h @ w("v").T).view(t, groups, vdim)
    lam, diff, size = difference_weight(weights, p, m), float(m["diff"]), int(m["mask"]["size"])
    out = []
    for head in range(heads):
        g = head // (heads // groups)
        a1, a2 = (window_softmax(q[:, head, n], k[:, g, n], v[:, g], float(m["scale"]), size) for n in (0, 1))
        out.append(combine_maps(a1, a2, lam, diff, eps))
    return torch.cat(out, dim=-1) @ w("o").T


def retain(q, k, v, decay):
    """The recurrence of one head: q, k [T, D] (k already scaled), v [T, V]; S^T q with S after every token."""
    state = torch.zeros((q.shape[1], v.shape[1]), dtype=F)
    out = []
    for i in range(q.shape[0]):
        state = decay * state + k[i][:, None] * v[i][None, :]
        out.append(state.T @ q[i])
    return torch.stack(out)


def retention(weights, p, m, h, eps):
    t = h.shape[0]
    heads, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    w = lambda name: weights[p + name].to(F)
    positions = torch.arange(t)
    q = turn((h @ w("q").T).view(t, heads, dim), positions, m["rot"])
    k = turn((h @ w("k").T).view(t, heads, dim), positions, m["rot"]) * dim ** -0.5
    v = (h @ w("v").T).view(t, heads, vdim)
    o = torch.cat([rms(retain(q[:, n], k[:, n], v[:, n], float(m["decay"][n])), None, eps) for n in range(heads)], dim=-1)
    return (o * silu(h @ w("g").T)) @ w("o").T


# ------------------------------------------------------------------ feed-forwards
def clamped_ff(weights, p, h, limit):
    w = lambda name: weights[p + name].to(F)
    g, u = (h @ w("gate").T).clamp(max=limit), (h @ w("up").T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(SLOPE * g) * (u + 1.0)) @ w("down").T


def router(weights, p, mlp, h):
    """Per token: the chosen experts (in falling order of their scores), their weights, and the margin (in logits) between the
    last choice and the best one left out (among those that may be chosen, and between the groups)."""
    r = mlp["router"]
    experts, top = int(r["experts"]), int(r["top"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    count, keep = int(groups["count"]), int(groups["keep"])
    size = experts // count
    z = h @ weights[p + "router"].to(F).T
    s = torch.softmax(z, dim=-1)
    chosen, weight, margin = [], [], []
    for t in range(h.shape[0]):
        score = s[t].view(count, size).max(-1).values
        order = torch.argsort(score, descending=True, stable=True)
        kept = order[:keep]
        gap = float(torch.log(score[order[keep - 1]]) - torch.log(score[order[keep]])) if keep < count else float("inf")
        allowed = torch.full((experts,), float("-inf"), dtype=F)
        for g in kept.tolist():
            allowed[g * size:(g + 1) * size] = s[t, g * size:(g + 1) * size]
        ranked = torch.argsort(allowed, descending=True, stable=True)
        pick = ranked[:top]
        if top < keep * size:
            gap = min(gap, float(z[t, ranked[top - 1]] - z[t, ranked[top]]))
        chosen.append(pick)
        weight.append(s[t, pick] / (s[t, pick].sum() + 1e-20))
        margin.append(gap)
    return torch.stack(chosen), torch.stack(weight), torch.tensor(margin, dtype=F)


def moe_ff(weights, p, mlp, h, margins=None):
    chosen, weight, margin = router(weights, p, mlp, h)
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weight[t]):
            out[t] += w * clamped_ff(weights, f"{p}e{e}.", h[t:t + 1], float(mlp["expert"]["limit"]))[0]
    return out


# ------------------------------------------------------------------ the model
def layer_forward(cfg, weights, index, x, margins=None):
    layer = cfg["layers"][index]
    p, eps, m = f"l{index}.", float(cfg["norm"]["eps"]), layer["mixer"]
    h = rms(x, weights[p + "norm1"], eps)
    if layer["type"] == "attention":
        y = differential_attention(weights, p + "mix.", m, h, eps)
    elif layer["type"] == "retention":
        y = retention(weights, p + "mix.", m, h, eps)
    else:
        raise ValueError(layer["type"])
    mlp = layer.get("mlp")
    if mlp is not None:
        h = rms(x, weights[p + "norm2"], eps)
        y = y + (clamped_ff(weights, p + "mlp.", h, float(mlp["limit"])) if mlp["kind"] == "dense"
                 else moe_ff(weights, p + "mlp.", mlp, h, margins))
    return x + y


def forward(cfg, weights, tokens, streams=None, margins=None):
    """Logits [T, vocab] of one whole sequence; `streams` collects the stream after every layer."""
    x = weights["embed"].to(F)[torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    for index in range(len(cfg["layers"])):
        x = layer_forward(cfg, weights, index, x, margins)
        if streams is not None:
            streams.append(x.clone())
    return rms(x, weights["final.norm"], float(cfg["norm"]["eps"])) @ weights["head"].to(F).T


def forward_logits(cfg, weights, tokens):
    return forward(cfg, weights, tokens)


def greedy_generate(cfg, weights, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]


# ------------------------------------------------------------------ shapes and random weights
def tensor_shapes(cfg):
    width, vocab = int(cfg["width"]), int(cfg["vocab"])
    shapes = {"embed": (vocab, width), "final.norm": (width,), "head": (vocab, width)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q, heads, dim, vdim = p + "mix.", m["heads"], m["dim"], m["vdim"]
        shapes[p + "norm1"] = (width,)
        if layer["type"] == "attention":
            g = m["kv_heads"]
            shapes.update({q + "q": (heads * 2 * dim, width), q + "k": (g * 2 * dim, width), q + "v": (g * vdim, width)})
            shapes.update({q + name: (dim,) for name in ("lq1", "lk1", "lq2", "lk2")})
        else:
            shapes.update({q + "q": (heads * dim, width), q + "k": (heads * dim, width), q + "v": (heads * vdim, width),
                           q + "g": (heads * vdim, width)})
        shapes[q + "o"] = (width, heads * vdim)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        shapes[p + "norm2"] = (width,)
        ff, experts = (mlp["ff"], [""]) if mlp["kind"] == "dense" else (mlp["expert"]["ff"], [f"e{e}." for e in range(mlp["router"]["experts"])])
        for e in experts:
            shapes.update({f"{p}mlp.{e}gate": (ff, width), f"{p}mlp.{e}up": (ff, width), f"{p}mlp.{e}down": (width, ff)})
        if mlp["kind"] == "moe":
            shapes[p + "mlp.router"] = (mlp["router"]["experts"], width)
    return shapes


def random_weights(cfg, seed):
    """Weights that keep every mechanism alive: norms around one, both maps of an attention and their weight at work."""
    gen = torch.Generator().manual_seed(seed)
    scale = float(cfg["embedding"]["scale"])
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        normal = lambda std, mean=0.0: (torch.randn(shape, generator=gen) * std + mean)
        if last in ("norm1", "norm2") or name == "final.norm":
            t = normal(0.1, 1.0)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = normal(0.5 * shape[0] ** -0.25)
        elif last == "router":
            t = normal(2.0 * shape[-1] ** -0.5)
        elif name == "embed":
            t = normal(1.0 / scale)
        else:
            t = normal(shape[-1] ** -0.5)
        out[name] = t.to(torch.bfloat16).to(torch.float32)   # exact in both storage precisions
    return out
