"""Differential attention over the cache: two softmax maps per head over the same values, one subtracted from the other.

  q = Wq h  [heads, 2, dim],  k = Wk h  [kv_heads, 2, dim],  v = Wv h  [kv_heads, vdim]     map 1 and map 2 one after the other
  q, k turned map by map           the position part (its factor on cosine and sine included)
  a_m = softmax(q_m k_m^T * scale) v      for both maps, key j visible iff max(0, p - window + 1) <= j <= p
  lam = exp(lq1 . lk1) - exp(lq2 . lk2) + offset        one number per layer, formed once when the weights are bound
  o = a_1 - lam a_2;   o <- (1 - offset) o / sqrt(mean(o^2) + eps) per head;   out = Wo concat_heads

The attention kernels know nothing of maps. A cached head is [k_1 | k_2] and v, and a query enters as a head of that size that is
zero outside its own map's half, so its product with the cached row is q_m . k_m: 2 * heads plain query heads over kv_heads cached
heads. Both maps of a head read the same cached row and the same value, which the cache keeps once. Heads whose size no tensor-core
kernel has are filled up with zeros to the next size that one has."""
from __future__ import annotations

import math

import torch

from .. import ops
from ..config.spec import PartSpec
from .attention import TC_PREFILL_MIN_TOKENS, GqaAttention
from .base import TensorSpec
from .registry import build_part, register_part

MAPS = 2


class DifferentialAttention(GqaAttention):
    """params: hidden_size, num_heads, num_kv_heads, head_dim (of one map), value_dim, scale, window, position (PartSpec | None), offset
    (`diff` above), eps. tensors: q_weight [heads * 2 * dim, W], k_weight [kv_heads * 2 * dim, W], v_weight [kv_heads * vdim, W],
    o_weight [W, heads * vdim], lq1, lk1, lq2, lk2 [dim]."""

    def __init__(self, spec):
        p = dict(spec.params)
        self.pairs, self.map_dim, vdim = int(p["num_heads"]), int(p["head_dim"]), int(p["value_dim"])
        size = max(MAPS * self.map_dim, vdim)
        size = next((d for d in ops.FAST_ATTENTION_HEAD_DIMS if d >= size), size)
        if size > 256 or vdim > ops.MAP_DIFFERENCE_MAX_VDIM:
            raise ValueError(f"differential_attention: heads of two maps of {self.map_dim} and values of {vdim} are not supported (256 at most)")
        super().__init__(PartSpec(spec.kind, {"hidden_size": p["hidden_size"], "num_heads": self.pairs * MAPS, "num_kv_heads": p["num_kv_heads"],
                                              "head_dim": size, "scale": p["scale"], "window": p.get("window") or 0, "position": None}, spec.tensors))
        self.value_dim = vdim
        self.offset, self.eps = float(p["offset"]), float(p["eps"])
        self.position = build_part("position", p["position"]) if p.get("position") is not None else None
        if self.position is not None and getattr(self.position, "interleaved", True):
            raise ValueError("differential_attention: the position part pairs component j with j + half")
        self.plain = False       # (no fused form of the base class applies)
        self.map_weight = 0.0    # lam

    def tensor_specs(self):
        dim, f = self.map_dim, self.file_name
        return [TensorSpec(f("q_weight"), (self.pairs * MAPS * dim, self.hidden)), TensorSpec(f("k_weight"), (self.n_kv * MAPS * dim, self.hidden)),
                TensorSpec(f("v_weight"), (self.n_kv * self.value_dim, self.hidden)),
                TensorSpec(f("o_weight"), (self.hidden, self.pairs * self.value_dim))] + \
               [TensorSpec(f(name), (dim,), init="conv", keep="float32") for name in ("lq1", "lk1", "lq2", "lk2")]

    def kernel_libraries(self, dtype):
        libs = super().kernel_libraries(dtype) | {"norm"}
        if dtype != torch.float32 and self.head_dim in ops.TC_ATTENTION_HEAD_DIMS:
            libs.add("attention_prefill_tc")
        return libs

    def bind(self, tensors, dtype, device):
        t = lambda logical: tensors[self.file_name(logical)]
        self.qkv_weight = torch.cat((t("q_weight"), t("k_weight"), t("v_weight")), dim=0).contiguous()
        self.o_weight = t("o_weight")
        dot = lambda a, b: float((t(a).to(torch.float32).double() * t(b).to(torch.float32).double()).sum().item())
        self.map_weight = math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + self.offset

    def step_weights(self):
        return [self.qkv_weight, self.o_weight]

    def fused_takes(self, ctx) -> bool:
        return False

    def forward(self, x, ctx, site, writes_cache):
        n = x.shape[0]
        inv_freq, rot_dim = self.position.fused_rotary() if self.position is not None else (None, 0)
        amplitude = self.position.amplitude if self.position is not None else 1.0
        qkv = ops.linear_rows(x, self.qkv_weight)
        q = torch.empty((n, self.q_width), dtype=x.dtype, device=x.device)
        args = ops.KvSiteArgs(site.storage, site.table, self.n_kv, self.head_dim)
        ops.rope_maps_cache_write(qkv, ctx.tok_seq, ctx.tok_pos, ctx.slots, inv_freq, rot_dim, amplitude, self.pairs, MAPS, self.map_dim,
                                  self.value_dim, q, args, writes_cache, ctx.err)
        out = torch.empty((n, self.pairs * self.value_dim), dtype=x.dtype, device=x.device)
        fast = ctx.attention == "auto" and x.dtype == torch.bfloat16 and self.head_dim in ops.FAST_ATTENTION_HEAD_DIMS
        if fast and ctx.is_decode and n == ctx.n_seqs:   # single tokens: the maps meet inside the attention kernel
            ops.attention_decode(q, out, ctx.cu_q, ctx.tok_pos, ctx.slots, args, self.n_heads, ctx.n_seqs, self.scale, self.window,
                                 self.decode_splits(ctx), ctx.decode_scratch, ctx.err, self.decode_plan(ctx),
                                 pairs=(self.map_weight, self.eps, 1.0 - self.offset, self.value_dim))
            return ops.linear_rows(out, self.o_weight)
        attended = torch.empty_like(q)
        common = (q, attended, ctx.cu_q, ctx.tok_pos, ctx.slots, args, self.n_heads, ctx.n_seqs)
        if fast:
            least = TC_PREFILL_MIN_TOKENS.get(self.head_dim)
            run = ops.attention_prefill_tc if least is not None and n >= least and ctx.max_q_len >= 128 else ops.attention_prefill
            run(*common, ctx.max_q_len, self.scale, self.window, ctx.err, max_kv_len=ctx.max_kv_len)
        else:
            ops.attention_generic(*common, ctx.max_q_len, self.scale, self.window, ctx.err, scratch=ctx.decode_scratch,
                                  max_kv_len=ctx.max_kv_len)
        ops.map_difference(attended, self.head_dim, self.map_weight, self.eps, 1.0 - self.offset, out, self.pairs, self.value_dim)
        return ops.linear_rows(out, self.o_weight)


register_part("mixer", "differential_attention", DifferentialAttention)
