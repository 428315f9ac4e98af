"""Grouped-query softmax attention whose query and key heads are RMS-normed with a gain over the head's elements before the
rotation, with a cap on the scores, and the options that come with it in designs of that kind.

q, k, v (and the output gate) come from one fused projection; with ``bias``, q, k and v have biases, added in float32.  Per head
and in float32,

    q <- q / sqrt(mean(q^2) + eps) * gain_q,  k likewise with gain_k       (one gain [dim] for all query heads, one for all key heads);
    rotation of the first ``rotary_dim`` elements by absolute position     (``position``: any registered encoding, or none);
    score(i, j) = softcap tanh((q_i . k_j) * scale / softcap)              (``softcap`` None: the scaled product as it is);
    softmax over the visible keys j <= i                                   (``window``: i - j < window; ``chunk``: the same run of
                                                                           ``chunk`` positions, counted from position 0).

Query head h reads key/value head h // (heads / kv_heads).  ``value_mix``: "source" leaves this layer's values (with their bias)
for later layers of the same step; "mixed" stores v <- (1 - share) v + share * v_source instead of v, ``share`` a learned number
(a tensor of both kinds of layer; a source does not use its own).  ``output_gate``: the heads' results are multiplied by
sigmoid(W_g x), element by element.  ``out_scale``: a factor on the result.

The cache entry keeps one row per token and key/value head, key then value, and the kernels over rows read it.
"""

from __future__ import annotations

import torch

from .. import ops
from ..config.spec import PartSpec
from .base import CacheNeed, CacheView, Mixer, PagedKV, ParamSpec, StepContext
from .registry import make, register_mixer

SOURCE_VALUES = "source_values"  # ctx.extras: (projected values [T, kv_heads * vdim] of the layer that lends them, their bias)


class HeadNormAttention(Mixer):
    graph_safe = True  # device work depends only on tensor shapes and device-side inputs

    def __init__(self, params):
        super().__init__(params)
        self.hidden = int(params["hidden_size"])
        self.hq = int(params["num_heads"])
        self.hkv = int(params["num_kv_heads"])
        self.dim = int(params["dim"])
        self.vdim = int(params.get("vdim") or self.dim)
        self.scale = float(params["scale"])
        self.eps = float(params["eps"])
        self.softcap = None if params.get("softcap") is None else float(params["softcap"])
        self.window = params.get("window")
        self.chunk = params.get("chunk")
        self.has_bias = bool(params.get("bias", False))
        self.value_mix = params.get("value_mix")
        self.output_gate = bool(params.get("output_gate", False))
        self.out_scale = float(params.get("out_scale", 1.0))
        if self.hq % self.hkv:
            raise ValueError(f"{self.hq} query heads cannot share {self.hkv} key/value heads")
        if self.value_mix not in (None, "source", "mixed"):
            raise ValueError(f"value_mix {self.value_mix!r}: one of None, 'source', 'mixed'")
        if self.softcap is not None and not self.softcap > 0:
            raise ValueError(f"the cap on the scores must be positive, is {self.softcap}")
        self.position = make("position", params.get("position") or PartSpec("none"))
        self.rotary_dim = int(getattr(self.position, "rotary_dim", None) or self.dim)
        self.interleaved = getattr(self.position, "layout", "half") == "interleaved"
        self.rows_width = self.hq * self.vdim
        self.qkv = (self.hq + self.hkv) * self.dim + self.hkv * self.vdim  # columns of the projection before the output gate
        self.w_in = self.w_o = self.b_in = self.b_v = self.gain_q = self.gain_k = self.share = None

    def param_specs(self):
        specs = {}
        for n, rows in (("q", self.hq * self.dim), ("k", self.hkv * self.dim), ("v", self.hkv * self.vdim)):
            specs[f"{n}_proj"] = ParamSpec((rows, self.hidden))
            if self.has_bias:
                specs[f"{n}_bias"] = ParamSpec((rows,), role="vector", init="normal")
        specs["q_norm"] = ParamSpec((self.dim,), role="vector", init="ones")
        specs["k_norm"] = ParamSpec((self.dim,), role="vector", init="ones")
        if self.value_mix is not None:
            specs["value_share"] = ParamSpec((), role="vector", init="normal")
        if self.output_gate:
            specs["gate_proj"] = ParamSpec((self.rows_width, self.hidden))
        specs["o_proj"] = ParamSpec((self.hidden, self.rows_width))
        return specs

    def cache_need(self):
        return CacheNeed(paged=PagedKV(self.hkv, self.dim + self.vdim, self.window, "natural", planes=1, chunk=self.chunk))

    def load(self, tensors, *, compute_dtype, device):
        f32 = dict(device=device, dtype=torch.float32)
        pieces = [tensors[f"{n}_proj"] for n in ("q", "k", "v") + (("gate",) if self.output_gate else ())]
        dtype = torch.float32 if any(p.dtype == torch.float32 for p in pieces) else pieces[0].dtype
        fill = torch.zeros((-sum(p.shape[0] for p in pieces) % 8, self.hidden), dtype=dtype, device=pieces[0].device)
        self.w_in = torch.cat([p.to(dtype) for p in pieces] + [fill], dim=0).contiguous()  # rows of the product start on 16 bytes
        self.w_o = tensors["o_proj"].contiguous()
        if self.has_bias:
            self.b_in = torch.cat([tensors[f"{n}_bias"].to(**f32) for n in ("q", "k", "v")]).contiguous()
            if self.value_mix == "source":  # on its own, so that it starts where wide loads may
                self.b_v = tensors["v_bias"].to(**f32).clone().contiguous()
        self.gain_q, self.gain_k = (tensors[f"{n}_norm"].to(**f32).contiguous() for n in ("q", "k"))
        if self.value_mix == "mixed":
            self.share = tensors["value_share"].to(**f32).reshape(1).contiguous()

    def prepare(self, *, max_positions, compute_dtype, device):
        self.position.prepare(max_positions=max_positions, compute_dtype=compute_dtype, device=device)

    def input_weight(self) -> torch.Tensor:
        """The one matrix this mixer applies to its input first (see ``side_by_side``)."""
        return self.w_in

    def output_weight(self) -> torch.Tensor:
        return self.w_o

    def drop_output_weight(self) -> None:
        self.w_o = None

    def forward_rows_projected(self, proj, ctx: StepContext, cache: CacheView, *, out=None):
        if not cache.writes or cache.kv is None:
            raise RuntimeError("an attention part with projections of its own must write its cache entry")
        table = ctx.block_tables[cache.group]
        values = self.qkv - self.hkv * self.vdim
        first = first_bias = None
        if self.value_mix == "source":
            ctx.extras[SOURCE_VALUES] = (proj[:, values: self.qkv], self.b_v)
        elif self.value_mix == "mixed":
            first, first_bias = ctx.extras[SOURCE_VALUES]
        q = ops.attention_prepare_heads(proj[:, : self.qkv], cache.kv, table, ctx, num_heads=self.hq, num_kv_heads=self.hkv, dim=self.dim,
                                        vdim=self.vdim, page_size=cache.page_size, gain_q=self.gain_q, gain_k=self.gain_k, eps=self.eps,
                                        cos=self.position.cos, sin=self.position.sin, rotary_dim=self.rotary_dim,
                                        interleaved=self.interleaved, bias=self.b_in, first=first, first_bias=first_bias, share=self.share)
        gate = proj[:, self.qkv: self.qkv + self.rows_width] if self.output_gate else None
        return ops.attention_over_rows(q, cache.kv, table, ctx, num_heads=self.hq, num_kv_heads=self.hkv, dim=self.dim, vdim=self.vdim,
                                       page_size=cache.page_size, scale=self.scale, window=self.window, chunk=self.chunk,
                                       softcap=self.softcap, gate=gate, out_scale=self.out_scale, out=out)

    def forward_rows(self, x, ctx: StepContext, cache: CacheView, *, out):
        self.forward_rows_projected(ops.linear(x, self.w_in), ctx, cache, out=out)

    def forward_projected(self, proj, ctx: StepContext, cache: CacheView):
        return ops.last_product(self.forward_rows_projected(proj, ctx, cache), self.w_o, ctx)

    def forward(self, x, ctx: StepContext, cache: CacheView):
        return self.forward_projected(ops.linear(x, self.w_in), ctx, cache)


register_mixer("head_norm_attention", HeadNormAttention, replace=True)
