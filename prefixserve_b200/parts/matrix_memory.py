"""Matrix memory with exponential gates: a matrix state per head whose write and forget strengths are exponentials of capped
pre-activations, read out through a normalizer.

From the input x: q = W_q x * dim^-1/2 and k = W_k x (``heads`` heads of ``dim``), v = W_v x (``heads`` of ``vdim``), an output
gate W_g x, and per head i = cap tanh((W_i x + b_i) / cap), f = logsigmoid(cap tanh((W_f x + b_f) / cap)).  Per head and token,
in float32 from S = 0 [dim, vdim], n = 0 [dim] and m = 0,

    m' = max(f + m, i),   (S, n) <- exp(f + m - m') (S, n) + exp(i - m') (k v^T, k),
    o = S^T q / (max(|n . q|, exp(-m')) + 1e-6);

o is divided by its root mean square over vdim, multiplied by a gain per head and channel and by sigmoid(W_g x), and projected by
W_o.  A request carries S, n and m in its slot; a fresh slot is zeros.  Everything that reads x is one product.  ``out_scale``: a
factor on the result (it rides in the gain).
"""

from __future__ import annotations

import torch

from .. import ops
from .base import CacheNeed, CacheView, FixedState, Mixer, ParamSpec, StepContext
from .registry import register_mixer


class MatrixMemory(Mixer):
    graph_safe = True  # device work depends only on tensor shapes and device-side inputs

    def __init__(self, params):
        super().__init__(params)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["num_heads"])
        self.dim = int(params["dim"])
        self.vdim = int(params["vdim"])
        self.cap = float(params["gate_cap"])
        self.eps = float(params["eps"])
        self.out_scale = float(params.get("out_scale", 1.0))
        if not self.cap > 0:
            raise ValueError(f"the cap of the gates must be positive, is {self.cap}")
        self.rows_width = self.heads * self.vdim
        self.w_in = self.w_o = self.bias_i = self.bias_f = self.gain = None

    def param_specs(self):
        qk, v = self.heads * self.dim, self.heads * self.vdim
        return {
            "q_proj": ParamSpec((qk, self.hidden)), "k_proj": ParamSpec((qk, self.hidden)), "v_proj": ParamSpec((v, self.hidden)),
            "gate_proj": ParamSpec((v, self.hidden)),
            "input_proj": ParamSpec((self.heads, self.hidden)), "input_bias": ParamSpec((self.heads,), role="vector", init="normal"),
            "forget_proj": ParamSpec((self.heads, self.hidden)), "forget_bias": ParamSpec((self.heads,), role="vector", init="normal"),
            "out_norm": ParamSpec((v,), role="vector", init="ones"), "o_proj": ParamSpec((self.hidden, v)),
        }

    def cache_need(self):
        return CacheNeed(state=FixedState((ops.matrix_memory_state(self.heads, self.dim, self.vdim),), torch.float32))

    def load(self, tensors, *, compute_dtype, device):
        f32 = dict(device=device, dtype=torch.float32)
        wide = [tensors[f"{n}_proj"] for n in ("q", "k", "v", "gate", "input", "forget")]
        dtype = torch.float32 if any(p.dtype == torch.float32 for p in wide) else wide[0].dtype
        fill = torch.zeros((-sum(p.shape[0] for p in wide) % 8, self.hidden), dtype=dtype, device=wide[0].device)
        self.w_in = torch.cat([p.to(dtype) for p in wide] + [fill], dim=0).contiguous()  # rows of the product start on 16 bytes
        self.w_o = tensors["o_proj"].contiguous()
        self.bias_i, self.bias_f = (tensors[f"{n}_bias"].to(**f32).contiguous() for n in ("input", "forget"))
        self.gain = (tensors["out_norm"].to(**f32) * self.out_scale).contiguous()

    def input_weight(self) -> torch.Tensor:
        """The one matrix this mixer applies to its input first (see ``side_by_side``)."""
        return self.w_in

    def output_weight(self) -> torch.Tensor:
        return self.w_o

    def drop_output_weight(self) -> None:
        self.w_o = None

    def forward_rows_projected(self, proj, ctx: StepContext, cache: CacheView, *, out=None):
        if cache.state is None or not cache.writes:
            raise RuntimeError("a recurrent part needs the state of its own cache entry")
        return ops.matrix_memory(proj, self.bias_i, self.bias_f, self.gain, cache.state, ctx, heads=self.heads, dim=self.dim,
                                 vdim=self.vdim, cap=self.cap, eps=self.eps, out=out)

    def forward_rows(self, x, ctx: StepContext, cache: CacheView, *, out):
        self.forward_rows_projected(ops.linear(x, self.w_in), ctx, cache, out=out)

    def forward_projected(self, proj, ctx: StepContext, cache: CacheView):
        return ops.last_product(self.forward_rows_projected(proj, ctx, cache), self.w_o, ctx)

    def forward(self, x, ctx: StepContext, cache: CacheView):
        return self.forward_projected(ops.linear(x, self.w_in), ctx, cache)


register_mixer("matrix_memory", MatrixMemory, replace=True)
