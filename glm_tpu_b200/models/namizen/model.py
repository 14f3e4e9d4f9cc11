"""The Namizen decoder as a sequence of CUDA kernel launches on one GPU.

``run_rows`` is called as in the other model families (the runner drives them all the same way): ``R`` token rows through every layer,
decode (one row per lane, 1..8, captured in a CUDA graph by the runner) or prefill (many rows of one lane at consecutive positions).

Per layer, five launches in decode:

    parallel_norm     residual += last update (or = embedding); both normalized inputs
    dual_proj         q | k | v projection and gate / up / GELU of the feed-forward
    qkv_conv          short convolution, rotation, value mixing, ring and state write
    chunk_attention   over the lane's ring
    skinny_bf16       [attention | feed-forward] @ [W_o | W_down]: the fp32 update of the residual

In prefill the projections run on the tcgen05 GEMM (gate / up and activation are two launches).  A step whose rows lie in one chunk of a layer
attends over the lane's ring itself; one that crosses into another chunk attends over a linear buffer (the chunk so far, copied from the
ring, then the step's rows), and the rows of the last chunk enter the ring afterwards.

The residual, norms, angles, scores, softmax and sums are fp32 in every mode.  ``weights.dtype`` selects the rest: bf16 operands with fp32
accumulation, or fp32 throughout (plain FMA kernels: the 32-bit path exists to check the model, not to serve it).
"""

from __future__ import annotations

from dataclasses import dataclass, field

import torch

from glm_tpu_b200.config.cache import RingCacheConfig
from glm_tpu_b200.exceptions import PlanValidationError
from glm_tpu_b200.model_loader.directory import pad8, pad16
from glm_tpu_b200.models.namizen.weights import NamizenWeights
from glm_tpu_b200.ops import native
from glm_tpu_b200.parallel.peer import PeerGroup
from glm_tpu_b200.runner.lane_state import RING, LaneRegisters


@dataclass
class RingState(LaneRegisters):
    """Lane registers plus every layer's rings and convolution state.  Nothing is cleared for a new request: reads are bounded by the
    position, so what an earlier request left behind is never seen."""

    k: list = field(default_factory=list)
    v: list = field(default_factory=list)
    conv: list = field(default_factory=list)

    @classmethod
    def allocate(cls, cache: RingCacheConfig, device, dtype: torch.dtype) -> "RingState":
        layers = range(len(cache.geometry.layers))
        make = lambda shape: torch.zeros(shape, dtype=dtype, device=device)  # noqa: E731
        return cls(**cls.registers(cache.lanes, device), k=[make(cache.k_shape(i)) for i in layers], v=[make(cache.v_shape(i)) for i in layers],
                   conv=[make(cache.conv_shape(i)) for i in layers])


class NamizenWorkspace:
    """Scratch tensors for ``rows`` token rows, sized for the widest layer; ``prefill`` adds the linear key / value buffers."""

    def __init__(self, model: "NamizenModel", rows: int, *, prefill: bool):
        g, dev, T = model.g, model.device, model.w.dtype
        self.rows = rows
        mixers = [layer.mixer for layer in g.layers]
        t = lambda *s: torch.zeros(s, dtype=T, device=dev)  # noqa: E731
        self.residual = torch.zeros((rows, model.width), dtype=torch.float32, device=dev)
        self.update = torch.zeros((rows, model.width), dtype=torch.float32, device=dev)
        self.h1, self.h2 = t(rows, model.width), t(rows, model.width)
        # flat buffers: every layer views them with its own row size
        self.proj = t(rows * max(pad8(m.qkv_width) for m in mixers))
        self.q = t(rows * max(m.heads * pad16(m.dim) for m in mixers))
        self.branches = {cols: t(rows, cols) for cols in {(lw.attn_cols + lw.ff_cols) for lw in model.w.layers}}
        # linear keys and values of a prefill step that crosses a chunk
        lin = [model.cache.linear_rows(i, rows) if prefill else 0 for i in range(g.num_layers)]
        self.k_lin = t(max(n * m.kv_heads * pad16(m.dim) for n, m in zip(lin, mixers)))
        self.v_lin = t(max(n * m.kv_heads * pad16(m.vdim) for n, m in zip(lin, mixers)))
        self.v_first = t(rows * max([m.v_width for m in mixers if m.v_mix] or [8]))
        self.gate_up = t(rows * 2 * max(lw.ff_cols for lw in model.w.layers)) if prefill or model.is_f32 else None
        self.logits = torch.zeros((rows if not prefill else 0, pad8(g.vocab_size)), dtype=torch.float32, device=dev)
        self.local_best = torch.zeros(rows, dtype=torch.int64, device=dev)
        self.cand = torch.zeros((1, rows), dtype=torch.int64, device=dev)

    def bytes(self) -> int:
        tensors = [v for v in vars(self).values() if isinstance(v, torch.Tensor)] + list(self.branches.values())
        return sum(t.numel() * t.element_size() for t in tensors)


class NamizenModel:
    library_component = "namizen"

    def __init__(self, weights: NamizenWeights, cache: RingCacheConfig, peer: PeerGroup):
        self.w, self.cache, self.peer = weights, cache, peer
        self.g, self.device = weights.geometry, weights.embed.device
        self.is_f32 = weights.dtype == torch.float32
        self.width = weights.embed.shape[1]
        self.trace = None  # set to a dict to record the residual after every layer (tests)
        self.plain_attention = False  # tests: the size-independent attention kernel instead of the tensor-core ones
        self.fallbacks: dict[str, int] = {}
        for i, layer in enumerate(self.g.layers):
            m = layer.mixer
            if m.conv > native.qkv_conv_max_taps(max(m.dim, m.vdim)) or m.vdim > 1024 or m.dim > 8192:
                raise PlanValidationError(f"layer {i}: head sizes ({m.dim}, {m.vdim}) with {m.conv} taps exceed the kernels' limits")
        # one fp32 (cos, sin) table per distinct rotation, from float64 angles
        tables: dict = {}
        for layer in self.g.layers:
            key = (layer.mixer.rot_dims, layer.mixer.rot_base)
            if key not in tables:
                dims, base = key
                i = torch.arange(dims // 2, dtype=torch.float64)
                angle = torch.arange(cache.context_capacity, dtype=torch.float64)[:, None] * base ** (-2.0 * i / max(dims, 1))
                tables[key] = torch.stack([angle.cos(), angle.sin()], dim=-1).to(torch.float32).contiguous().to(self.device)
        self.rot = [tables[(layer.mixer.rot_dims, layer.mixer.rot_base)] for layer in self.g.layers]

    # ------------------------------------------------------------------------------ pieces of a layer
    def _mm(self, x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
        """``out = x @ w.T``; every operand is padded to the kernels' alignment."""
        if self.is_f32:
            native.gemm_f32(x, w, out)
        elif x.shape[0] <= native.MAX_ROWS:
            native.skinny_bf16(x, w, out, native.SK_OUT_F32 if out.dtype == torch.float32 else native.SK_OUT_BF16)
        else:
            native.gemm_bf16_tc(x, w, out, status=self.peer.status_ptr)

    def _attention(self, ws: NamizenWorkspace, state: RingState, layer: int, proj: torch.Tensor, out: torch.Tensor, rows: int, row_pos, row_lane,
                   row_active, decode: bool, start: int, lane: int) -> None:
        m, lw, cache = self.g.layers[layer].mixer, self.w.layers[layer], self.cache
        first = self.g.first_mixing_layer
        a = native.QkvConvArgs()
        a.proj, a.proj_stride = proj.data_ptr(), proj.stride(0)
        a.conv_w, a.taps, a.state = lw.conv.data_ptr(), m.conv, state.conv[layer].data_ptr()
        a.row_pos, a.row_lane = row_pos.data_ptr(), row_lane.data_ptr()
        a.row_active = row_active.data_ptr() if row_active is not None else None
        a.rot, a.rot_dims = self.rot[layer].data_ptr(), m.rot_dims
        a.q = ws.q.data_ptr()
        a.k_ring, a.v_ring, a.ring = state.k[layer].data_ptr(), state.v[layer].data_ptr(), cache.ring(layer)
        a.v_first, a.v_mode, a.mix = ws.v_first.data_ptr(), (0 if not m.v_mix else 1 if layer == first else 2), lw.mix
        a.H, a.G, a.dim, a.dimp, a.vdim, a.vdimp = m.heads, m.kv_heads, m.dim, pad16(m.dim), m.vdim, pad16(m.vdim)
        a.rows, a.decode, a.capacity, a.lanes = rows, int(decode), cache.context_capacity, cache.lanes
        a.status = self.peer.status_ptr
        b = native.ChunkAttnArgs()
        b.q, b.sink = a.q, lw.sink.data_ptr()
        b.row_pos, b.row_lane, b.row_active = a.row_pos, a.row_lane, a.row_active
        b.out, b.out_stride = out.data_ptr(), out.stride(0)
        b.rows, b.H, b.G, b.dim, b.dimp, b.vdim, b.vdimp = rows, m.heads, m.kv_heads, m.dim, a.dimp, m.vdim, a.vdimp
        b.decode, b.chunk, b.ring, b.capacity, b.lanes, b.scale = a.decode, cache.chunk(layer), a.ring, a.capacity, a.lanes, m.scale
        b.status = self.peer.status_ptr
        if decode:
            b.k, b.v = a.k_ring, a.v_ring
            native.qkv_conv(a, self.is_f32)
            native.chunk_attention(b, self.is_f32, plain=self.plain_attention)
            return
        k_row, v_row = (m.kv_heads * padded * state.k[layer].element_size() for padded in (a.dimp, a.vdimp))  # bytes of a cached row
        k_lane, v_lane = a.k_ring + lane * a.ring * k_row, a.v_ring + lane * a.ring * v_row
        b.start, b.base = start, cache.first_position(layer, start)
        b.keys = start + rows - b.base
        across = cache.crossing(layer, start, rows)
        if across is None:
            b.k, b.v = k_lane, v_lane
            native.qkv_conv(a, self.is_f32)
            native.chunk_attention(b, self.is_f32, plain=self.plain_attention)
            return
        before, after = across
        b.k, b.v = ws.k_lin.data_ptr(), ws.v_lin.data_ptr()
        if before:
            native.kv_copy(k_lane, b.k, before * k_row, v_lane, b.v, before * v_row)
        a.k_lin, a.v_lin = b.k + before * k_row, b.v + before * v_row
        native.qkv_conv(a, self.is_f32)
        native.chunk_attention(b, self.is_f32, plain=self.plain_attention)
        tail = b.keys - after
        native.kv_copy(b.k + tail * k_row, k_lane, after * k_row, b.v + tail * v_row, v_lane, after * v_row)

    def _layer(self, ws, state, layer: int, rows: int, row_pos, row_lane, row_active, decode: bool, start: int, lane: int) -> None:
        """Both branches of a layer from ``ws.h1`` / ``ws.h2``; the fp32 update of the residual lands in ``ws.update``."""
        lw = self.w.layers[layer]
        both = ws.branches[lw.attn_cols + lw.ff_cols][:rows]
        n = lw.qkv.shape[0]
        proj = ws.proj[: rows * n].view(rows, n)
        h1, h2 = ws.h1[:rows], ws.h2[:rows]
        act = both[:, lw.attn_cols :]
        # several layers share the row buffer: columns between a branch's width and its padding take whatever an earlier layer of the same
        # row size left there, and meet zero weights (all values are finite)
        if decode and not self.is_f32:
            if lw.ff_cols:
                native.dual_proj(h1, lw.qkv, proj, h2, lw.gate_up[: lw.ff_cols], lw.gate_up[lw.ff_cols :], act, native.GLU_GELU_TANH)
            else:
                native.dual_proj(h1, lw.qkv, proj)
        else:
            self._mm(h1, lw.qkv, proj)
            if lw.ff_cols:
                gate_up = ws.gate_up[: rows * 2 * lw.ff_cols].view(rows, 2 * lw.ff_cols)
                self._mm(h2, lw.gate_up, gate_up)
                native.glu_rows(gate_up[:, : lw.ff_cols], gate_up[:, lw.ff_cols :], act, native.GLU_GELU_TANH)
        self._attention(ws, state, layer, proj, both, rows, row_pos, row_lane, row_active, decode, start, lane)
        self._mm(both, lw.out, ws.update[:rows])

    # ------------------------------------------------------------------------------ whole model
    def run_rows(self, ws: NamizenWorkspace, state: RingState, tokens: torch.Tensor, row_pos: torch.Tensor, row_lane: torch.Tensor, row_active,
                 rows: int, *, decode: bool, max_ctx: int, head_rows=None, head: str = "logits", lane_of_rows: int | None = None):
        """Push ``rows`` token rows through the decoder; in prefill they are the positions ``max_ctx - rows .. max_ctx - 1`` of one lane.

        ``head='logits'`` returns the fp32 logits of ``head_rows`` (a slice or an index tensor; ``None``: all rows); ``head='argmax'``
        (decode) leaves the packed best candidates in ``ws.local_best`` and returns ``None``; ``head='none'`` stops after the layers.
        """
        g, w, eps = self.g, self.w, self.g.norm_eps
        start = 0 if decode else max_ctx - rows
        if not decode and not (0 <= start and max_ctx <= self.cache.context_capacity and lane_of_rows is not None and 0 <= lane_of_rows < self.cache.lanes):
            raise ValueError("prefill rows lie within the context of one lane")
        residual, update = ws.residual[:rows], None
        for i, lw in enumerate(w.layers):
            source = dict(tokens=tokens, table=w.embed, vocab=g.vocab_size) if i == 0 else dict(update=update)
            native.parallel_norm(residual, g.hidden_size, lw.norm1, ws.h1[:rows], eps, w2=lw.norm2, out2=ws.h2 if lw.norm2 is not None else None,
                                 status=self.peer.status_ptr, **source)
            self._layer(ws, state, i, rows, row_pos, row_lane, row_active, decode, start, lane_of_rows)
            update = ws.update[:rows]
            if self.trace is not None:
                self.trace.setdefault("residual", {})[i] = (residual + update)[:, : g.hidden_size].clone()
        if head == "none":
            return None
        native.parallel_norm(residual, g.hidden_size, w.final_norm, ws.h1[:rows], eps, update=update, status=self.peer.status_ptr)
        x = ws.h1[:rows] if head_rows is None else ws.h1[:rows][head_rows]
        if head == "argmax" and not self.is_f32:
            native.skinny_bf16(x, w.head, ws.local_best, native.SK_OUT_ARGMAX_F32, N=g.vocab_size, comm=self.peer.comm, channel=0, os_=0)
            return None
        logits = ws.logits if decode else torch.empty((x.shape[0], w.head.shape[0]), dtype=torch.float32, device=self.device)
        self._mm(x, w.head, logits[: x.shape[0]])
        return logits[: x.shape[0], : g.vocab_size]

    def sample(self, ws: NamizenWorkspace, state: RingState, logits, rows: int, row_active, *, advance: int, tokens_out=None, positions=None,
               out=None) -> None:
        """Greedy sampling (ties to the lowest id); the registers and the output ring are written as by the other families."""
        local_best = ws.local_best if logits is None else None
        if logits is not None:
            native.argmax_rows(logits, rows, self.g.vocab_size, 0, ws.cand, status=self.peer.status_ptr)
        counter, ring = (state.step_counter, RING) if out is None else (None, 1)
        native.step_finalize(ws.cand, 1, rows, row_active, state.tokens if tokens_out is None else tokens_out,
                             state.positions if positions is None else positions, state.out_tokens if out is None else out, counter, ring, advance,
                             local_best=local_best)
