"""The Zikevik decoder as a sequence of CUDA kernel launches on one GPU.

``run_rows`` is called as in the other model families (the runner drives them all the same way): ``R`` token rows through every layer,
decode (one row per lane, 1..8, captured in a CUDA graph by the runner) or prefill (many rows of one lane at consecutive positions).

A layer is a norm (which first adds the previous update to the fp32 residual), the mixer, a norm, the feed-forward.  The mixers:

    delta rule   projection -> convolution, unit vectors, decays -> recurrence over the lane's state -> norm and gate -> projection
    latent       projection -> latents (the cache write) -> queries -> attention -> projection.  Decode and short steps compare queries
                 that went through the key projection with the cache rows as they are; longer prefill steps expand the lane's cache to
                 keys and values per head, some heads at a time, and attend with those.

The residual, norms, router, angles, scores, softmax, sums, recurrent state and everything that enters the recurrence after the projections and
convolutions are fp32 in every mode.  ``weights.dtype`` selects the rest: bf16 operands with fp32 accumulation, or fp32 throughout (plain FMA
kernels: the 32-bit path exists to check the model, not to serve it).
"""

from __future__ import annotations

from dataclasses import dataclass, field

import torch

from glm_tpu_b200.config.cache import HybridCacheConfig
from glm_tpu_b200.config.zikevik import DeltaSpec, LatentSpec, RoutedSpec
from glm_tpu_b200.exceptions import PlanValidationError
from glm_tpu_b200.model_loader.directory import pad8, pad16, pad_to
from glm_tpu_b200.models.zikevik.weights import ZikevikWeights
from glm_tpu_b200.ops import native
from glm_tpu_b200.parallel.peer import PeerGroup
from glm_tpu_b200.runner.lane_state import RING, LaneRegisters

EXPAND_BYTES = 1 << 30  # keys and values of as many heads at a time as fit here
RECORD_BYTES = 128 << 20  # what the chunked recurrence keeps between its two kernels
ABSORB_ROWS = native.MAX_ROWS  # steps of up to this many rows attend over the cache rows as they are
MAX_EXPERTS, MAX_TOP = 256, 32  # limits of the route sort and the router kernel


@dataclass
class HybridState(LaneRegisters):
    """Lane registers plus every layer's cache or state (``None`` where a layer has none of the kind).  Nothing is cleared for a new request:
    reads are bounded by the position, and a sequence at position 0 starts from zeros."""

    latent: list = field(default_factory=list)
    state: list = field(default_factory=list)
    conv: list = field(default_factory=list)

    @classmethod
    def allocate(cls, cache: HybridCacheConfig, device, dtype: torch.dtype) -> "HybridState":
        layers = range(len(cache.geometry.layers))
        make = lambda shape, t: torch.zeros(shape, dtype=t, device=device)  # noqa: E731
        return cls(**cls.registers(cache.lanes, device), latent=[make(cache.latent_shape(i), dtype) if cache.is_latent(i) else None for i in layers],
                   state=[None if cache.is_latent(i) else make(cache.state_shape(i), torch.float32) for i in layers],
                   conv=[None if cache.is_latent(i) else make(cache.conv_shape(i), dtype) for i in layers])


def delta_record_bytes(m: DeltaSpec) -> int:
    """Bytes per 16 tokens and head that the chunked recurrence keeps between its two kernels (0: other sizes, token by token)."""
    dimp, blocks = pad_to(m.dim, 32), pad16(m.vdim) // 16
    if m.dim > 128 or m.dim % 8 or m.vdim % 8 or m.conv > 4:
        return 0
    return 6 * 16 * (dimp + 8) * 2 + 4 * 16 * 24 * 2 + dimp * 4 + blocks * 16 * 20 * 4


def expand_heads(m: LatentSpec, capacity: int, element_bytes: int) -> int:
    """Heads whose keys and values are expanded at a time."""
    per_head = capacity * (pad16(m.dim + m.rot_dim) + pad16(m.vdim)) * element_bytes
    return max(1, min(m.heads, EXPAND_BYTES // per_head))


def workspace_elements(g, cache: HybridCacheConfig, rows: int, *, prefill: bool, is_f32: bool) -> dict:
    """Elements per scratch buffer: ``(model dtype, fp32)`` sizes by name, the widest layer each."""
    t: dict[str, int] = {}
    f: dict[str, int] = {}

    def need(sizes: dict, name: str, n: int) -> None:
        sizes[name] = max(sizes.get(name, 0), n)

    for i, layer in enumerate(g.layers):
        m = layer.mixer
        need(t, "mixed", rows * pad8(m.out_width))
        if isinstance(m, DeltaSpec):
            dimp = pad_to(m.dim, 32)
            need(t, "proj", rows * (pad8(m.conv_width) + pad8(m.heads) + pad8(m.decay_rank) + pad8(m.gate_rank)))
            need(t, "gate", rows * pad8(m.v_width))
            need(f, "a", rows * pad8(m.heads * m.dim))
            for name in ("dq", "dk"):
                need(f, name, rows * m.kv_heads * dimp)
            need(f, "lg", rows * m.heads * dimp)
            for name in ("dv", "do"):
                need(f, name, rows * m.v_width)
            need(f, "beta", rows * m.heads)
            if prefill and not is_f32 and delta_record_bytes(m):
                chunks = min(-(-rows // 16), max(1, RECORD_BYTES // (m.heads * delta_record_bytes(m))))
                need(f, "records", chunks * m.heads * delta_record_bytes(m) // 4)
        else:
            lat, pe = cache.latent_columns(i)
            need(t, "proj", rows * (pad8(m.q_rank) + pad8(m.kv_rank + m.rot_dim) + pad8(m.heads)))
            need(t, "cq", rows * pad8(m.q_rank))
            need(t, "q", rows * m.heads * pad16(m.dim + m.rot_dim))
            few = min(rows, ABSORB_ROWS) if prefill else rows
            need(t, "qa", few * m.heads * (lat + pe))
            need(t, "o_lat", few * m.heads * m.kv_rank)
            need(f, "part_o", max(few, 32) * m.heads * lat)
            need(f, "part_ml", max(few, 32) * m.heads * 2)
            if prefill and rows > ABSORB_ROWS:
                heads = expand_heads(m, cache.context_capacity, cache.element_bytes)
                need(t, "keys", cache.context_capacity * heads * pad16(m.dim + m.rot_dim))
                need(t, "values", cache.context_capacity * heads * pad16(m.vdim))
        if layer.mlp is not None:
            F = pad8(layer.mlp.ff)
            routes = rows * (layer.mlp.top if isinstance(layer.mlp, RoutedSpec) else 1)
            need(t, "act", routes * F)
            if prefill or is_f32:
                need(t, "gate_up", routes * 2 * F)
            if isinstance(layer.mlp, RoutedSpec):
                need(f, "router", rows * pad8(layer.mlp.experts))
                if prefill and not is_f32:
                    need(t, "sorted", routes * pad8(g.hidden_size))
                    need(f, "expert_out", routes * pad8(g.hidden_size))
    return {"model": t, "f32": f}


class ZikevikWorkspace:
    """Scratch tensors for ``rows`` token rows, sized for the widest layer: flat buffers that every layer views with its own row size."""

    def __init__(self, model: "ZikevikModel", rows: int, *, prefill: bool):
        g, dev = model.g, model.device
        self.rows = rows
        sizes = workspace_elements(g, model.cache, rows, prefill=prefill, is_f32=model.is_f32)
        self.flat = {name: torch.zeros(n, dtype=model.w.dtype, device=dev) for name, n in sizes["model"].items()}
        self.flat |= {name: torch.zeros(n, dtype=torch.float32, device=dev) for name, n in sizes["f32"].items()}
        self.residual = torch.zeros((rows, model.width), dtype=torch.float32, device=dev)
        self.update = torch.zeros((rows, model.width), dtype=torch.float32, device=dev)
        self.h = torch.zeros((rows, model.width), dtype=model.w.dtype, device=dev)
        routed = [layer.mlp for layer in g.layers if isinstance(layer.mlp, RoutedSpec)]
        routes = rows * max([m.top for m in routed] or [0])
        i32 = lambda *s: torch.zeros(s, dtype=torch.int32, device=dev)  # noqa: E731
        self.route_ids, self.route_weights = i32(routes), torch.zeros(routes, dtype=torch.float32, device=dev)
        self.perm, self.place, self.n_tiles = i32(routes), i32(routes), i32(1)
        self.tiles = i32(routes // 128 + max([m.experts for m in routed] or [0]) + 1, 4)
        self.logits = torch.zeros((rows if not prefill else 0, pad8(g.vocab_size)), dtype=torch.float32, device=dev)
        self.local_best = torch.zeros(rows, dtype=torch.int64, device=dev)
        self.cand = torch.zeros((1, rows), dtype=torch.int64, device=dev)

    def view(self, name: str, rows: int, cols: int) -> torch.Tensor:
        return self.flat[name][: rows * cols].view(rows, cols)

    def bytes(self) -> int:
        tensors = [v for v in vars(self).values() if isinstance(v, torch.Tensor)] + list(self.flat.values())
        return sum(t.numel() * t.element_size() for t in tensors)


class ZikevikModel:
    library_component = "zikevik"

    def __init__(self, weights: ZikevikWeights, cache: HybridCacheConfig, peer: PeerGroup):
        self.w, self.cache, self.peer = weights, cache, peer
        self.g, self.device = weights.geometry, weights.embed.device
        self.is_f32 = weights.dtype == torch.float32
        self.width = weights.embed.shape[1]
        self.trace = None  # set to a dict to record the residual after every layer (tests)
        self.plain_kernels = False  # tests: the size-independent kernels instead of the specialised ones
        self.fallbacks: dict[str, int] = {}
        for i, layer in enumerate(self.g.layers):
            m = layer.mixer
            if isinstance(m, DeltaSpec) and (m.dim > 256 or m.conv > native.delta_max_taps()):
                raise PlanValidationError(f"layer {i}: {m.dim} key channels with {m.conv} taps exceed the kernels' limits")
            if isinstance(m, LatentSpec) and max(m.kv_rank, m.vdim, m.dim) > 1024:
                raise PlanValidationError(f"layer {i}: a latent of {m.kv_rank} with head sizes ({m.dim}, {m.vdim}) exceeds the kernels' limits")
            if isinstance(layer.mlp, RoutedSpec) and (layer.mlp.experts > MAX_EXPERTS or layer.mlp.top > MAX_TOP):
                raise PlanValidationError(f"layer {i}: at most {MAX_EXPERTS} experts, {MAX_TOP} of them per token")
        # one fp32 (cos, sin) table per distinct rotation, from float64 angles
        tables: dict = {}
        self.rot: list = []
        for layer in self.g.layers:
            m = layer.mixer
            if not isinstance(m, LatentSpec):
                self.rot.append(None)
                continue
            key = (m.rot_dim, m.rot_base)
            if key not in tables:
                i = torch.arange(m.rot_dim // 2, dtype=torch.float64)
                angle = torch.arange(cache.context_capacity, dtype=torch.float64)[:, None] * m.rot_base ** (-2.0 * i / m.rot_dim)
                tables[key] = torch.stack([angle.cos(), angle.sin()], dim=-1).to(torch.float32).contiguous().to(self.device)
            self.rot.append(tables[key])

    # ------------------------------------------------------------------------------ pieces of a layer
    def _mm(self, x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
        """``out = x @ w.T``; every operand is padded to the kernels' alignment."""
        if self.is_f32:
            native.gemm_f32(x, w, out)
        elif x.shape[0] <= native.MAX_ROWS:
            native.skinny_bf16(x, w, out, native.SK_OUT_F32 if out.dtype == torch.float32 else native.SK_OUT_BF16)
        else:
            native.gemm_bf16_tc(x, w, out, status=self.peer.status_ptr)

    def _rows(self, a, rows: int, row_pos, row_lane, row_active) -> None:
        """The arguments every row-wise structure has."""
        a.row_pos, a.row_lane = row_pos.data_ptr(), row_lane.data_ptr()
        a.row_active = row_active.data_ptr() if row_active is not None else None
        a.rows, a.lanes, a.capacity, a.status = rows, self.cache.lanes, self.cache.context_capacity, self.peer.status_ptr

    def _delta(self, ws: ZikevikWorkspace, state: HybridState, layer: int, rows: int, row_pos, row_lane, row_active, decode: bool) -> torch.Tensor:
        m, t = self.g.layers[layer].mixer, self.w.layers[layer].mixer
        h = ws.h[:rows]
        proj = ws.view("proj", rows, t.proj.shape[0])
        self._mm(h, t.proj, proj)
        out = ws.view("mixed", rows, t.out.shape[1])
        a = native.DeltaArgs()
        self._rows(a, rows, row_pos, row_lane, row_active)
        a.proj, a.proj_stride, a.off_b = proj.data_ptr(), proj.stride(0), t.off_b
        a.conv_w, a.taps, a.conv_state = t.conv.data_ptr(), m.conv, state.conv[layer].data_ptr()
        a.a_rate, a.dt_bias, a.norm = t.a_rate.data_ptr(), t.dt_bias.data_ptr(), t.norm.data_ptr()
        a.q, a.k, a.v, a.lg, a.beta, a.o = (ws.flat[n].data_ptr() for n in ("dq", "dk", "dv", "lg", "beta", "do"))
        a.state = state.state[layer].data_ptr()
        a.out, a.out_stride = out.data_ptr(), out.stride(0)
        a.H, a.G, a.dim, a.dimp, a.vdim, a.decode, a.eps = m.heads, m.kv_heads, m.dim, pad_to(m.dim, 32), m.vdim, int(decode), self.g.norm_eps
        ra, rg = t.a2.shape[1], t.g2.shape[1]
        if decode and not (self.is_f32 or self.plain_kernels) and native.delta_step_takes(m.vdim, ra + rg):
            a.a2, a.g2, a.off_a, a.off_g, a.ra, a.rg = t.a2.data_ptr(), t.g2.data_ptr(), t.off_a, t.off_g, ra, rg
            native.delta_step(a)
            return out
        decay, gate = ws.view("a", rows, t.a2.shape[0]), ws.view("gate", rows, t.g2.shape[0])
        self._mm(proj[:, t.off_a : t.off_a + ra], t.a2, decay)
        self._mm(proj[:, t.off_g : t.off_g + rg], t.g2, gate)
        a.a, a.a_stride, a.gate, a.gate_stride = decay.data_ptr(), decay.stride(0), gate.data_ptr(), gate.stride(0)
        if not decode and "records" in ws.flat and delta_record_bytes(m) and not self.plain_kernels:
            native.delta_chunk(a, ws.flat["records"])
        else:
            native.delta_prep(a, self.is_f32)
            native.delta_scan(a)
        native.delta_out(a, self.is_f32)
        return out

    def _latent(self, ws: ZikevikWorkspace, state: HybridState, layer: int, rows: int, row_pos, row_lane, row_active, decode: bool, start: int,
                lane: int | None) -> torch.Tensor:
        m, t, cache = self.g.layers[layer].mixer, self.w.layers[layer].mixer, self.cache
        lat, pe = cache.latent_columns(layer)
        proj = ws.view("proj", rows, t.proj.shape[0])
        self._mm(ws.h[:rows], t.proj, proj)
        cq, q = ws.view("cq", rows, t.uq.shape[1]), ws.view("q", rows, t.uq.shape[0])
        out = ws.view("mixed", rows, t.out.shape[1])
        a = native.LatentArgs()
        self._rows(a, rows, row_pos, row_lane, row_active)
        a.proj, a.proj_stride, a.off_kv, a.off_gate = proj.data_ptr(), proj.stride(0), t.off_kv, t.off_gate
        a.q_norm, a.kv_norm, a.rot = t.q_norm.data_ptr(), t.kv_norm.data_ptr(), self.rot[layer].data_ptr()
        a.cq, a.cq_stride, a.cache, a.q = cq.data_ptr(), cq.stride(0), state.latent[layer].data_ptr(), q.data_ptr()
        a.uk, a.uv, a.out, a.out_stride = t.uk.data_ptr(), t.uv.data_ptr(), out.data_ptr(), out.stride(0)
        a.H, a.dim, a.rot_dim, a.dimp, a.vdim, a.q_rank, a.kv_rank, a.lat, a.pe = m.heads, m.dim, m.rot_dim, t.dimp, m.vdim, m.q_rank, m.kv_rank, lat, pe
        a.eps = self.g.norm_eps
        native.latent_rows(a, self.is_f32)
        self._mm(cq, t.uq, q)
        b = native.ChunkAttnArgs()
        self._rows(b, rows, row_pos, row_lane, row_active)
        b.H, b.scale, b.chunk, b.ring, b.sink = m.heads, m.scale, cache.context_capacity, cache.context_capacity, t.sink.data_ptr()
        if decode or rows <= ABSORB_ROWS:
            # one key head: the cache row is the key, its first columns are the value
            a.qa, a.o_lat = ws.flat["qa"].data_ptr(), ws.flat["o_lat"].data_ptr()
            native.latent_absorb(a, self.is_f32)
            if not (self.is_f32 or self.plain_kernels) and native.latent_decode_takes(lat, pe):
                a.sink, a.scale, a.part_o, a.part_ml = t.sink.data_ptr(), m.scale, ws.flat["part_o"].data_ptr(), ws.flat["part_ml"].data_ptr()
                native.latent_decode(a)
                return out
            b.q, b.k, b.v, b.out, b.out_stride = a.qa, a.cache, a.cache, a.o_lat, m.heads * m.kv_rank
            b.G, b.dim, b.dimp, b.vdim, b.vdimp, b.decode = 1, lat + pe, lat + pe, m.kv_rank, lat + pe, 1
            native.chunk_attention(b, self.is_f32, plain=self.plain_kernels)
            native.latent_value(a, self.is_f32)
            return out
        native.latent_query(a, self.is_f32)
        keys = start + rows
        cached = state.latent[layer][lane, :keys]
        b.start, b.base, b.keys, b.dim, b.dimp, b.vdim, b.vdimp = start, 0, keys, m.dim + m.rot_dim, t.dimp, m.vdim, t.vdimp
        group = expand_heads(m, cache.context_capacity, cache.element_bytes)
        for h0 in range(0, m.heads, group):
            n = min(group, m.heads - h0)
            k, v = ws.view("keys", keys, n * t.dimp), ws.view("values", keys, n * t.vdimp)
            self._mm(cached, t.expand_k[h0 * t.dimp : (h0 + n) * t.dimp], k)
            self._mm(cached[:, :lat], t.expand_v[h0 * t.vdimp : (h0 + n) * t.vdimp], v)
            b.H = b.G = n
            b.q, b.q_stride, b.k, b.v = q.data_ptr() + h0 * t.dimp * q.element_size(), q.stride(0), k.data_ptr(), v.data_ptr()
            b.out, b.out_stride = out.data_ptr() + h0 * m.vdim * out.element_size(), out.stride(0)
            b.gate, b.gate_stride = proj.data_ptr() + (t.off_gate + h0) * proj.element_size(), proj.stride(0)
            b.sink = t.sink.data_ptr() + h0 * 4
            native.chunk_attention(b, self.is_f32, plain=self.plain_kernels)
        return out

    def _feed_forward(self, ws: ZikevikWorkspace, layer: int, rows: int) -> None:
        m, t = self.g.layers[layer].mlp, self.w.layers[layer].mlp
        h, update, F = ws.h[:rows], ws.update[:rows], t.ff_cols
        if not isinstance(m, RoutedSpec):
            act = ws.view("act", rows, F)
            if rows <= native.MAX_ROWS and not self.is_f32:
                native.skinny_bf16_swiglu(h, t.gate_up[:F], t.gate_up[F:], act)
            else:
                gate_up = ws.view("gate_up", rows, 2 * F)
                self._mm(h, t.gate_up, gate_up)
                native.glu_rows(gate_up[:, :F], gate_up[:, F:], act, native.GLU_SILU)
            self._mm(act, t.down, update)
            return
        routes = rows * m.top
        scores = ws.view("router", rows, t.router.shape[0])
        self._mm(h, t.router, scores)
        ids, weights = ws.route_ids[:routes].view(rows, m.top), ws.route_weights[:routes].view(rows, m.top)
        native.router_topk(scores[:, : m.experts], None, m.top, ids, weights, normalize=False)
        act = ws.view("act", routes, F)
        if rows <= native.MAX_ROWS or self.is_f32:
            native.expert_glu(h, ids, weights, t.gate_up, act, native.GLU_SILU, status=self.peer.status_ptr)
            native.expert_down(act, ids, t.down, update)
            return
        tiles, perm, place = ws.tiles[: routes // 128 + m.experts + 1], ws.perm[:routes], ws.place[:routes]
        native.route_sort128(ids, 0, m.experts, tiles, ws.n_tiles, perm)
        x, gate_up, y = ws.view("sorted", routes, self.width), ws.view("gate_up", routes, 2 * F), ws.view("expert_out", routes, self.width)
        native.gather_routes(h, perm, m.top, place, x)
        native.gemm_bf16_tc(x, t.gate_up, gate_up, experts=m.experts, tiles=tiles, n_tiles=ws.n_tiles, status=self.peer.status_ptr)
        native.glu_rows(gate_up[:, :F], gate_up[:, F:], act, native.GLU_SILU, scale=ws.route_weights, scale_at=perm)
        native.gemm_bf16_tc(act, t.down, y, experts=m.experts, tiles=tiles, n_tiles=ws.n_tiles, status=self.peer.status_ptr)
        native.route_combine(y, place, m.top, update)

    # ------------------------------------------------------------------------------ whole model
    def run_rows(self, ws: ZikevikWorkspace, state: HybridState, tokens: torch.Tensor, row_pos: torch.Tensor, row_lane: torch.Tensor, row_active,
                 rows: int, *, decode: bool, max_ctx: int, head_rows=None, head: str = "logits", lane_of_rows: int | None = None):
        """Push ``rows`` token rows through the decoder; in prefill they are the positions ``max_ctx - rows .. max_ctx - 1`` of one lane.

        ``head='logits'`` returns the fp32 logits of ``head_rows`` (a slice or an index tensor; ``None``: all rows); ``head='argmax'``
        (decode) leaves the packed best candidates in ``ws.local_best`` and returns ``None``; ``head='none'`` stops after the layers.
        """
        g, w = self.g, self.w
        start = 0 if decode else max_ctx - rows
        if not decode and not (0 <= start and max_ctx <= self.cache.context_capacity and lane_of_rows is not None and 0 <= lane_of_rows < self.cache.lanes):
            raise ValueError("prefill rows lie within the context of one lane")
        residual, update, h = ws.residual[:rows], ws.update[:rows], ws.h[:rows]

        def norm(weight, source: dict) -> None:
            native.parallel_norm(residual, g.hidden_size, weight, h, g.norm_eps, weight_offset=1.0, status=self.peer.status_ptr, **source)

        for i, lw in enumerate(w.layers):
            norm(lw.norm1, dict(tokens=tokens, table=w.embed, vocab=g.vocab_size, table_scale=g.embedding_scale) if i == 0 else dict(update=update))
            if isinstance(g.layers[i].mixer, DeltaSpec):
                mixed = self._delta(ws, state, i, rows, row_pos, row_lane, row_active, decode)
            else:
                mixed = self._latent(ws, state, i, rows, row_pos, row_lane, row_active, decode, start, lane_of_rows)
            self._mm(mixed, lw.mixer.out, update)
            if lw.mlp is not None:
                norm(lw.norm2, dict(update=update))
                self._feed_forward(ws, i, rows)
            if self.trace is not None:
                self.trace.setdefault("residual", {})[i] = (residual + update)[:, : g.hidden_size].clone()
        if head == "none":
            return None
        norm(w.final_norm, dict(update=update))
        x = h if head_rows is None else h[head_rows]
        if head == "argmax" and not self.is_f32:
            native.skinny_bf16(x, w.head, ws.local_best, native.SK_OUT_ARGMAX_F32, N=g.vocab_size, comm=self.peer.comm, channel=0, os_=0)
            return None
        logits = ws.logits if decode else torch.empty((x.shape[0], w.head.shape[0]), dtype=torch.float32, device=self.device)
        self._mm(x, w.head, logits[: x.shape[0]])
        return logits[: x.shape[0], : g.vocab_size]

    def sample(self, ws: ZikevikWorkspace, state: HybridState, logits, rows: int, row_active, *, advance: int, tokens_out=None, positions=None,
               out=None) -> None:
        """Greedy sampling (ties to the lowest id); the registers and the output ring are written as by the other families."""
        local_best = ws.local_best if logits is None else None
        if logits is not None:
            native.argmax_rows(logits, rows, self.g.vocab_size, 0, ws.cand, status=self.peer.status_ptr)
        counter, ring = (state.step_counter, RING) if out is None else (None, 1)
        native.step_finalize(ws.cand, 1, rows, row_active, state.tokens if tokens_out is None else tokens_out,
                             state.positions if positions is None else positions, state.out_tokens if out is None else out, counter, ring, advance,
                             local_best=local_best)
