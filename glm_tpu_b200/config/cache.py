"""Cache configuration and the numerical contracts of attention, the DSA indexer and the MoE.

The KV cache holds one row per position and layer: ``[latent (kv_lora_rank) | rotated RoPE key]`` in
bf16 (no padding column: a 1152-byte row is already 16-byte aligned for vector and TMA access).  The
index cache holds one bf16 key of ``index_head_dim`` per position for every *full* indexer layer.

Both caches are striped by position over the ``world`` GPUs of the box: positions are cut into stripes
of ``stripe`` rows, stripe ``s`` belongs to GPU ``s % world``, and a GPU stores its stripes back to back.
A page is ``stripe * world`` positions, so with 8 GPUs and 64-row stripes the layout is the 512-position
page of the reference (``glm_tpu/config/cache.py:67-95``, owner ``(pos % 512) // 64``).

Parity: reference ``glm_tpu/config/cache.py:21-64`` (MLA contract), ``:98-143`` (DSA contract),
``:221-367`` (``CacheConfig``).
"""

from __future__ import annotations

from dataclasses import dataclass, field

from glm_tpu_b200.config.model import ModelGeometry
from glm_tpu_b200.exceptions import PlanValidationError

CAPACITY_PROFILES = (8192, 32768, 166912, 262144)


@dataclass(frozen=True)
class MlaNumericalContract:
    """Absorbed multi-head latent attention arithmetic.

    Scores are fp32 ``(q_c . latent + q_rope . k_rope) * qk_head_dim**-0.5``; softmax statistics are fp32;
    the unnormalized probability is rounded to bf16 before it multiplies the latent; the result is
    normalized once at the end and rounded to bf16.  A row with no valid key yields zeros.
    """

    score_dtype: str = "float32"
    probability_rounding: str = "unnormalized_bf16_before_pv"
    position_order: str = "ascending_global_position"
    empty_row: str = "zeros"


@dataclass(frozen=True)
class DsaNumericalContract:
    """Lightning-indexer arithmetic and the top-k order.

    ``score = sum_h w_h * relu(q_h . k * index_head_dim**-0.5)`` in fp32 with ``w = (x @ weights_proj.T) *
    index_heads**-0.5``.  Selection is by descending score, ties to the lowest position, under the total
    fp32 order in which ``+0 > -0``; positions at or beyond the context length never win; the tail of a
    short selection is ``-1``; the selected list is returned in ascending position order.
    """

    tie_policy: str = "descending_score_then_lowest_position"
    sentinel: int = -1
    key_norm_eps: float = 1e-6
    nonfinite_score: str = "health_false"


@dataclass(frozen=True)
class MoeNumericalContract:
    """Router and expert arithmetic.

    Router logits, sigmoid and weights are fp32; the correction bias enters the choice only; ties go to the
    lowest expert id; weights are ``s / (sum s + 1e-20)``.  Expert gate/up accumulate in fp32 and round to
    bf16; ``act = bf16(silu(g) * u)`` from the rounded values; the down output rounds to bf16 and is scaled by
    the bf16 route weight; routes are summed in fp32; ``out = bf16(bf16(routed * scale) + shared)``.
    """

    router_dtype: str = "float32"
    route_sum_dtype: str = "float32"
    weight_decode: str = "bf16(f32(e4m3)*scale_inv)"


@dataclass(frozen=True)
class CacheConfig:
    geometry: ModelGeometry
    context_capacity: int
    world: int = 1
    stripe: int = 64
    lanes: int = 1
    mla: MlaNumericalContract = field(default_factory=MlaNumericalContract)
    dsa: DsaNumericalContract = field(default_factory=DsaNumericalContract)
    moe: MoeNumericalContract = field(default_factory=MoeNumericalContract)

    def __post_init__(self) -> None:
        if self.world < 1 or self.stripe < 1 or self.lanes < 1:
            raise PlanValidationError("world, stripe and lanes must be positive")
        if self.lanes > 8:
            raise PlanValidationError("at most 8 concurrent lanes are supported")
        if self.context_capacity % self.page:
            raise PlanValidationError(f"context capacity {self.context_capacity} is not a multiple of the page ({self.page})")

    @property
    def page(self) -> int:
        return self.stripe * self.world

    @property
    def local_capacity(self) -> int:
        return self.context_capacity // self.world

    def owner(self, position: int) -> int:
        return (position // self.stripe) % self.world

    def local_row(self, position: int) -> int:
        return (position // self.page) * self.stripe + position % self.stripe

    def global_position(self, rank: int, local_row: int) -> int:
        return (local_row // self.stripe) * self.page + rank * self.stripe + local_row % self.stripe

    def owned_count(self, rank: int, context_length: int) -> int:
        """How many of the positions ``0..context_length-1`` are stored on ``rank``."""
        full_pages, rest = divmod(context_length, self.page)
        extra = min(max(rest - rank * self.stripe, 0), self.stripe)
        return full_pages * self.stripe + extra

    @property
    def kv_cache_shape(self) -> tuple[int, int, int, int]:
        g = self.geometry
        return (self.lanes, g.num_layers, self.local_capacity, g.kv_row_width)

    @property
    def index_cache_shape(self) -> tuple[int, int, int, int]:
        g = self.geometry
        return (self.lanes, len(g.full_layers), self.local_capacity, g.index_head_dim)

    def cache_bytes_per_gpu(self) -> int:
        kv = 1
        for n in self.kv_cache_shape:
            kv *= n
        ix = 1
        for n in self.index_cache_shape:
            ix *= n
        return 2 * (kv + ix)


@dataclass(frozen=True)
class RingCacheConfig:
    """Caches of a model whose layers see a bounded stretch of the sequence, one GPU.

    Every layer has its own ring of key and value rows per lane: position ``p`` lives in slot ``p % ring(layer)``.  A layer that attends
    inside chunks of ``chunk`` positions needs the rows of the current chunk only, so its ring has ``min(chunk, capacity)`` slots whatever
    the context capacity; a layer that sees the whole sequence has one slot per position.  A layer with a short convolution over time also
    keeps the last ``taps - 1`` projected rows of every lane.  Head rows are padded to a multiple of 16 elements (whole tensor-core
    steps, 16-byte vectors).

    ``geometry.layers[i].mixer`` gives a layer's ``kv_heads``, ``dim``, ``vdim``, ``chunk``, ``conv`` and ``qkv_width``.
    """

    geometry: object
    context_capacity: int
    lanes: int = 1
    element_bytes: int = 2
    page: int = 1

    def __post_init__(self) -> None:
        if self.context_capacity < 1 or not 1 <= self.lanes <= 8:
            raise PlanValidationError("the context capacity must be positive and the lanes between 1 and 8")

    def _mixer(self, layer: int):
        return self.geometry.layers[layer].mixer

    def ring(self, layer: int) -> int:
        chunk = self._mixer(layer).chunk
        return self.context_capacity if chunk is None else min(chunk, self.context_capacity)

    def chunk(self, layer: int) -> int:
        """Chunk length in positions (a chunk that nothing ends within the capacity is the capacity)."""
        chunk = self._mixer(layer).chunk
        return self.context_capacity if chunk is None else min(chunk, self.context_capacity)

    def first_position(self, layer: int, position: int) -> int:
        """The first position that ``position`` can see."""
        return position // self.chunk(layer) * self.chunk(layer)

    def crossing(self, layer: int, start: int, rows: int) -> tuple[int, int] | None:
        """``None`` if the rows ``start .. start + rows - 1`` of a step lie in one chunk: they enter the ring right away and the ring then
        holds every key they see, in order.  Otherwise ``(before, after)``: the ring's first ``before`` rows (the beginning of the first
        row's chunk) are still needed by the step, and its last ``after`` rows (the last row's chunk) take their places afterwards."""
        first, last = self.first_position(layer, start), self.first_position(layer, start + rows - 1)
        return None if first == last else (start - first, start + rows - last)

    def linear_rows(self, layer: int, rows: int) -> int:
        """Rows of the linear key / value buffer a step of up to ``rows`` rows may need (0: its chunk is never crossed)."""
        return 0 if self.chunk(layer) >= self.context_capacity else self.chunk(layer) - 1 + rows

    def k_shape(self, layer: int) -> tuple[int, int, int, int]:
        m = self._mixer(layer)
        return (self.lanes, self.ring(layer), m.kv_heads, -(-m.dim // 16) * 16)

    def v_shape(self, layer: int) -> tuple[int, int, int, int]:
        m = self._mixer(layer)
        return (self.lanes, self.ring(layer), m.kv_heads, -(-m.vdim // 16) * 16)

    def conv_shape(self, layer: int) -> tuple[int, int, int]:
        m = self._mixer(layer)
        return (self.lanes, m.conv - 1, m.qkv_width)

    def cache_bytes_per_gpu(self) -> int:
        total = 0
        for layer in range(len(self.geometry.layers)):
            for shape in (self.k_shape(layer), self.v_shape(layer), self.conv_shape(layer)):
                count = 1
                for n in shape:
                    count *= n
                total += count * self.element_bytes
        return total


@dataclass(frozen=True)
class HybridCacheConfig:
    """Caches of a model whose layers are recurrent or attend over a shared latent, one GPU.

    A latent layer keeps one row per position and lane, ``[normalized latent | rotated key part]``, both parts padded to a multiple of 16
    elements (whole tensor-core steps, 16-byte vectors).  A recurrent layer keeps, per lane and whatever the context, an fp32 state per head
    (stored ``[vdim, dim]``: a value channel's row of key channels, padded to a multiple of 32) and a ring of the last ``taps`` projected
    rows for its convolution.

    ``geometry.layers[i].mixer`` gives the layer's sizes; a recurrent mixer has ``conv_width``, a latent one ``kv_rank``.
    """

    geometry: object
    context_capacity: int
    lanes: int = 1
    element_bytes: int = 2
    page: int = 1

    def __post_init__(self) -> None:
        if self.context_capacity < 1 or not 1 <= self.lanes <= 8:
            raise PlanValidationError("the context capacity must be positive and the lanes between 1 and 8")

    def _mixer(self, layer: int):
        return self.geometry.layers[layer].mixer

    def is_latent(self, layer: int) -> bool:
        return hasattr(self._mixer(layer), "kv_rank")

    def latent_columns(self, layer: int) -> tuple[int, int]:
        """Padded columns of the latent and of the rotated key part."""
        m = self._mixer(layer)
        return (-(-m.kv_rank // 16) * 16, -(-m.rot_dim // 16) * 16)

    def latent_shape(self, layer: int) -> tuple[int, int, int]:
        return (self.lanes, self.context_capacity, sum(self.latent_columns(layer)))

    def state_shape(self, layer: int) -> tuple[int, int, int, int]:
        m = self._mixer(layer)
        return (self.lanes, m.heads, m.vdim, -(-m.dim // 32) * 32)

    def conv_shape(self, layer: int) -> tuple[int, int, int]:
        m = self._mixer(layer)
        return (self.lanes, m.conv, m.conv_width)

    def layer_bytes(self, layer: int) -> int:
        def count(shape):
            n = 1
            for x in shape:
                n *= x
            return n

        if self.is_latent(layer):
            return count(self.latent_shape(layer)) * self.element_bytes
        return count(self.state_shape(layer)) * 4 + count(self.conv_shape(layer)) * self.element_bytes

    def cache_bytes_per_gpu(self) -> int:
        return sum(self.layer_bytes(i) for i in range(len(self.geometry.layers)))
