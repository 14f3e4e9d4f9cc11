"""Namizen on a B200: every kernel alone against plain tensor operations, the model against the plain implementation in both number formats,
and the engine's own entry points.

The 32-bit path is held to a tight tolerance (no fault hides behind rounding there); the bf16 path to what bf16 operands give.  The weights
are made sharp (``sharp_checkpoint``): attention follows a few keys, wherever they are in the chunk."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from glm_tpu_b200.engine import request as rq
from glm_tpu_b200.engine.llm_engine import LLMEngine
from glm_tpu_b200.oracle import namizen as oracle
from tests.namizen_cases import attention, expected, geometries, row_errors, sharp_checkpoint, tokens_for

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
F32, BF16 = torch.float32, torch.bfloat16
LIMIT = {F32: 2e-5, BF16: 0.06}  # of the logits' root mean square
DEV = "cuda:0"


def runner_for(g, checkpoint, dtype=BF16, *, capacity=320, lanes=2, prefill_chunk=64, graphs=True):
    from glm_tpu_b200.runner.gpu_runner import build_runner

    return build_runner(g, device=DEV, checkpoint=checkpoint, context_capacity=capacity, lanes=lanes, prefill_chunk=prefill_chunk, dtype=dtype,
                        use_graphs=graphs)


def feed(runner, lane, tokens, cuts):
    """Run ``tokens`` on ``lane`` in portions ending at ``cuts``, single ones through the decode program; all logits."""
    runner.open_lane(lane)
    out, at = [], 0
    for cut in [*cuts, len(tokens)]:
        part = tokens[at:cut]
        if len(part) == 1 and at > 0:
            out.append(runner.decode_logits({lane: part[0]})[lane][None])
        elif part:
            out.append(runner.extend(lane, part, range(len(part))))
        at = cut
    return torch.cat(out)


def check(got, want, dtype, factor=1.0):
    errors = row_errors(got, want)
    worst = int(errors.argmax())
    assert torch.isfinite(got).all() and float(errors[worst]) < LIMIT[dtype] * factor, f"position {worst}: {float(errors[worst]):.3g}"


# ------------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [40, 100, 4104, 6000])
def test_parallel_norm(native_lib, dtype, width):
    native, pad = native_lib, (width + 7) // 8 * 8
    gen = torch.Generator().manual_seed(width)
    rows, vocab = 5, 11
    make = lambda *s: torch.nn.functional.pad(torch.randn(s, generator=gen), (0, pad - width)).to(DEV)  # noqa: E731
    table, w1, w2, update = make(vocab, width).to(dtype), make(width).to(dtype), make(width).to(dtype), make(rows, width)
    tokens = torch.tensor([3, 0, 10, 3, 7], dtype=torch.int32, device=DEV)
    residual = torch.full((rows, pad), 7.0, device=DEV)
    out1, out2 = torch.empty(rows, pad, dtype=dtype, device=DEV), torch.empty(rows, pad, dtype=dtype, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    native.parallel_norm(residual, width, w1, out1, 0.25, w2=w2, out2=out2, tokens=tokens, table=table, vocab=vocab, status=status)
    x = table.double()[tokens.long()]
    assert torch.equal(residual.double(), x)
    native.parallel_norm(residual, width, w1, out1, 0.25, w2=w2, out2=out2, update=update, status=status)
    x = x + update.double()
    for out, w in ((out1, w1), (out2, w2)):
        want = oracle.rms_norm(x[:, :width], w.double()[:width], 0.25)
        assert float(((out.double()[:, :width] - want).abs() / (1 + want.abs())).max()) < (1e-5 if dtype is F32 else 0.005) and not out[:, width:].any()
    assert float((residual.double() - x).abs().max()) < 1e-5 and int(status) == 0
    tokens[2] = vocab
    native.parallel_norm(residual, width, w1, out1, 0.25, tokens=tokens, table=table, vocab=vocab, status=status)
    assert int(status) == native.STATUS_BAD_INDEX


@pytest.mark.parametrize("rows,K,N,F", [(1, 104, 30, 0), (2, 512, 48, 24), (3, 1024, 7, 40), (8, 4096, 520, 264)])
def test_dual_projection(native_lib, rows, K, N, F):
    native = native_lib
    gen = torch.Generator().manual_seed(K)
    make = lambda *s: torch.randn(s, generator=gen).to(BF16).to(DEV)  # noqa: E731
    x1, x2, w, wg, wu = make(rows, K), make(rows, K), make(N, K) * K**-0.5, make(max(F, 1), K) * K**-0.5, make(max(F, 1), K) * K**-0.5
    out, act = torch.zeros(rows, N, dtype=BF16, device=DEV), torch.zeros(rows, F + 16, dtype=BF16, device=DEV)
    if F:
        native.dual_proj(x1, w, out, x2, wg, wu, act[:, 16:], native.GLU_GELU_TANH)
        want = oracle.gelu_tanh(x2.double() @ wg.double().T) * (x2.double() @ wu.double().T)
        assert float((act[:, 16:].double() - want).abs().max()) < 0.04 and not act[:, :16].any()
    else:
        native.dual_proj(x1, w, out)
    assert float((out.double() - x1.double() @ w.double().T).abs().max()) < 0.03


def test_gated_rows_and_plain_gemm(native_lib):
    native = native_lib
    x = torch.randn(37, 160, device=DEV)
    for dtype in (F32, BF16):
        both = x.to(dtype)
        out = torch.zeros(37, 96, dtype=dtype, device=DEV)
        native.glu_rows(both[:, :80], both[:, 80:], out[:, 16:], native.GLU_GELU_TANH)
        want = oracle.gelu_tanh(both[:, :80].double()) * both[:, 80:].double()
        assert float((out[:, 16:].double() - want).abs().max()) < (1e-5 if dtype is F32 else 0.05)
        native.glu_rows(both[:, :80], both[:, 80:], out[:, 16:], native.GLU_SILU)
        want = torch.nn.functional.silu(both[:, :80].double()) * both[:, 80:].double()
        assert float((out[:, 16:].double() - want).abs().max()) < (1e-5 if dtype is F32 else 0.05)
    for rows, N, K in ((1, 3, 5), (70, 129, 33), (8, 64, 200)):
        a, b, c = torch.randn(rows, K, device=DEV), torch.randn(N, K, device=DEV), torch.empty(rows, N, device=DEV)
        native.gemm_f32(a, b, c)
        assert float((c.double() - a.double() @ b.double().T).abs().max()) < 1e-4


CONV_SHAPES = [  # heads, key heads, dim, vdim, taps, rotated, chunk
    (4, 2, 32, 48, 4, 16, 24), (3, 1, 21, 13, 3, 10, 7), (2, 2, 128, 64, 2, 128, 40), (2, 1, 40, 40, 6, 24, 1000), (1, 1, 24, 8, 1, 0, 5), (2, 1, 320, 256, 4, 64, 33),
]


@pytest.mark.parametrize("shape", CONV_SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_convolution_rotation_mixing_and_caches(native_lib, shape, dtype):
    """One layer's q | k | v in portions of many sizes and in single decode steps: queries, keys and mixed values as they enter the
    attention, whatever the cuts; another lane's state is not touched."""
    native = native_lib
    H, G, dim, vdim, taps, rot, chunk = shape
    capacity, lanes, lane, total = 200, 3, 1, 150
    C, dp, vp = (H + G) * dim + G * vdim, (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    gen = torch.Generator().manual_seed(dim)
    u, w = torch.randn(total, C, generator=gen).to(dtype).to(DEV), torch.randn(C, taps, generator=gen)
    v_first = torch.randn(total, G * vdim, generator=gen).to(dtype).to(DEV)
    weights = w.T.contiguous().to(DEV)
    angle = torch.arange(capacity, dtype=torch.float64)[:, None] * 300.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))
    table = torch.stack([angle.cos(), angle.sin()], -1).float().contiguous().to(DEV)
    y = oracle.causal_conv(u.double().cpu(), w.double())
    want_q = oracle.rotate_half(y[:, : H * dim].reshape(total, H, dim), rot, 300.0)
    want_k = oracle.rotate_half(y[:, H * dim : (H + G) * dim].reshape(total, G, dim), rot, 300.0)
    own_v = y[:, (H + G) * dim :].reshape(total, G, vdim)
    want_v = oracle.mix_values(own_v, v_first.double().cpu().reshape(total, G, vdim), 0.25)
    ring = min(chunk, capacity)
    k_ring, v_ring = torch.full((lanes, ring, G, dp), 9.0, dtype=dtype, device=DEV), torch.full((lanes, ring, G, vp), 9.0, dtype=dtype, device=DEV)
    state = torch.full((lanes, taps - 1, C), 5.0, dtype=dtype, device=DEV)  # what an earlier request left
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    tol = 2e-5 if dtype is F32 else 0.06

    def step(at, rows, decode, mode, stored):
        pos = torch.arange(at, at + rows, dtype=torch.int32, device=DEV)
        lane_t, active = torch.full((rows,), lane, dtype=torch.int32, device=DEV), torch.ones(rows, dtype=torch.int32, device=DEV)
        proj = u[at : at + rows].contiguous()
        q = torch.full((rows, H, dp), 3.0, dtype=dtype, device=DEV)
        linear = not decode and rows > 20  # to linear buffers as well as to the ring
        k_lin, v_lin = torch.full((rows, G, dp), 3.0, dtype=dtype, device=DEV), torch.full((rows, G, vp), 3.0, dtype=dtype, device=DEV)
        vf = stored[at : at + rows].contiguous()
        a = native.QkvConvArgs()
        a.proj, a.proj_stride, a.conv_w, a.taps, a.state = proj.data_ptr(), C, weights.data_ptr(), taps, state.data_ptr()
        a.row_pos, a.row_lane, a.row_active = pos.data_ptr(), lane_t.data_ptr(), active.data_ptr()
        a.rot, a.rot_dims, a.q, a.ring = table.data_ptr(), rot, q.data_ptr(), ring
        a.k_ring, a.v_ring = k_ring.data_ptr(), v_ring.data_ptr()
        if linear:
            a.k_lin, a.v_lin = k_lin.data_ptr(), v_lin.data_ptr()
        a.v_first, a.v_mode, a.mix = vf.data_ptr(), mode, 0.25
        a.H, a.G, a.dim, a.dimp, a.vdim, a.vdimp = H, G, dim, dp, vdim, vp
        a.rows, a.decode, a.capacity, a.lanes, a.status = rows, int(decode), capacity, lanes, status.data_ptr()
        native.qkv_conv(a, dtype is F32)
        torch.cuda.synchronize()
        assert float((q[..., :dim].double().cpu() - want_q[at : at + rows]).abs().max()) < tol and not q[..., dim:].any()
        if linear:
            k, v = k_lin, v_lin
        else:
            keep = range(max(at, at + rows - ring), at + rows)
            k, v = k_ring[lane, [p % ring for p in keep]], v_ring[lane, [p % ring for p in keep]]
            at, rows = keep[0], len(keep)
        assert float((k[..., :dim].double().cpu() - want_k[at : at + rows]).abs().max()) < tol and not k[..., dim:].any()
        value = want_v if mode == 2 else own_v
        assert float((v[..., :vdim].double().cpu() - value[at : at + rows]).abs().max()) < tol and not v[..., vdim:].any()
        return vf

    at = 0
    for rows, decode in ((2, False), (1, True), (3, False), (45, False), (1, True), (1, True), (2, False), (9, False), (60, False), (1, True)):
        if rows > ring and rows <= 20:
            rows = ring
        step(at, rows, decode, 2, v_first)
        at += rows
    state.fill_(5.0)
    stored = step(0, 40, False, 1, torch.zeros(total, G * vdim, dtype=dtype, device=DEV))  # a new request on the lane; this layer's values are kept
    assert float((stored.double().cpu() - own_v[:40].reshape(40, -1)).abs().max()) < tol
    assert taps == 1 or ((state[0] == 5.0).all() and (state[2] == 5.0).all())
    assert (k_ring[0] == 9.0).all() and (v_ring[2] == 9.0).all() and int(status) == 0


def attention_case(H, G, dim, vdim, rows, start, chunk, seed=0, sharp=2.0):
    """Random q, k, v of a sequence up to ``start + rows`` and the expected outputs of the last ``rows`` positions (float64)."""
    total = start + rows
    gen = torch.Generator().manual_seed(seed)
    q = (torch.randn(total, H, dim, generator=gen) * sharp).to(BF16)
    k, v = torch.randn(total, G, dim, generator=gen).to(BF16), torch.randn(total, G, vdim, generator=gen).to(BF16)
    sink = torch.randn(H, generator=gen) + 1.0
    scale = dim**-0.5
    kk, vv = k.double().repeat_interleave(H // G, 1), v.double().repeat_interleave(H // G, 1)
    scores = torch.einsum("ihd,jhd->hij", q.double(), kk) * scale
    p = oracle.sink_softmax(scores, sink.double(), oracle.chunk_mask(total, chunk))
    out = torch.einsum("hij,jhd->ihd", p, vv)
    return q, k, v, sink, scale, out[start:].reshape(rows, -1)


def pad_heads(x, to):
    return torch.nn.functional.pad(x, (0, to - x.shape[-1])).contiguous().to(DEV)


def attention_args(native, q, k, v, sink, scale, out, H, G, dim, vdim, status):
    a = native.ChunkAttnArgs()
    a.q, a.k, a.v, a.sink = q.data_ptr(), k.data_ptr(), v.data_ptr(), sink.data_ptr() if sink is not None else None
    a.out, a.out_stride = out.data_ptr(), out.stride(0)
    a.H, a.G, a.dim, a.dimp, a.vdim, a.vdimp = H, G, dim, (dim + 15) // 16 * 16, vdim, (vdim + 15) // 16 * 16
    a.scale, a.status = scale, status.data_ptr()
    return a


PREFILL_SHAPES = [  # heads, key heads, dim, vdim, rows, start, chunk
    (2, 1, 128, 128, 300, 0, 1000), (4, 2, 64, 48, 257, 70, 128), (3, 3, 20, 12, 130, 5, 7), (2, 1, 96, 80, 500, 250, 300), (8, 1, 40, 128, 2, 127, 129),
    (2, 2, 16, 16, 128, 128, 128), (1, 1, 112, 64, 700, 31, 100000), (2, 1, 200, 256, 150, 33, 64), (2, 1, 136, 40, 70, 0, 50), (2, 1, 128, 112, 1, 255, 256),
    (2, 1, 32, 33, 256, 1, 1),
]


@pytest.mark.parametrize("shape", PREFILL_SHAPES)
@pytest.mark.parametrize("kernel", ["tc", "mma", "any"])
def test_prefill_attention(native_lib, shape, kernel):
    """Chunk borders inside and at the edges of tiles, rows that start anywhere, sinks, junk behind the last key."""
    native = native_lib
    H, G, dim, vdim, rows, start, chunk = shape
    q, k, v, sink, scale, want = attention_case(H, G, dim, vdim, rows, start, chunk, seed=rows)
    dp, vp = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    base = start // chunk * chunk
    junk = lambda t, to: torch.cat([pad_heads(t[base:], to), torch.full((200, t.shape[1], to), float("nan"), dtype=BF16, device=DEV)])  # noqa: E731
    qd, kd, vd = pad_heads(q[start:], dp), junk(k, dp), junk(v, vp)
    out = torch.full((rows, H * vdim + 8), 2.0, dtype=BF16, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    sink_d = sink.to(DEV)
    a = attention_args(native, qd, kd, vd, sink_d, scale, out, H, G, dim, vdim, status)
    a.rows, a.start, a.base, a.keys, a.chunk = rows, start, base, start + rows - base, chunk
    native.set_chunk_prefill_tc(1 if kernel == "tc" else 0)
    try:
        native.chunk_attention(a, False, plain=kernel == "any")
    finally:
        native.set_chunk_prefill_tc(1)
    torch.cuda.synchronize()
    assert int(status) == 0 and (out[:, H * vdim :] == 2.0).all()
    got = out[:, : H * vdim].double().cpu()
    assert torch.isfinite(got).all() and float((got - want).abs().max()) < 0.02, int((got - want).abs().max(1).values.argmax())
    a.keys -= 1  # a query whose own key is not in the buffer is refused on the host
    with pytest.raises(RuntimeError):
        native.chunk_attention(a, False)


def test_prefill_attention_without_a_sink_and_with_one_far_key(native_lib):
    """One key far back, at a chunk's first slot, carries the weight of a late query; the sink is optional."""
    native = native_lib
    H, G, dim, vdim, rows, chunk = 1, 1, 64, 64, 640, 640
    q, k, v, _, scale, _ = attention_case(H, G, dim, vdim, rows, 0, chunk, seed=5, sharp=0.2)
    q[600], k[0] = k[0] * 4, k[0] * 4  # only query 600 points at key 0
    scores = torch.einsum("ihd,jhd->hij", q.double(), k.double()) * scale
    p = oracle.sink_softmax(scores, torch.full((1,), -1e30, dtype=torch.float64), oracle.chunk_mask(rows, chunk))
    want = torch.einsum("hij,jhd->ihd", p, v.double()).reshape(rows, -1)
    assert float(p[0, 600, 0]) > 0.99
    for tc in (1, 0):
        out = torch.zeros(rows, vdim, dtype=BF16, device=DEV)
        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        qd, kd, vd = q.to(DEV), k.to(DEV), v.to(DEV)
        a = attention_args(native, qd, kd, vd, None, scale, out, H, G, dim, vdim, status)
        a.rows, a.start, a.base, a.keys, a.chunk = rows, 0, 0, rows, chunk
        native.set_chunk_prefill_tc(tc)
        native.chunk_attention(a, False)
        native.set_chunk_prefill_tc(1)
        torch.cuda.synchronize()
        assert int(status) == 0 and float((out.double().cpu() - want).abs().max()) < 0.02


DECODE_SHAPES = [  # heads, key heads, dim, vdim, chunk, capacity
    (8, 2, 128, 128, 700, 1024), (20, 1, 48, 64, 64, 512), (3, 3, 20, 12, 7, 256), (4, 1, 200, 256, 130, 512), (2, 1, 96, 80, 4096, 2048), (6, 2, 36, 44, 1, 64),
]


@pytest.mark.parametrize("shape", DECODE_SHAPES)
@pytest.mark.parametrize("plain", [False, True])
def test_decode_attention(native_lib, shape, plain):
    """One row per lane at unequal positions, just before, at and after chunk borders; NaN in every ring row the rows must not see; an
    inactive lane gives zeros."""
    native = native_lib
    H, G, dim, vdim, chunk, capacity = shape
    chunk = min(chunk, capacity)
    ring, lanes = chunk, 6
    dp, vp = (dim + 15) // 16 * 16, (vdim + 15) // 16 * 16
    positions = [0, min(chunk - 1, capacity - 1), min(chunk, capacity - 1), capacity - 1, chunk // 2, 3]
    k_ring = torch.full((lanes, ring, G, dp), float("nan"), dtype=BF16, device=DEV)
    v_ring = torch.full((lanes, ring, G, vp), float("nan"), dtype=BF16, device=DEV)
    rows, wants = [], []
    sink = None
    for lane, pos in enumerate(positions):
        first = pos // chunk * chunk
        n = pos - first + 1
        q, k, v, s, scale, want = attention_case(H, G, dim, vdim, 1, n - 1, n, seed=lane)
        sink = s if sink is None else sink
        p = oracle.sink_softmax(torch.einsum("ihd,jhd->hij", q.double()[-1:], k.double().repeat_interleave(H // G, 1)) * scale, sink.double(),
                                torch.ones(1, n, dtype=torch.bool))
        wants.append(torch.einsum("hij,jhd->ihd", p, v.double().repeat_interleave(H // G, 1)).reshape(1, -1))
        k_ring[lane, :n], v_ring[lane, :n] = pad_heads(k, dp), pad_heads(v, vp)
        rows.append(q[-1:])
    qd = pad_heads(torch.cat(rows), dp)
    out = torch.full((lanes, H * vdim), 2.0, dtype=BF16, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    pos_t = torch.tensor(positions, dtype=torch.int32, device=DEV)
    lane_t = torch.arange(lanes, dtype=torch.int32, device=DEV)
    active = torch.tensor([1, 1, 1, 1, 0, 1], dtype=torch.int32, device=DEV)
    sink_d = sink.to(DEV)
    a = attention_args(native, qd, k_ring, v_ring, sink_d, scale, out, H, G, dim, vdim, status)
    a.row_pos, a.row_lane, a.row_active = pos_t.data_ptr(), lane_t.data_ptr(), active.data_ptr()
    a.rows, a.decode, a.chunk, a.ring, a.capacity, a.lanes = lanes, 1, chunk, ring, capacity, lanes
    native.chunk_attention(a, False, plain=plain)
    torch.cuda.synchronize()
    got = out.double().cpu()
    assert int(status) == 0 and torch.isfinite(got).all() and not got[4].any()
    for lane, want in enumerate(wants):
        if lane != 4:
            assert float((got[lane] - want[0]).abs().max()) < 0.02, (lane, positions[lane])


# ------------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("name", sorted(geometries()))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prefill_portions_and_decoding_agree_with_the_plain_model(native_lib, name, dtype):
    """Whole prompts, prompts in portions of many sizes (two tokens among them, cut at and around chunk borders), token-by-token decoding:
    the logits of every position."""
    g = geometries()[name]
    ck, total = sharp_checkpoint(g, 1), 210
    tokens = tokens_for(g, total, 1)
    want = expected(g, ck, tokens)
    runner = runner_for(g, ck, dtype)
    try:
        whole = feed(runner, 0, tokens, [])
        check(whole, want, dtype)
        for lane, cuts in ((1, list(range(1, total))),                                   # one first token, then decoding only
                           (0, [2, 4, 7, 8, 40, 42, 95, 96, 97, 99, 130, 131, 133, 190, 192]),
                           (1, list(range(2, total, 2))),                                # portions of two tokens
                           (0, [150] + list(range(151, total)))):                        # a prompt, then a long decoding
            got = feed(runner, lane, tokens, cuts)
            check(got, want, dtype)
            assert float(row_errors(got, whole).max()) < LIMIT[dtype]
    finally:
        runner.close()


@pytest.mark.parametrize("name", ["tiny", "tiles", "wide"])
def test_layer_by_layer_in_32_bits(native_lib, name):
    g = geometries()[name]
    ck, tokens = sharp_checkpoint(g, 2), tokens_for(g, 60, 2)
    layers: list = []
    expected(g, ck, tokens, layers_out=layers)
    runner = runner_for(g, ck, F32)
    try:
        runner.model.trace = {}
        runner.open_lane(0)
        runner.extend(0, tokens, [59])
        for i, want in enumerate(layers):
            got = runner.model.trace["residual"][i].double().cpu()
            assert float((got - want).abs().max()) < 1e-4 * float(want.abs().max()), i
    finally:
        runner.close()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_lanes_do_not_see_each_other_and_are_used_again(native_lib, dtype):
    """Unequal requests decoding together against each alone; lanes given back with their rings full, then used for other requests."""
    g = geometries()["tiny"]
    ck = sharp_checkpoint(g, 3)
    lengths = [1, 40, 97, 150]
    seqs = [tokens_for(g, n + 30, 10 + n) for n in lengths]
    wants = [expected(g, ck, s) for s in seqs]
    runner = runner_for(g, ck, dtype, lanes=4)
    try:
        for turn in range(2):
            order = list(range(4)) if turn == 0 else [2, 0, 3, 1]  # request order[lane] runs on `lane`; the second time over what the first left
            for lane, r in enumerate(order):
                runner.open_lane(lane)
                runner.extend(lane, seqs[r][: lengths[r]], [])
            for step in range(30):
                live = [lane for lane, r in enumerate(order) if step < 30 - 7 * r]  # lanes stop at different times
                if not live:
                    break
                got = runner.decode_logits({lane: seqs[order[lane]][lengths[order[lane]] + step] for lane in live})
                for lane in live:
                    r = order[lane]
                    check(got[lane][None], wants[r][lengths[r] + step][None], dtype)
    finally:
        runner.close()


def test_rows_of_a_batch_have_the_bits_of_the_same_rows_in_another(native_lib):
    """bf16: what else is in the batch, and which lane a request sits on, changes nothing at all in its decode logits."""
    g = geometries()["tiles"]
    ck, a, b = sharp_checkpoint(g, 4), tokens_for(g, 90, 4), tokens_for(g, 33, 5)
    results = []
    for lane_a, lane_b in ((0, 1), (3, 0), (2, None)):
        runner = runner_for(g, ck, BF16, lanes=4)
        runner.open_lane(lane_a)
        runner.extend(lane_a, a[:80], [])
        if lane_b is not None:
            runner.open_lane(lane_b)
            runner.extend(lane_b, b[:23], [])
        rows = []
        for i in range(10):
            feeds = {lane_a: a[80 + i]} | ({lane_b: b[23 + i]} if lane_b is not None else {})
            rows.append(runner.decode_logits(feeds)[lane_a])
        results.append(torch.stack(rows))
        runner.close()
    assert torch.equal(results[0], results[1]) and torch.equal(results[0], results[2])


def test_long_context_far_keys_and_long_decoding(native_lib):
    """A chunk of hundreds of tokens whose last queries look for its first keys, in a prompt and in decoding, then across its end."""
    from glm_tpu_b200.config.namizen import LayerSpec, NamizenGeometry

    g = NamizenGeometry(vocab_size=384, hidden_size=128, norm_eps=1e-5, layers=(
        LayerSpec(attention(4, 1, 64, 64, 3, 16, 1e6, 600, True), 192), LayerSpec(attention(4, 2, 64, 32, 3, 16, 1e6, 450, True), 160)))
    ck = sharp_checkpoint(g, 6, factor=4.0)
    tokens = tokens_for(g, 1250, 6)
    for at, back in ((598, 1), (599, 0), (601, 600), (899, 450), (1199, 601)):  # repeated tokens far back: like attracts like
        tokens[at] = tokens[back]
    want = expected(g, ck, tokens, dtype=torch.float64)
    for dtype in (F32, BF16):
        runner = runner_for(g, ck, dtype, capacity=1280, lanes=1, prefill_chunk=512)
        try:
            check(feed(runner, 0, tokens, []), want, dtype)
            check(feed(runner, 0, tokens, [560] + list(range(561, 640)) + [860] + list(range(861, 920)) + [1190] + list(range(1191, 1250))), want, dtype)
        finally:
            runner.close()


def test_a_failed_position_is_reported_and_refused(native_lib):
    g = geometries()["tiny"]
    runner = runner_for(g, sharp_checkpoint(g, 7), BF16, capacity=64, lanes=1)
    try:
        runner.open_lane(0)
        runner.extend(0, tokens_for(g, 60), [])
        with pytest.raises(ValueError):
            runner.extend(0, tokens_for(g, 5), [])
        for t in tokens_for(g, 4):
            runner.decode_logits({0: t})
        with pytest.raises(ValueError):
            runner.decode_logits({0: 1})
        with pytest.raises(ValueError):
            runner.extend(0, [1], [1])
    finally:
        runner.close()


def test_a_lane_filled_to_the_last_position_does_not_disturb_the_others(native_lib):
    g = geometries()["tiny"]
    ck = sharp_checkpoint(g, 11)
    full, other = tokens_for(g, 64, 1), tokens_for(g, 12, 2)
    runner = runner_for(g, ck, F32, capacity=64, lanes=2)
    try:
        check(feed(runner, 0, full, [50] + list(range(51, 64))), expected(g, ck, full), F32)
        check(feed(runner, 1, other, [5] + list(range(6, 12))), expected(g, ck, other), F32)
    finally:
        runner.close()


# ------------------------------------------------------------------------------------------------ the engine's own entry points
def near_greedy(g, ck, prompt, tokens, slack):
    """Every generated token is the plain model's best, or within ``slack`` (of the logits' spread) of it."""
    logits = expected(g, ck, list(prompt) + list(tokens))[len(prompt) - 1 : -1]
    best, spread = logits.amax(-1), logits.std(-1)
    chosen = logits[torch.arange(len(tokens)), torch.as_tensor(tokens)]
    return bool(((best - chosen) <= slack * spread).all())


@pytest.mark.parametrize("dtype,slack", [(F32, 1e-4), (BF16, 0.15)])
@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation_through_the_engine(native_lib, dtype, slack, graphs):
    from glm_tpu_b200.worker.gpu_worker import profile_for

    g = geometries()["tiny"]
    ck = sharp_checkpoint(g, 8)
    profile = profile_for(g, 256)
    runner = runner_for(g, ck, dtype, capacity=256, lanes=4, graphs=graphs)
    try:
        rec = runner.build_decode_program()
        assert rec.kind == ("cuda_graph" if graphs else "eager") and rec.launches > 0
        engine = LLMEngine(runner, profile=profile)
        prompts = [tokens_for(g, n, 20 + n) for n in (1, 30, 70, 140)]
        requests = [rq.from_token_ids(p, request_id=f"r{i}", max_new_tokens=20 + 10 * i, context_capacity=256, profile=profile) for i, p in enumerate(prompts)]
        events: list = []
        alone = []
        for r, p in zip(requests, prompts):
            events.clear()
            report = engine.generate(r, events.append)
            alone.append([e.token_id for e in events])
            assert report["emitted"] == len(alone[-1]) and near_greedy(g, ck, p, alone[-1], slack)
        events.clear()
        engine.generate_concurrent(rq.batch(requests, concurrent=True, profile=profile), events.append)
        for i, p in enumerate(prompts):
            together = [e.token_id for e in events if e.request_id == f"r{i}"]
            assert together == alone[i]
    finally:
        runner.close()


def test_replay_program(native_lib, tmp_path):
    """``bin/trace_run`` on a directory, in both number formats, with interleaved requests."""
    from glm_tpu_b200.model_loader.sharded_state import format as fmt

    g = geometries()["odd"]
    ck = sharp_checkpoint(g, 9)
    model = tmp_path / "model"
    model.mkdir()
    (model / "config.json").write_text(json.dumps(g.to_config()))
    fmt.write_file(model / "model.safetensors", ck, {})
    a, b = tokens_for(g, 40, 30), tokens_for(g, 12, 31)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": [11]}, {"id": "a", "tokens": a[33:34], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[34:], "want": [5]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b[:2], "want": [0, 1]}], "end": ["c"]}]
    la, lb = expected(g, ck, a), expected(g, ck, b)
    want = {0: la[[0, 32]], 1: torch.stack([lb[11], la[33]]), 2: la[[39]], 3: lb[[0, 1]]}
    for dtype, name in ((BF16, "bfloat16"), (F32, "float32")):
        out = tmp_path / name
        out.mkdir()
        done = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(model), "--dtype", name, "--out", str(out), "--max-tokens", "52"],
                              input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert done.returncode == 0 and done.stdout.split() == "done 0 done 1 done 2 done 3".split(), done.stderr[-2000:]
        for n, rows in want.items():
            got = torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(-1, g.vocab_size)
            check(got, rows, dtype)


def test_glm_lanes_take_given_tokens_too(native_lib):
    """The shared part of the runner: portions and single tokens of given ids give the GLM family the logits of the whole prompt."""
    from glm_tpu_b200.config.model import tiny_geometry
    from glm_tpu_b200.entrypoints.cli.trace import TraceReplay
    from glm_tpu_b200.models.glm_moe_dsa.weights import random_checkpoint
    from glm_tpu_b200.runner.gpu_runner import build_runner

    g = tiny_geometry()
    runner = build_runner(g, checkpoint=random_checkpoint(g, seed=0), device=DEV, context_capacity=64, stripe=8, prefill_chunk=32, lanes=2)
    try:
        tokens = tokens_for(g, 12, 1)
        session = TraceReplay(runner)
        whole = torch.stack(session.step({"step": 0, "entries": [{"id": "a", "tokens": tokens, "want": list(range(12))}], "end": ["a"]}))
        rows = session.step({"step": 1, "entries": [{"id": "b", "tokens": tokens[:9], "want": [8]}], "end": []})
        for t in tokens[9:]:
            rows += session.step({"step": 2, "entries": [{"id": "b", "tokens": [t], "want": [0]}], "end": []})
        assert float(row_errors(torch.stack(rows), whole[8:]).max()) < 0.1
    finally:
        runner.close()


def test_component_library_holds_what_the_family_launches(native_lib, tmp_path):
    """The family's own library, built alone and loaded in a fresh process, runs a prompt and a decode step."""
    code = """
import sys
from pathlib import Path
from glm_tpu_b200.csrc import build as b
from glm_tpu_b200.ops import native
b.LIB = Path(sys.argv[1]) / "never_there.so"
b.OUT_DIR = Path(sys.argv[1])
native.select_library(b.build(component="namizen"))
from tests.namizen_cases import geometries, sharp_checkpoint, tokens_for
from glm_tpu_b200.runner.gpu_runner import build_runner
g = geometries()["tiles"]
r = build_runner(g, device="cuda:0", checkpoint=sharp_checkpoint(g), context_capacity=128, prefill_chunk=64)
first = r.prefill(0, tokens_for(g, 70))
r.build_decode_program(); r.decode_step()
print("tokens", first, r.read_last_tokens()[0], native.LIB_PATH.name)
r.close()
"""
    done = subprocess.run([sys.executable, "-c", code, str(tmp_path)], capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert done.returncode == 0 and done.stdout.startswith("tokens") and "libglmb200_namizen.so" in done.stdout, done.stderr[-2000:]

