"""Zikevik on a B200: every kernel alone against plain tensor operations, the model against the plain implementation in both number formats,
and the engine's own entry points.

The 32-bit path is held to a tight tolerance (no fault hides behind rounding there); the bf16 path to what bf16 operands give.  The weights
are made sharp (``sharp_checkpoint``): attention follows a few keys, wherever they are, and parts of the recurrent state never fade."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from glm_tpu_b200.engine import request as rq
from glm_tpu_b200.engine.llm_engine import LLMEngine
from glm_tpu_b200.oracle import zikevik as oracle
from tests.zikevik_cases import delta, expected, geometries, latent, row_errors, settled_tokens, sharp_checkpoint, tokens_for

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
F32, BF16 = torch.float32, torch.bfloat16
LIMIT = {F32: 1e-4, BF16: 0.08}  # of the logits' root mean square
DEV = "cuda:0"


def runner_for(g, checkpoint, dtype=BF16, *, capacity=320, lanes=2, prefill_chunk=64, graphs=True, plain=False):
    from glm_tpu_b200.runner.gpu_runner import build_runner

    runner = build_runner(g, device=DEV, checkpoint=checkpoint, context_capacity=capacity, lanes=lanes, prefill_chunk=prefill_chunk, dtype=dtype,
                          use_graphs=graphs)
    runner.model.plain_kernels = plain
    return runner


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


def close(got, want, tolerance):
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.isfinite(got).all()
    worst = float(((got - want).abs() / (want.abs() + want.abs().mean())).max())
    assert worst < tolerance, worst


# ------------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_norm_weights_around_zero_and_scaled_embedding(native_lib, dtype):
    native, width, pad, rows, vocab = native_lib, 100, 104, 3, 7
    gen = torch.Generator().manual_seed(0)
    make = lambda *s: torch.nn.functional.pad(torch.randn(s, generator=gen), (0, pad - width)).to(DEV)  # noqa: E731
    table, w = make(vocab, width).to(dtype), (make(width) * 0.1).to(dtype)
    tokens = torch.tensor([6, 0, 3], dtype=torch.int32, device=DEV)
    residual, out = torch.full((rows, pad), 5.0, device=DEV), torch.empty(rows, pad, dtype=dtype, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    native.parallel_norm(residual, width, w, out, 0.1, tokens=tokens, table=table, vocab=vocab, table_scale=12.5, weight_offset=1.0, status=status)
    x = table.double()[tokens.long()] * 12.5
    close(residual, x, 1e-6)
    close(out[:, :width], oracle.zero_centred_norm(x[:, :width], w.double()[:width], 0.1), 1e-5 if dtype is F32 else 0.006)
    assert int(status) == 0 and not out[:, width:].any()


def delta_case(m, rows, seed):
    """Projection rows and everything else a delta-rule mixer's kernels read, on the CPU in fp64 (bf16 values where the engine keeps bf16)."""
    gen = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(s, generator=gen).double()  # noqa: E731
    C = m.conv_width
    case = {"x": r(rows, C).to(BF16).double(), "conv": (0.4 * r(C, m.conv)).to(BF16).double(), "b": r(rows, m.heads).to(BF16).double(),
            "a": (2 * r(rows, m.heads * m.dim)).float().double(), "a_log": 0.8 * r(m.heads), "bias": -4 + 4 * r(m.heads * m.dim), "norm": 1 + 0.1 * r(m.vdim),
            "gate": r(rows, m.v_width).to(BF16).double()}
    case["conv"][:, -1] += 0.8
    return case


def delta_expected(m, c, eps):
    """The mixer between its projections, from the plain statement's pieces; the state too."""
    T = c["x"].shape[0]
    y = oracle.silu(oracle.causal_conv(c["x"], c["conv"]))
    q, k, v = y[:, : m.k_width], y[:, m.k_width : 2 * m.k_width], y[:, 2 * m.k_width :]
    per = m.heads // m.kv_heads
    q, k = (oracle.unit(t.reshape(T, m.kv_heads, m.dim)).repeat_interleave(per, 1) for t in (q, k))
    decay = torch.exp(-torch.exp(c["a_log"])[:, None] * oracle.softplus(c["a"] + c["bias"]).reshape(T, m.heads, m.dim))
    o, state = oracle.delta_rule(q * m.dim**-0.5, k, v.reshape(T, m.heads, m.vdim), torch.sigmoid(c["b"]), decay)
    out = oracle.rms_norm(o, c["norm"], eps) * torch.sigmoid(c["gate"]).reshape(T, m.heads, m.vdim)
    return out.reshape(T, -1), o, state


class DeltaHarness:
    """Device buffers of one delta-rule layer for some lanes; ``run`` pushes rows of a case through the kernels."""

    def __init__(self, native, m, dtype, lanes, capacity=4096, eps=1e-3):
        self.native, self.m, self.dtype, self.lanes, self.capacity, self.eps = native, m, dtype, lanes, capacity, eps
        self.dimp = -(-m.dim // 32) * 32
        self.state = torch.full((lanes, m.heads, m.vdim, self.dimp), float("nan"), device=DEV)  # a fresh sequence must not see any of it
        self.ring = torch.full((lanes, m.conv, m.conv_width), float("nan"), dtype=dtype, device=DEV)
        self.status = torch.zeros(1, dtype=torch.int32, device=DEV)
        from glm_tpu_b200.models.zikevik.model import delta_record_bytes

        assert native.delta_chunk_record(m.dim, m.vdim, m.conv) == delta_record_bytes(m)
        self.records = torch.empty(3 * m.heads * max(delta_record_bytes(m), 4) // 4, device=DEV)  # three chunks at a time

    def run(self, c, sl, positions, lanes, *, decode, chunked=False, fused=False, active=None):
        native, m, T = self.native, self.m, self.dtype
        rows = len(range(*sl.indices(c["x"].shape[0]))) if isinstance(sl, slice) else len(sl)
        off_b = (m.conv_width + 7) // 8 * 8
        proj = torch.full((rows, off_b + (m.heads + 7) // 8 * 8 + 8), 3.0, dtype=T, device=DEV)
        proj[:, : m.conv_width], proj[:, off_b : off_b + m.heads] = c["x"][sl].to(T), c["b"][sl].to(T)
        t = lambda x, d=F32: x.to(d).contiguous().to(DEV)  # noqa: E731
        keep = dict(proj=proj, conv=t(c["conv"].T), a=t(c["a"][sl]), rate=t(c["a_log"].exp()), bias=t(c["bias"]), norm=t(c["norm"]), gate=t(c["gate"][sl], T),
                    pos=t(torch.as_tensor(positions), torch.int32), lane=t(torch.as_tensor(lanes), torch.int32))
        f = lambda *s: torch.full(s, float("nan"), device=DEV)  # noqa: E731
        q, k, v, lg = f(rows, m.kv_heads, self.dimp), f(rows, m.kv_heads, self.dimp), f(rows, m.v_width), f(rows, m.heads, self.dimp)
        beta, o, out = f(rows, m.heads), f(rows, m.heads, m.vdim), torch.full((rows, m.v_width + 8), 2.0, dtype=T, device=DEV)
        act = t(torch.as_tensor(active), torch.int32) if active is not None else None
        a = native.DeltaArgs()
        p = lambda x: x.data_ptr()  # noqa: E731
        a.proj, a.proj_stride, a.off_b, a.conv_w, a.taps, a.conv_state = p(proj), proj.stride(0), off_b, p(keep["conv"]), m.conv, p(self.ring)
        a.a, a.a_stride, a.a_rate, a.dt_bias = p(keep["a"]), keep["a"].stride(0), p(keep["rate"]), p(keep["bias"])
        a.row_pos, a.row_lane, a.row_active = p(keep["pos"]), p(keep["lane"]), p(act) if act is not None else None
        a.q, a.k, a.v, a.lg, a.beta, a.state, a.o = p(q), p(k), p(v), p(lg), p(beta), p(self.state), p(o)
        a.gate, a.gate_stride, a.norm, a.out, a.out_stride = p(keep["gate"]), keep["gate"].stride(0), p(keep["norm"]), p(out), out.stride(0)
        a.H, a.G, a.dim, a.dimp, a.vdim, a.rows, a.decode = m.heads, m.kv_heads, m.dim, self.dimp, m.vdim, rows, int(decode)
        a.lanes, a.capacity, a.eps, a.status = self.lanes, self.capacity, self.eps, p(self.status)
        if fused:  # the low-rank halves: ranks as wide as the products, whose second table is the identity on this head's rows
            ra, rg = -(-m.heads * m.dim // 8) * 8, -(-m.v_width // 8) * 8
            wide = torch.zeros(rows, proj.shape[1] + ra + rg, dtype=T, device=DEV)
            wide[:, : proj.shape[1]] = proj
            wide[:, proj.shape[1] : proj.shape[1] + m.heads * m.dim], wide[:, proj.shape[1] + ra : proj.shape[1] + ra + m.v_width] = keep["a"].to(T), keep["gate"]
            a2, g2 = torch.zeros(m.heads * m.dim, ra, dtype=T, device=DEV), torch.zeros(m.v_width, rg, dtype=T, device=DEV)
            a2.fill_diagonal_(1.0), g2.fill_diagonal_(1.0)
            a.proj, a.proj_stride, a.off_a, a.off_g, a.ra, a.rg, a.a2, a.g2 = p(wide), wide.stride(0), proj.shape[1], proj.shape[1] + ra, ra, rg, p(a2), p(g2)
            native.delta_step(a)
            torch.cuda.synchronize()
            assert int(self.status) == 0 and (out[:, m.v_width :] == 2.0).all()
            return out[:, : m.v_width], None
        if chunked:
            native.delta_chunk(a, self.records)
        else:
            native.delta_prep(a, T is F32)
            native.delta_scan(a)
        native.delta_out(a, T is F32)
        torch.cuda.synchronize()
        assert int(self.status) == 0 and (out[:, m.v_width :] == 2.0).all()
        return out[:, : m.v_width], o


DELTA_SHAPES = [  # heads, key heads, dim, vdim, taps
    (4, 2, 128, 128, 4), (3, 1, 24, 40, 3), (2, 2, 64, 96, 2), (1, 1, 8, 8, 1), (2, 1, 96, 24, 4), (3, 3, 21, 13, 6), (2, 1, 200, 72, 4),
]


@pytest.mark.parametrize("shape", DELTA_SHAPES)
@pytest.mark.parametrize("kernel", ["f32", "bf16", "chunked"])
def test_delta_rule_in_portions(native_lib, shape, kernel):
    """Prompts in portions of many sizes (also shorter than the convolution, and cut inside and at 16-token chunks), a lane that held NaN."""
    m = delta(*shape)
    dtype = F32 if kernel == "f32" else BF16
    if kernel == "chunked" and not native_lib.delta_chunk_record(m.dim, m.vdim, m.conv):
        pytest.skip("not a size of the chunked kernels")
    total = 150
    c = delta_case(m, total, seed=m.dim)
    want, want_o, want_state = delta_expected(m, c, 1e-3)
    for cuts in ([], [1, 2, 4, 7, 23, 39, 40, 56, 120], [64], [149]):
        hx = DeltaHarness(native_lib, m, dtype, lanes=3)
        at = 0
        for cut in [*cuts, total]:
            out, o = hx.run(c, slice(at, cut), range(at, cut), [1] * (cut - at), decode=False, chunked=kernel == "chunked")
            close(o.reshape(cut - at, -1), want_o[at:cut].reshape(cut - at, -1), 2e-4)
            close(out, want[at:cut], 5e-4 if dtype is F32 else 0.02)
            at = cut
        close(hx.state[1, :, :, : m.dim].transpose(1, 2), want_state, 2e-4)
        assert torch.isnan(hx.state[[0, 2]]).all() and torch.isnan(hx.ring[[0, 2]].float()).all()


@pytest.mark.parametrize("shape", DELTA_SHAPES)
@pytest.mark.parametrize("kernel", ["f32", "bf16", "fused"])
def test_delta_rule_decoding_in_unequal_lanes(native_lib, shape, kernel):
    """One row per lane at unequal positions, an inactive lane whose state stays as it is, and a lane that starts over."""
    m = delta(*shape)
    dtype = F32 if kernel == "f32" else BF16
    cases = [delta_case(m, 40, seed=10 + i) for i in range(3)]
    for c in cases:
        c |= {key: cases[0][key] for key in ("conv", "a_log", "bias", "norm")}
        c["a"] = c["a"].to(BF16).double()  # what a bf16 product with the identity gives back
    wants = [delta_expected(m, c, 1e-3) for c in cases]
    hx = DeltaHarness(native_lib, m, dtype, lanes=3)
    hx.run(cases[0], slice(0, 5), range(5), [2] * 5, decode=False)
    for step in range(12):
        at = [5 + step, step if step < 6 else step - 6, 0 if step < 8 else step - 8]  # lane 1 starts over after six tokens
        active = [1, 1, int(step >= 8)]
        rows = {key: torch.stack([cases[i][key][at[i]] for i in range(3)]) if key in ("x", "b", "a", "gate") else cases[0][key] for key in cases[0]}
        out, _ = hx.run(rows, slice(0, 3), at, [2, 1, 0], decode=True, fused=kernel == "fused", active=active)
        for i in range(3):
            if active[i]:
                close(out[i], wants[i][0][at[i]], 1e-3 if dtype is F32 else 0.03)
        if step < 8:
            assert torch.isnan(hx.state[0]).all() and torch.isnan(hx.ring[0].float()).all()


def latent_case(m, total, seed, sharp=2.0):
    gen = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(s, generator=gen)  # noqa: E731
    b = lambda x: x.to(BF16).double()  # noqa: E731
    return {"cq": b(r(total, m.q_rank)), "kv": b(r(total, m.kv_rank + m.rot_dim)), "g": b(r(total, m.heads)), "q_norm": 1 + 0.1 * r(m.q_rank).double(),
            "kv_norm": 1 + 0.1 * r(m.kv_rank).double(), "uq": b(sharp * r(m.heads * (m.dim + m.rot_dim), m.q_rank) * m.q_rank**-0.5),
            "uk": b(r(m.heads * m.dim, m.kv_rank) * m.kv_rank**-0.5), "uv": b(r(m.heads * m.vdim, m.kv_rank) * m.kv_rank**-0.5), "sink": 1 + r(m.heads).double()}


def test_latent_pieces(native_lib):
    """Latents, cache rows, rotation, absorbed queries and gated values, with sizes that need padding everywhere."""
    native = native_lib
    for m, dtype, rows in ((latent(5, 19, 6, 11, 33, 27, base=777.0), F32, 11), (latent(5, 19, 6, 11, 33, 27), BF16, 11), (latent(4, 64, 64, 40, 96, 512), BF16, 11),
                           (latent(5, 19, 6, 11, 33, 27), BF16, 1), (latent(1, 2, 2, 3, 8, 6), BF16, 1), (latent(3, 5, 4, 7, 9, 300), BF16, 3)):
        lat, pe, dimp, lanes, capacity = -(-m.kv_rank // 16) * 16, -(-m.rot_dim // 16) * 16, -(-(m.dim + m.rot_dim) // 16) * 16, 3, 64
        c = latent_case(m, rows, 1)
        q_cols = (m.q_rank + 7) // 8 * 8
        off_kv, off_gate = q_cols, q_cols + (m.kv_rank + m.rot_dim + 7) // 8 * 8
        proj = torch.zeros(rows, off_gate + 8 + m.heads // 8 * 8, dtype=dtype, device=DEV)
        proj[:, : m.q_rank], proj[:, off_kv : off_kv + m.kv_rank + m.rot_dim], proj[:, off_gate : off_gate + m.heads] = c["cq"].to(dtype), c["kv"].to(dtype), c["g"].to(dtype)
        pos = torch.tensor([0, 1, 2, 3, 9, 8, 40, 63, 5, 6, 7], dtype=torch.int32)[-rows:]
        lane = torch.tensor([0, 0, 1, 1, 1, 2, 2, 2, 0, 0, 0], dtype=torch.int32)[-rows:]
        i = torch.arange(m.rot_dim // 2, dtype=torch.float64)
        angle = torch.arange(capacity, dtype=torch.float64)[:, None] * m.rot_base ** (-2 * i / m.rot_dim)
        rot = torch.stack([angle.cos(), angle.sin()], -1).float().to(DEV)
        cache = torch.full((lanes, capacity, lat + pe), float("nan"), dtype=dtype, device=DEV)
        cq = torch.full((rows, q_cols), 9.0, dtype=dtype, device=DEV)
        gen = torch.Generator().manual_seed(3)
        q0 = torch.nn.functional.pad(torch.randn(rows, m.heads, m.dim + m.rot_dim, generator=gen), (0, dimp - m.dim - m.rot_dim)).to(dtype)
        q, qa = q0.to(DEV), torch.full((rows, m.heads, lat + pe), 9.0, dtype=dtype, device=DEV)
        uk = torch.nn.functional.pad(c["uk"].reshape(m.heads, m.dim, m.kv_rank), (0, lat - m.kv_rank)).to(dtype).to(DEV)
        uv = torch.nn.functional.pad(c["uv"].reshape(m.heads, m.vdim, m.kv_rank), (0, lat - m.kv_rank)).to(dtype).to(DEV)
        o_lat = torch.randn(rows, m.heads, m.kv_rank, generator=gen).to(dtype).to(DEV)
        out = torch.full((rows, m.heads * m.vdim + 3), 9.0, dtype=dtype, device=DEV)
        status = torch.zeros(1, dtype=torch.int32, device=DEV)
        keep = [pos.to(DEV), lane.to(DEV), c["q_norm"].float().to(DEV), c["kv_norm"].float().to(DEV)]
        a = native.LatentArgs()
        a.proj, a.proj_stride, a.off_kv, a.off_gate, a.rot = proj.data_ptr(), proj.stride(0), off_kv, off_gate, rot.data_ptr()
        a.row_pos, a.row_lane, a.q_norm, a.kv_norm = (t.data_ptr() for t in keep)
        a.cq, a.cq_stride, a.cache, a.q, a.uk, a.qa, a.o_lat, a.uv = cq.data_ptr(), q_cols, cache.data_ptr(), q.data_ptr(), uk.data_ptr(), qa.data_ptr(), o_lat.data_ptr(), uv.data_ptr()
        a.out, a.out_stride, a.rows, a.H, a.dim, a.rot_dim, a.dimp, a.vdim = out.data_ptr(), out.stride(0), rows, m.heads, m.dim, m.rot_dim, dimp, m.vdim
        a.q_rank, a.kv_rank, a.lat, a.pe, a.lanes, a.capacity, a.eps, a.status = m.q_rank, m.kv_rank, lat, pe, lanes, capacity, 0.01, status.data_ptr()
        is_f32, tol = dtype is F32, 1e-4 if dtype is F32 else 0.02
        native.latent_rows(a, is_f32)
        native.latent_absorb(a, is_f32)  # reads q before it is rotated in place
        native.latent_query(a, is_f32)
        native.latent_value(a, is_f32)
        torch.cuda.synchronize()
        assert int(status) == 0
        close(cq[:, : m.q_rank], oracle.rms_norm(c["cq"], c["q_norm"], 0.01), tol)
        written = cache[lane.long(), pos.long()].double().cpu()
        close(written[:, : m.kv_rank], oracle.rms_norm(c["kv"][:, : m.kv_rank], c["kv_norm"], 0.01), tol)
        turn = lambda x: torch.stack([oracle.rotate_pairs(torch.cat([torch.zeros(int(p), *x.shape[1:], dtype=x.dtype), x[r : r + 1]]), m.rot_dim, m.rot_base)[-1]  # noqa: E731
                                      for r, p in enumerate(pos)])
        close(written[:, lat : lat + m.rot_dim], turn(c["kv"][:, None, m.kv_rank :])[:, 0], tol)
        assert not written[:, m.kv_rank : lat].any() and not written[:, lat + m.rot_dim :].any() and not cq[:, m.q_rank :].any()
        assert int(torch.isnan(cache[..., 0].float()).sum()) == lanes * capacity - rows
        q_d = q0.double()
        turned = turn(q_d[..., m.dim : m.dim + m.rot_dim])
        close(q[..., m.dim : m.dim + m.rot_dim], turned, tol)
        assert torch.equal(q[..., : m.dim].cpu(), q0[..., : m.dim])
        close(qa[..., : m.kv_rank], torch.einsum("rhd,hdl->rhl", q_d[..., : m.dim], c["uk"].reshape(m.heads, m.dim, m.kv_rank)), 3 * tol)
        close(qa[..., lat : lat + m.rot_dim], turned, tol)
        value = torch.einsum("rhl,hvl->rhv", o_lat.double().cpu(), c["uv"].reshape(m.heads, m.vdim, m.kv_rank)) * torch.sigmoid(c["g"])[..., None]
        close(out[:, : m.heads * m.vdim].reshape(rows, m.heads, m.vdim), value, 3 * tol)
        assert (out[:, m.heads * m.vdim :] == 9.0).all()


LATENT_DECODE = [  # heads, rotated, vdim, latent, rows, capacity
    (32, 64, 128, 512, 1, 4096), (40, 64, 128, 512, 8, 1024), (16, 32, 64, 192, 3, 700), (5, 6, 11, 27, 4, 64), (1, 2, 3, 6, 2, 320), (8, 128, 40, 496, 2, 2048),
]


@pytest.mark.parametrize("shape", LATENT_DECODE)
def test_latent_decode_attention(native_lib, shape):
    """Rows at unequal positions, around tile borders and at both ends; NaN in every cache row they must not see; an inactive row."""
    native = native_lib
    H, rot_dim, vdim, rank, rows, capacity = shape
    lat, pe = -(-rank // 16) * 16, -(-rot_dim // 16) * 16
    positions = [capacity - 1, 0, 63, 64, capacity // 2, 65, 127, 3][:rows]
    positions = [min(p, capacity - 1) for p in positions]
    gen = torch.Generator().manual_seed(rank)
    cache = torch.full((rows, capacity, lat + pe), float("nan"), dtype=BF16, device=DEV)
    zero = lambda *s: torch.zeros(s, dtype=torch.float64)  # noqa: E731
    qa, gate = zero(rows, H, lat + pe), torch.randn(rows, H, generator=gen).to(BF16)
    uv = (torch.randn(H, vdim, rank, generator=gen) * rank**-0.5).to(BF16)
    sink = 2 + torch.randn(H, generator=gen)
    scale, want = 0.07, []
    for r, pos in enumerate(positions):
        keys = zero(pos + 1, lat + pe)
        keys[:, :rank], keys[:, lat : lat + rot_dim] = torch.randn(pos + 1, rank, generator=gen), torch.randn(pos + 1, rot_dim, generator=gen)
        query = zero(H, lat + pe)
        query[:, :rank], query[:, lat : lat + rot_dim] = torch.randn(H, rank, generator=gen), torch.randn(H, rot_dim, generator=gen)
        far = 0 if r % 2 else pos // 3  # one key far back stands out for one head
        query[r % H] = keys[far] * 2
        keys, query = keys.to(BF16).double(), query.to(BF16).double()
        cache[r, : pos + 1], qa[r] = keys.to(BF16).to(DEV), query
        p = oracle.sink_softmax((query @ keys.T * scale)[:, None, :], sink.double(), torch.ones(1, pos + 1, dtype=torch.bool))[:, 0]
        o = torch.einsum("hl,hvl->hv", p @ keys[:, :rank], uv.double()) * torch.sigmoid(gate[r].double())[:, None]
        want.append(o.reshape(-1))
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full((rows, H * vdim + 8), 9.0, dtype=BF16, device=DEV)
    f = lambda n: torch.full((n,), float("nan"), device=DEV)  # noqa: E731
    active = [1] * rows
    if rows > 2:
        active[2] = 0
    keep = [torch.tensor(positions, dtype=torch.int32, device=DEV), torch.arange(rows, dtype=torch.int32, device=DEV), torch.tensor(active, dtype=torch.int32, device=DEV)]
    qa_d, gate_d, sink_d, part_o, part_ml = qa.to(BF16).to(DEV), gate.to(DEV), sink.to(DEV), f(max(rows, 32) * H * lat), f(max(rows, 32) * H * 2)
    uv_d = torch.nn.functional.pad(uv, (0, lat - rank)).contiguous().to(DEV)
    a = native.LatentArgs()
    a.proj, a.proj_stride, a.off_gate = gate_d.data_ptr(), H, 0
    a.row_pos, a.row_lane, a.row_active = (t.data_ptr() for t in keep)
    a.cache, a.qa, a.uv, a.sink, a.part_o, a.part_ml = cache.data_ptr(), qa_d.data_ptr(), uv_d.data_ptr(), sink_d.data_ptr(), part_o.data_ptr(), part_ml.data_ptr()
    a.out, a.out_stride, a.rows, a.H, a.dim, a.rot_dim, a.dimp, a.vdim = out.data_ptr(), out.stride(0), rows, H, 1, rot_dim, -(-(1 + rot_dim) // 16) * 16, vdim
    a.q_rank, a.kv_rank, a.lat, a.pe, a.lanes, a.capacity, a.scale, a.status = 1, rank, lat, pe, rows, capacity, scale, status.data_ptr()
    native.latent_decode(a)
    torch.cuda.synchronize()
    assert int(status) == 0 and (out[:, H * vdim :] == 9.0).all()
    for r in range(rows):
        if active[r]:
            close(out[r, : H * vdim], want[r], 0.03)
        else:
            assert not out[r, : H * vdim].any()


@pytest.mark.parametrize("dims", [(128, 128), (64, 40), (200, 256), (264, 272)])
def test_attention_with_a_gate_and_some_heads_of_wider_rows(native_lib, dims):
    native, (dim, vdim) = native_lib, dims
    H, rows, start = 2, 150, 70
    gen = torch.Generator().manual_seed(dim)
    dp, vp, total = -(-dim // 16) * 16, -(-vdim // 16) * 16, start + rows
    wide = torch.randn(rows, 3 * dp, generator=gen).to(BF16)
    wide.view(rows, 3, dp)[..., dim:] = 0
    k, v = torch.zeros(total, H, dp, dtype=BF16), torch.zeros(total, H, vp, dtype=BF16)
    k[..., :dim], v[..., :vdim] = torch.randn(total, H, dim, generator=gen), torch.randn(total, H, vdim, generator=gen)
    gate, sink = torch.randn(rows, 5, generator=gen).to(BF16), torch.randn(H, generator=gen)
    q = wide.view(rows, 3, dp)[:, 1:, :dim].double()
    scores = torch.einsum("ihd,jhd->hij", q, k[..., :dim].double()) * dim**-0.5
    visible = torch.arange(total)[None, :] <= torch.arange(start, total)[:, None]
    want = torch.einsum("hij,jhd->ihd", oracle.sink_softmax(scores, sink.double(), visible), v[..., :vdim].double()) * torch.sigmoid(gate[:, 3:].double())[..., None]
    wd, kd, vd, gd, sd = (t.to(DEV) for t in (wide, k, v, gate, sink))
    out = torch.full((rows, 3 * vdim), 9.0, dtype=BF16, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    a = native.ChunkAttnArgs()
    a.q, a.q_stride, a.k, a.v, a.sink = wd.data_ptr() + dp * 2, 3 * dp, kd.data_ptr(), vd.data_ptr(), sd.data_ptr()
    a.out, a.out_stride, a.gate, a.gate_stride = out.data_ptr() + vdim * 2, 3 * vdim, gd.data_ptr() + 6, 5
    a.rows, a.H, a.G, a.dim, a.dimp, a.vdim, a.vdimp, a.start, a.keys, a.chunk = rows, H, H, dim, dp, vdim, vp, start, total, 4096
    a.scale, a.status = dim**-0.5, status.data_ptr()
    native.chunk_attention(a, False)
    torch.cuda.synchronize()
    assert int(status) == 0 and (out[:, :vdim] == 9.0).all()
    assert float((out[:, vdim:].double().cpu().reshape(rows, H, vdim) - want).abs().max()) < 0.02


ROUTED = [(5, 7, 2, 64, 40), (8, 3, 3, 104, 24), (200, 8, 3, 256, 96), (130, 1, 1, 64, 24), (33, 16, 1, 128, 64)]  # rows, experts, top, width, ff


@pytest.mark.parametrize("shape", ROUTED)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_router_and_experts_with_the_weight_on_the_input(native_lib, shape, dtype):
    native = native_lib
    rows, E, top, width, ff = shape
    gen = torch.Generator().manual_seed(rows)
    b = lambda x: x.to(BF16)  # noqa: E731
    h = b(torch.randn(rows, width, generator=gen))
    weights = {"router": b(torch.randn(E, width, generator=gen) * 3 * width**-0.5)}
    for e in range(E):
        weights[f"e{e}.gate"], weights[f"e{e}.up"] = b(torch.randn(ff, width, generator=gen) * width**-0.5), b(torch.randn(ff, width, generator=gen) * width**-0.5)
        weights[f"e{e}.down"] = b(torch.randn(width, ff, generator=gen) * ff**-0.5)
    want = oracle.routed_experts(h.double(), {"experts": E, "top": top}, lambda n: weights[n].double())
    hd = h.to(dtype).to(DEV)
    scores = torch.full((rows, E + 5), 100.0, device=DEV)  # columns past the experts must not be looked at
    scores[:, :E] = (h.double() @ weights["router"].double().T).float().to(DEV)
    ids, w = torch.zeros(rows, top, dtype=torch.int32, device=DEV), torch.zeros(rows, top, device=DEV)
    native.router_topk(scores[:, :E], None, top, ids, w, normalize=False)
    close(w, torch.sigmoid(scores[:, :E].double()).topk(top, -1).values, 1e-5)
    gate_up = torch.stack([torch.cat([weights[f"e{e}.gate"], weights[f"e{e}.up"]]) for e in range(E)]).to(dtype).to(DEV)
    down = torch.stack([weights[f"e{e}.down"] for e in range(E)]).to(dtype).to(DEV)
    routes = rows * top
    act, out = torch.empty(routes, ff, dtype=dtype, device=DEV), torch.empty(rows, width, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    tol = 1e-4 if dtype is F32 else 0.03
    native.expert_glu(hd, ids, w, gate_up, act, native.GLU_SILU, status=status)
    native.expert_down(act, ids, down, out)
    close(out, want, tol)
    if dtype is BF16:  # the grouped form of prefill
        i32 = lambda *s: torch.zeros(s, dtype=torch.int32, device=DEV)  # noqa: E731
        tiles, n_tiles, perm, place = i32(routes // 128 + E + 1, 4), i32(1), i32(routes), i32(routes)
        x, gu, y = torch.empty(routes, width, dtype=BF16, device=DEV), torch.empty(routes, 2 * ff, dtype=BF16, device=DEV), torch.empty(routes, width, device=DEV)
        native.route_sort128(ids, 0, E, tiles, n_tiles, perm)
        native.gather_routes(hd, perm, top, place, x)
        assert torch.equal(perm[place.long()].cpu(), torch.arange(routes, dtype=torch.int32))
        native.gemm_bf16_tc(x, gate_up, gu, experts=E, tiles=tiles, n_tiles=n_tiles, status=status.data_ptr())
        native.glu_rows(gu[:, :ff], gu[:, ff:], act, native.GLU_SILU, scale=w, scale_at=perm)
        native.gemm_bf16_tc(act, down, y, experts=E, tiles=tiles, n_tiles=n_tiles, status=status.data_ptr())
        out.zero_()
        native.route_combine(y, place, top, out)
        close(out, want, tol)
    torch.cuda.synchronize()
    assert int(status) == 0


# ------------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("name", sorted(geometries()))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prefill_portions_and_decoding_agree_with_the_plain_model(native_lib, name, dtype):
    """Whole prompts, prompts in portions of many sizes (two tokens among them, cut at and around chunk and tile borders), token-by-token
    decoding: the logits of every position."""
    g = geometries()[name]
    ck, total = sharp_checkpoint(g, 1), 210
    tokens = settled_tokens(g, ck, total, 1)
    want = expected(g, ck, tokens)
    runner = runner_for(g, ck, dtype)
    try:
        whole = feed(runner, 0, tokens, [])
        check(whole, want, dtype)
        for lane, cuts in ((1, list(range(1, total))),                                   # one first token, then decoding only
                           (0, [2, 4, 7, 8, 24, 40, 42, 63, 64, 65, 96, 130, 131, 133, 190, 192]),
                           (1, list(range(2, total, 2))),                                # portions of two tokens
                           (0, [150] + list(range(151, total)))):                        # a prompt, then a long decoding
            got = feed(runner, lane, tokens, cuts)
            check(got, want, dtype)
            assert float(row_errors(got, whole).max()) < LIMIT[dtype]
    finally:
        runner.close()


@pytest.mark.parametrize("name", ["tiny", "tiles", "again"])
def test_specialised_kernels_against_the_size_independent_ones(native_lib, name):
    g = geometries()[name]
    ck = sharp_checkpoint(g, 2)
    tokens, rows = settled_tokens(g, ck, 150, 2), []
    for plain in (False, True):
        runner = runner_for(g, ck, BF16, plain=plain)
        rows.append(feed(runner, 0, tokens, [70, 71, 75] + list(range(76, 150))))
        runner.close()
    assert float(row_errors(rows[0], rows[1]).max()) < 0.05


@pytest.mark.parametrize("name", sorted(geometries()))
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


@pytest.mark.parametrize("name", ["tiny", "tiles"])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_lanes_do_not_see_each_other_and_are_used_again(native_lib, name, dtype):
    """Unequal requests decoding together against each alone; lanes given back with caches and states full, then used for other requests."""
    g = geometries()[name]
    ck = sharp_checkpoint(g, 3)
    lengths = [1, 40, 97, 150]
    seqs = [settled_tokens(g, ck, n + 30, 10 + n) for n in lengths]
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


def test_long_context_far_keys_slow_states_and_long_decoding(native_lib):
    """Hundreds of tokens whose last queries look for the first keys, states that hardly fade, keys and values expanded some heads at a
    time, in a prompt and in decoding."""
    from glm_tpu_b200.config.zikevik import DenseSpec, LayerSpec, ZikevikGeometry
    from glm_tpu_b200.models.zikevik import model as zm

    g = ZikevikGeometry(vocab_size=384, hidden_size=128, norm_eps=1e-5, embedding_scale=1.0, layers=(
        LayerSpec(latent(4, 32, 32, 48, 64, 96, base=1e6), DenseSpec(192)), LayerSpec(delta(4, 4, 32, 32), None), LayerSpec(latent(3, 16, 16, 32, 64, 64, base=1e6), DenseSpec(160))))
    ck = sharp_checkpoint(g, 6, factor=4.0)
    ck["l1.mix.dt_bias"][:32] = -14.0  # the first head forgets nothing to speak of
    tokens = tokens_for(g, 1250, 6)
    for at, back in ((598, 1), (599, 0), (601, 600), (899, 450), (1199, 0)):  # repeated tokens far back: like attracts like
        tokens[at] = tokens[back]
    want = expected(g, ck, tokens, dtype=torch.float64)
    for dtype in (F32, BF16):
        runner = runner_for(g, ck, dtype, capacity=1280, lanes=1, prefill_chunk=512)
        saved, zm.EXPAND_BYTES = zm.EXPAND_BYTES, 1280 * 250  # one or two heads at a time
        try:
            check(feed(runner, 0, tokens, []), want, dtype)
            check(feed(runner, 0, tokens, [560] + list(range(561, 640)) + [860] + list(range(861, 920)) + [1190] + list(range(1191, 1250))), want, dtype)
        finally:
            zm.EXPAND_BYTES = saved
            runner.close()


def test_a_full_lane_is_refused(native_lib):
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


@pytest.mark.parametrize("dtype,slack", [(F32, 1e-3), (BF16, 0.2)])
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
    """``bin/trace_run`` on a directory without the ranks in its config, in both number formats, with interleaved requests."""
    from glm_tpu_b200.model_loader.sharded_state import format as fmt

    g = geometries()["odd"]
    ck = sharp_checkpoint(g, 9)
    model = tmp_path / "model"
    model.mkdir()
    config = g.to_config()
    for layer in config["layers"]:
        layer["mixer"].pop("decay_rank", None)
        layer["mixer"].pop("gate_rank", None)
    (model / "config.json").write_text(json.dumps(config))
    fmt.write_file(model / "model.safetensors", ck, {})
    a, b = settled_tokens(g, ck, 40, 30), settled_tokens(g, ck, 12, 31)
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


def test_component_library_holds_what_the_family_launches(native_lib, tmp_path):
    """The family's own library, built alone and loaded in a fresh process, runs a prompt and a decode step."""
    code = """
import sys
from pathlib import Path
from glm_tpu_b200.csrc import build as b
from glm_tpu_b200.ops import native
b.LIB = Path(sys.argv[1]) / "never_there.so"
b.OUT_DIR = Path(sys.argv[1])
native.select_library(b.build(component="zikevik"))
from tests.zikevik_cases import geometries, sharp_checkpoint, tokens_for
from glm_tpu_b200.runner.gpu_runner import build_runner
g = geometries()["tiles"]
r = build_runner(g, device="cuda:0", checkpoint=sharp_checkpoint(g), context_capacity=128, prefill_chunk=64)
first = r.prefill(0, tokens_for(g, 70))
r.build_decode_program(); r.decode_step()
print("tokens", first, r.read_last_tokens()[0], native.LIB_PATH.name)
r.close()
"""
    done = subprocess.run([sys.executable, "-c", code, str(tmp_path)], capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert done.returncode == 0 and done.stdout.startswith("tokens") and "libglmb200_zikevik.so" in done.stdout, done.stderr[-2000:]
