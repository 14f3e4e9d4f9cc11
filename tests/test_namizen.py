"""Namizen without a GPU: the plain implementation mechanism by mechanism, configuration, cache arithmetic, weights, the registry, the
replay of traces and the engine on the CPU backend."""

import io
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from glm_tpu_b200.config.cache import RingCacheConfig
from glm_tpu_b200.config.namizen import AttentionSpec, LayerSpec, NamizenGeometry, bench_namizen, tiny_namizen
from glm_tpu_b200.engine import request as rq
from glm_tpu_b200.engine.llm_engine import LLMEngine
from glm_tpu_b200.entrypoints.cli import trace as trace_cli
from glm_tpu_b200.exceptions import CheckpointValidationError, ConfigValidationError, PlanValidationError, RequestValidationError
from glm_tpu_b200.model_loader.directory import pad8
from glm_tpu_b200.model_loader.sharded_state import format as fmt
from glm_tpu_b200.models import registry
from glm_tpu_b200.models.namizen import weights as nw
from glm_tpu_b200.oracle import namizen as oracle
from glm_tpu_b200.runner.oracle_runner import OracleRunner
from glm_tpu_b200.worker.gpu_worker import profile_for
from tests.namizen_cases import attention, expected, geometries, row_errors, sharp_checkpoint, tokens_for

ROOT = Path(__file__).resolve().parents[1]


def write_model(directory: Path, g: NamizenGeometry, checkpoint: dict) -> Path:
    directory.mkdir(parents=True, exist_ok=True)
    (directory / "config.json").write_text(json.dumps(g.to_config()))
    fmt.write_file(directory / "model.safetensors", checkpoint, {})
    return directory


# ------------------------------------------------------------------------------------------------ the plain implementation
def test_convolution_starts_from_zeros_and_its_last_tap_is_now():
    u = torch.randn(6, 3, dtype=torch.float64)
    w = torch.randn(3, 4, dtype=torch.float64)
    y = oracle.causal_conv(u, w)
    for t in range(6):
        for c in range(3):
            want = sum(float(w[c, j]) * (float(u[t - 3 + j, c]) if t - 3 + j >= 0 else 0.0) for j in range(4))
            assert abs(float(y[t, c]) - want) < 1e-12


def test_rotation_pairs_halves_and_leaves_the_rest():
    x = torch.randn(5, 2, 10, dtype=torch.float64)
    y = oracle.rotate_half(x, 6, 50.0)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
    for p in range(5):
        for i in range(3):
            z = complex(x[p, 1, i], x[p, 1, i + 3]) * complex(torch.polar(torch.tensor(1.0, dtype=torch.float64), torch.tensor(p * 50.0 ** (-2 * i / 6), dtype=torch.float64)))
            assert abs(float(y[p, 1, i]) - z.real) < 1e-9 and abs(float(y[p, 1, i + 3]) - z.imag) < 1e-9


def test_chunks_are_counted_from_the_start():
    m = oracle.chunk_mask(10, 4)
    assert [j for j in range(10) if m[7, j]] == [4, 5, 6, 7] and [j for j in range(10) if m[8, j]] == [8] and [j for j in range(10) if m[3, j]] == [0, 1, 2, 3]


def test_a_sink_takes_its_share_and_counts_once():
    scores = torch.tensor([[[0.3, -9.0], [1.0, 2.0]]], dtype=torch.float64)
    sink = torch.tensor([0.5], dtype=torch.float64)
    p = oracle.sink_softmax(scores, sink, oracle.chunk_mask(2, 8))
    e = lambda v: float(torch.exp(torch.tensor(v, dtype=torch.float64)))  # noqa: E731
    assert abs(float(p[0, 0, 0]) - e(0.3) / (e(0.3) + e(0.5))) < 1e-12 and float(p[0, 0, 1]) == 0.0
    assert abs(float(p[0, 1, 1]) - e(2.0) / (e(1.0) + e(2.0) + e(0.5))) < 1e-12
    far = oracle.sink_softmax(scores * 0 - 500.0, sink + 300.0, oracle.chunk_mask(2, 8))
    assert torch.isfinite(far).all() and float(far.sum()) < 1e-100


def test_norm_activation_and_value_mixing():
    x = torch.tensor([[3.0, -4.0]], dtype=torch.float64)
    assert torch.allclose(oracle.rms_norm(x, torch.tensor([2.0, 1.0], dtype=torch.float64), 0.5), x / (12.5 + 0.5) ** 0.5 * torch.tensor([2.0, 1.0]))
    z = torch.linspace(-4, 4, 33, dtype=torch.float64)
    assert torch.allclose(oracle.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert float(oracle.mix_values(torch.tensor(2.0), torch.tensor(10.0), torch.tensor(0.25))) == 4.0


def test_only_layers_that_mix_share_values_and_both_branches_read_the_same_residual():
    g = tiny_namizen()
    ck = sharp_checkpoint(g, 1)
    tokens = tokens_for(g, 30)
    base = expected(g, ck, tokens)
    other = dict(ck)
    other["l1.mix.vmix"] = torch.tensor(0.9, dtype=torch.bfloat16)  # the first mixing layer: unused
    assert torch.equal(expected(g, other, tokens), base)
    other["l2.mix.vmix"] = torch.tensor(0.9, dtype=torch.bfloat16)
    assert float(row_errors(expected(g, other, tokens), base).max()) > 0.02
    layers: list = []
    expected(g, ck, tokens, layers_out=layers)
    x0 = ck["embed"].double()[tokens]
    cfg, get = g.to_config(), lambda n: ck[n].double()  # noqa: E731
    attn, _ = oracle.attention(oracle.rms_norm(x0, get("l0.norm1"), 1e-5), cfg["layers"][0]["mixer"], lambda n: get("l0.mix." + n), None)
    ff = oracle.feed_forward(oracle.rms_norm(x0, get("l0.norm2"), 1e-5), lambda n: get("l0.mlp." + n))
    assert torch.allclose(layers[0], x0 + attn + ff)


@pytest.mark.parametrize("mistake", ["chunk", "sink", "history", "far_key"])
def test_sharp_weights_show_a_small_mistake(mistake, monkeypatch):
    """What the engine tests rely on: each of these faults, planted here, moves some logits far beyond the tolerance they use."""
    g = geometries()["tiles"]
    ck, tokens = sharp_checkpoint(g, 3), tokens_for(g, 150, 3)
    right = expected(g, ck, tokens)
    if mistake == "chunk":
        plain = oracle.chunk_mask
        monkeypatch.setattr(oracle, "chunk_mask", lambda total, size: plain(total, size + 1))
    elif mistake == "sink":
        plain_softmax = oracle.sink_softmax
        monkeypatch.setattr(oracle, "sink_softmax", lambda s, sink, visible: plain_softmax(s, sink - 1e4, visible))
    elif mistake == "history":
        plain_conv = oracle.causal_conv
        monkeypatch.setattr(oracle, "causal_conv", lambda u, w: torch.cat([plain_conv(u[:100], w), plain_conv(u[100:], w)]))  # state lost at row 100
    else:
        plain_mask = oracle.chunk_mask

        def without_first(total, size):
            m = plain_mask(total, size)
            m[95, 0] = False  # the farthest key of the longest chunk row
            return m

        monkeypatch.setattr(oracle, "chunk_mask", without_first)
        ck = dict(ck)
        ck["l0.mix.q"] = ck["l0.mix.q"] * 0.25
        ck["embed"] = ck["embed"].clone()
        ck["embed"][tokens[0]] = ck["embed"][tokens[95]]  # like tokens attract one another
        right = None
    wrong = expected(g, ck, tokens)
    if right is None:
        monkeypatch.undo()
        right = expected(g, ck, tokens)
    worst = float(row_errors(wrong, right).max())
    assert worst > (0.002 if mistake == "far_key" else 0.1), worst


# ------------------------------------------------------------------------------------------------ configuration
def test_config_round_trip_and_refusals():
    for g in geometries().values():
        assert NamizenGeometry.from_config(json.loads(json.dumps(g.to_config()))) == g and len(g.geometry_hash) == 64
    assert len({g.geometry_hash for g in geometries().values()}) == len(geometries())
    good = tiny_namizen().to_config()
    for change in ({"architecture": "Other"}, {"layers": []}, {"norm": {}}, {"vocab": 0}):
        with pytest.raises(ConfigValidationError):
            NamizenGeometry.from_config({**good, **change})
    for path, value in ((("type",), "recurrent"), (("mlp", "kind"), "routed"), (("mixer", "heads"), 5), (("mixer", "rot", "dims"), 7), (("mixer", "mask", "size"), 0)):
        bad = json.loads(json.dumps(good))
        at = bad["layers"][0]
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(ConfigValidationError):
            NamizenGeometry.from_config(bad)
    with pytest.raises(ConfigValidationError):  # mixing layers need equal value heads
        NamizenGeometry(64, 32, (LayerSpec(attention(2, 1, 8, 8, 2, 8, 1e4, 8, True)), LayerSpec(attention(2, 1, 8, 16, 2, 8, 1e4, 8, True))), 1e-5)


def test_every_constant_of_the_file_matters():
    """Changing any number of config.json (weights of the same shapes) changes the logits or the shapes: nothing is assumed."""
    g = tiny_namizen()
    ck, tokens = sharp_checkpoint(g, 2), tokens_for(g, 70, 2)
    base = expected(g, ck, tokens)
    for key, value in (("scale", 0.5), ("rot", {"dims": 8, "base": 10000.0}), ("rot", {"dims": 16, "base": 300.0}), ("mask", {"size": 47})):
        config = g.to_config()
        config["layers"][0]["mixer"][key] = value
        assert float(row_errors(oracle.forward(config, ck, tokens), base).max()) > 1e-3, key
        assert NamizenGeometry.from_config(config) != g
    config = g.to_config()
    config["norm"]["eps"] = 0.5
    assert float(row_errors(oracle.forward(config, ck, tokens), base).max()) > 1e-3 and NamizenGeometry.from_config(config).norm_eps == 0.5


def test_registry():
    g, source = registry.resolve_model("random:namizen-tiny")
    assert source == ("random", None) and registry.family_of(g) is registry.NAMIZEN and not registry.NAMIZEN.multi_gpu
    assert registry.family_of_config(g.to_config()) is registry.NAMIZEN and registry.family_of_config({"model_type": "glm_moe_dsa"}) is registry.GLM
    assert registry.resolve_model("random:namizen-tiny:2")[0].num_layers == 2
    assert registry.family_of(registry.resolve_model("random:tiny")[0]) is registry.GLM
    assert "float32" in registry.NAMIZEN.dtypes and "float32" not in registry.GLM.dtypes
    for spec in ("random:unknown",):
        with pytest.raises(ConfigValidationError):
            registry.resolve_model(spec)
    with pytest.raises(ConfigValidationError):
        registry.family_of_config({"architecture": "unknown"})
    with pytest.raises(ConfigValidationError):
        registry.family_of(object())
    big = bench_namizen(2, width=64, heads=4, kv_heads=2, head_dim=16, ff=96, vocab=154880, chunk=32)
    assert profile_for(big, 256).model_id == "Namizen"  # a vocabulary of GLM's size does not make it GLM


# ------------------------------------------------------------------------------------------------ cache arithmetic
def test_ring_cache_shapes_and_slots():
    g = geometries()["odd"]
    c = RingCacheConfig(g, 64, lanes=3)
    assert [c.ring(i) for i in range(3)] == [7, 64, 19] and c.k_shape(0) == (3, 7, 3, 32) and c.v_shape(1) == (3, 64, 1, 48) and c.conv_shape(1) == (3, 4, 5 * 36 + 36 + 44)
    assert c.cache_bytes_per_gpu() == 2 * sum(a * b * d * e for i in range(3) for a, b, d, e in (c.k_shape(i), c.v_shape(i))) + 2 * sum(
        a * b * d for a, b, d in (c.conv_shape(i) for i in range(3)))
    for bad in (dict(context_capacity=0), dict(context_capacity=8, lanes=9), dict(context_capacity=8, lanes=0)):
        with pytest.raises(PlanValidationError):
            RingCacheConfig(g, **bad)


@pytest.mark.parametrize("chunk", [1, 2, 7, 64, 1000])
def test_a_step_finds_every_key_it_sees(chunk):
    """A lane driven by portions of many sizes, with the ring and the linear buffer as plain lists: every query's visible keys are where the
    step looks for them."""
    g = NamizenGeometry(16, 8, (LayerSpec(attention(1, 1, 4, 4, 2, 4, 1e4, chunk)),), 1e-5)
    c = RingCacheConfig(g, 300)
    gen = torch.Generator().manual_seed(chunk)
    ring, at = [None] * c.ring(0), 0
    while at < 300:
        rows = min(int(torch.randint(1, 90, (1,), generator=gen)), 300 - at)
        base, across = c.first_position(0, at), c.crossing(0, at, rows)
        if across is None:
            for p in range(at, at + rows):
                ring[p % c.ring(0)] = p
            keys = ring[: at + rows - base]
        else:
            before, after = across
            keys = ring[:before] + list(range(at, at + rows))
            assert len(keys) <= c.linear_rows(0, rows) and before == at - base
            ring[:after] = keys[len(keys) - after :]
        for p in range(at, at + rows):
            first = p // c.chunk(0) * c.chunk(0)
            assert keys[first - base : p - base + 1] == list(range(first, p + 1))
        at += rows
        last = c.first_position(0, at - 1)
        assert ring[: at - last] == list(range(last, at))  # what decoding reads next


# ------------------------------------------------------------------------------------------------ weights
def test_resident_tables_from_a_directory(tmp_path):
    g = geometries()["odd"]
    ck = sharp_checkpoint(g, 4)
    path = write_model(tmp_path / "model", g, ck)
    geometry, source = registry.resolve_model(str(path))
    assert geometry == g and source == ("checkpoint", path)
    tensors = registry.NAMIZEN.load_checkpoint(path)
    assert set(tensors) == set(ck) and all(torch.equal(tensors[n], ck[n]) for n in ck) and len(tensors) == len(ck)
    w = nw.resident_weights(g, tensors, "cpu", torch.float32)
    lw = w.layers[0]
    assert lw.qkv.shape == (pad8(3 * 21 * 2 + 3 * 13), 104) and torch.equal(lw.qkv[:63, :100], ck["l0.mix.q"].float()) and not lw.qkv[:, 100:].any()
    assert torch.equal(lw.qkv[126 : 126 + 39, :100], ck["l0.mix.v"].float()) and torch.equal(lw.conv[0, 63:126], ck["l0.mix.k.conv"][:, 0].float())
    assert torch.equal(lw.out[:100, :39], ck["l0.mix.o"].float()) and torch.equal(lw.out[:100, 40 : 40 + 51], ck["l0.mlp.down"].float())
    assert not lw.out[:, 39].any() and lw.mix == 0.0 and w.layers[2].mix == float(ck["l2.mix.vmix"]) and w.layers[1].gate_up is None
    assert w.head.shape == (304, 104) and w.bytes_resident > 0
    assert nw.resident_weights(g, tensors, "cpu").embed.dtype == torch.bfloat16
    with pytest.raises(CheckpointValidationError):
        registry.NAMIZEN.load_checkpoint(path, pins={"manifest_sha256": "ab" * 32})


def test_missing_and_misshapen_tensors_are_refused():
    g = tiny_namizen()
    ck = nw.random_checkpoint(g)
    short = {n: t for n, t in ck.items() if n != "l2.mix.k.conv"}
    with pytest.raises(CheckpointValidationError, match="l2.mix.k.conv"):
        nw.resident_weights(g, short, "cpu")
    with pytest.raises(CheckpointValidationError, match="shape"):
        nw.resident_weights(g, {**ck, "l0.mix.o": ck["l0.mix.o"][:, :-1]}, "cpu")
    without = {n: t for n, t in ck.items() if n != "l1.mix.vmix"}  # the first mixing layer's amount is never used
    assert nw.resident_weights(g, without, "cpu").layers[1].mix == 0.0
    nw.check_tensors(g, ck, shape_of=lambda n: ck[n].shape)
    with pytest.raises(CheckpointValidationError, match="embed"):
        nw.check_tensors(g, ck, shape_of=lambda n: (1,))


# ------------------------------------------------------------------------------------------------ replay
class PlainRunner:
    """The replay's view of a runner, answered by the plain implementation."""

    def __init__(self, g, checkpoint, lanes=2):
        self.g, self.ck, self.lanes = g, checkpoint, lanes
        self.lengths, self.tokens, self.calls = [0] * lanes, [[] for _ in range(lanes)], []

    def open_lane(self, lane):
        self.lengths[lane], self.tokens[lane] = 0, []
        self.calls.append(("open", lane))

    def extend(self, lane, ids, want):
        self.calls.append(("extend", lane, len(ids)))
        first = len(self.tokens[lane])
        self.tokens[lane] += ids
        self.lengths[lane] = len(self.tokens[lane])
        out = expected(self.g, self.ck, self.tokens[lane]).float()
        return out[[first + w for w in want]]

    def decode_logits(self, tokens):
        self.calls.append(("decode", tuple(sorted(tokens))))
        return {lane: self.extend(lane, [t], [0])[0] for lane, t in tokens.items()}

    def close(self):
        pass


def test_replay_routes_tokens_writes_logits_and_gives_lanes_back(tmp_path):
    g = tiny_namizen()
    ck = nw.random_checkpoint(g, 5)
    a, b, c = tokens_for(g, 9, 1), tokens_for(g, 4, 2), tokens_for(g, 3, 3)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:6], "want": [5, 1]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[:1], "want": [0]}, {"id": "a", "tokens": a[6:7], "want": [0]}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": a[7:], "want": []}], "end": ["a"]},
        {"step": 7, "entries": [{"id": "b", "tokens": b[1:2], "want": [0]}, {"id": "c", "tokens": c, "want": [2, 0]}], "end": ["b", "c"]},
    ]
    runner, lines = PlainRunner(g, ck), []
    trace_cli.replay(runner, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), tmp_path, emit=lambda line, flush: lines.append(line))
    assert lines == ["done 0", "done 1", "done 2", "done 7"] and sorted(p.name for p in tmp_path.iterdir()) == ["0.f32", "1.f32", "7.f32"]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / n).read_bytes()), dtype=torch.float32).reshape(-1, g.vocab_size)  # noqa: E731
    la, lb, lc = (expected(g, ck, t).float() for t in (a, b, c))
    assert torch.allclose(read("0.f32"), la[[5, 1]]) and torch.allclose(read("1.f32"), torch.stack([lb[0], la[6]])) and torch.allclose(
        read("7.f32"), torch.stack([lb[1], lc[2], lc[0]]))
    calls = runner.calls
    assert ("decode", (0,)) in calls and ("decode", (1,)) in calls  # later single tokens go through the decode program
    assert ("extend", 1, 1) in calls  # a first token alone is a prompt
    assert calls.count(("open", 0)) == 2  # the lane of `a` serves `c`
    with pytest.raises(RequestValidationError):
        session = trace_cli.TraceReplay(PlainRunner(g, ck, lanes=1))
        session.step({"step": 0, "entries": [{"id": "x", "tokens": [1], "want": []}, {"id": "y", "tokens": [1], "want": []}]})
    with pytest.raises(RequestValidationError):
        trace_cli.TraceReplay(PlainRunner(g, ck)).step({"step": 0, "entries": [{"id": "x", "tokens": [1], "want": []}] * 2})


def test_replay_program_refuses_a_format_no_kernel_has(tmp_path):
    done = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", "random:tiny", "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "8"],
                          input="", capture_output=True, text=True, timeout=300)
    assert done.returncode == 3 and done.stdout == "" and os.access(ROOT / "bin" / "trace_run", os.X_OK)


# ------------------------------------------------------------------------------------------------ engine, worker, command line
def greedy(g, ck, prompt, n, dtype=torch.float32):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(torch.argmax(expected(g, ck, seq, dtype=dtype)[-1])))
        if seq[-1] in g.eos_ids:
            break
    return seq[len(prompt) :]


def test_engine_generates_greedily_on_the_cpu_backend():
    g = tiny_namizen()
    ck = nw.random_checkpoint(g, 0)
    profile = profile_for(g, 128)
    runner = OracleRunner(g, ck, context_capacity=128, lanes=2)
    prompts = [tokens_for(g, 20, 1), tokens_for(g, 5, 2)]
    requests = [rq.from_token_ids(p, request_id=f"r{i}", max_new_tokens=4 + i, context_capacity=128, profile=profile) for i, p in enumerate(prompts)]
    events: list = []
    engine = LLMEngine(runner, profile=profile)
    assert engine.generate(requests[0], events.append)["emitted"] == len(greedy(g, ck, prompts[0], 4))
    assert [e.token_id for e in events] == greedy(g, ck, prompts[0], 4)
    events.clear()
    engine.generate_concurrent(rq.batch(requests, concurrent=True, profile=profile), events.append)
    for i, p in enumerate(prompts):
        assert [e.token_id for e in events if e.request_id == f"r{i}"] == greedy(g, ck, p, 4 + i)


def test_ask_serves_a_directory_end_to_end_on_the_cpu_backend(tmp_path):
    """The command line, the controller and a worker process with a Namizen directory as the model."""
    g = NamizenGeometry(vocab_size=320, hidden_size=32, norm_eps=1e-5, eos_ids=(318, 319), layers=(
        LayerSpec(attention(2, 1, 16, 8, 3, 8, 1e4, 24, True), 48), LayerSpec(attention(4, 2, 8, 4, 2, 8, 1e4, 16, True), 40)))  # the same eight value channels in two heads
    model = write_model(tmp_path / "model", g, nw.random_checkpoint(g, 7))
    env = dict(os.environ, GLM_B200_RUN_ROOT=str(tmp_path / "runs"), GLM_B200_SITE_CONFIG=str(tmp_path / "none.toml"))
    (tmp_path / "runs").mkdir()
    done = subprocess.run([sys.executable, "-m", "glm_tpu_b200", "ask", "hi", "--model", str(model), "--backend", "oracle", "--gpus", "1", "--capacity", "128",
                           "--max-new-tokens", "3"], capture_output=True, text=True, timeout=280, env=env, cwd=ROOT)
    assert done.returncode == 0, done.stdout[-2000:] + done.stderr[-2000:]
    record = next((tmp_path / "runs").rglob("runner.rank0.json"))
    body = json.loads(record.read_text())
    assert body["geometry_hash"] == g.geometry_hash and body["requests"][0]["emitted"] >= 1
    prompt = json.loads(next((tmp_path / "runs").rglob("prepared-000.json")).read_text())["prompt_ids"]
    tokens = [json.loads(line)["token_id"] for line in next((tmp_path / "runs").rglob("tokens.jsonl")).read_text().splitlines()]
    assert tokens == greedy(g, nw.random_checkpoint(g, 7), prompt, 3)


def test_attention_parameters_are_checked():
    with pytest.raises(ConfigValidationError):
        AttentionSpec(heads=4, kv_heads=3, dim=8, vdim=8, scale=1.0)
    with pytest.raises(ConfigValidationError):
        AttentionSpec(heads=4, kv_heads=2, dim=8, vdim=8, scale=1.0, rot_dims=10)
    assert AttentionSpec(heads=4, kv_heads=2, dim=8, vdim=6, scale=1.0).out_width == 24


def test_the_family_library_is_complete(tmp_path, monkeypatch):
    """What the family launches links without the rest of the kernels, loads, and has every entry point its bindings call."""
    from glm_tpu_b200.csrc import build as builder

    if not Path(builder.NVCC).exists():
        pytest.skip("no CUDA compiler")
    builder.build()
    monkeypatch.setattr(builder, "LIB", tmp_path / "complete.so")  # as in a checkout where nothing is built
    monkeypatch.setattr(builder, "OUT_DIR", tmp_path)
    path = builder.build(component="namizen")
    assert path == tmp_path / "libglmb200_namizen.so"
    code = ("import sys; from glm_tpu_b200.ops import native; native.select_library(sys.argv[1]); lib = native.lib(); "
            "[getattr(lib, 'glmb_' + n) for n in ('parallel_norm', 'dual_proj', 'qkv_conv', 'kv_copy', 'chunk_attn_prefill', 'chunk_attn_decode', "
            "'chunk_attn_any', 'glu_rows', 'gemm_f32', 'skinny_bf16', 'gemm_bf16_tcgen05', 'argmax_rows_f32', 'step_finalize', 'fill_random_bf16', "
            "'peer_create')]; print(hasattr(lib, 'glmb_moe_gateup_fp8'))")
    done = subprocess.run([sys.executable, "-c", code, str(path)], capture_output=True, text=True, timeout=120, cwd=ROOT)
    assert done.returncode == 0 and done.stdout.strip() == "False", done.stderr[-2000:]
