"""Zikevik without a GPU: the plain implementation mechanism by mechanism, planted mistakes the sharp weights must show, configuration, cache
shapes, weights, registry, engine and command line on the CPU backend."""

import dataclasses
import json
import math
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from glm_tpu_b200.config.cache import HybridCacheConfig
from glm_tpu_b200.config.zikevik import DenseSpec, LayerSpec, RoutedSpec, ZikevikGeometry, bench_zikevik, tiny_zikevik
from glm_tpu_b200.engine import request as rq
from glm_tpu_b200.engine.llm_engine import LLMEngine
from glm_tpu_b200.exceptions import CheckpointValidationError, ConfigValidationError, PlanValidationError
from glm_tpu_b200.model_loader.directory import SourceTensors, pad8
from glm_tpu_b200.model_loader.sharded_state import format as fmt
from glm_tpu_b200.models import registry
from glm_tpu_b200.models.zikevik import weights as zw
from glm_tpu_b200.oracle import zikevik as oracle
from glm_tpu_b200.runner.oracle_runner import OracleRunner
from glm_tpu_b200.worker.gpu_worker import profile_for
from tests.zikevik_cases import MARGIN, delta, expected, geometries, latent, row_errors, settled_tokens, sharp_checkpoint, tokens_for

ROOT = Path(__file__).resolve().parents[1]


def rand(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def write_model(directory: Path, g: ZikevikGeometry, checkpoint: dict, *, ranks: bool = True) -> Path:
    directory.mkdir(parents=True, exist_ok=True)
    config = g.to_config()
    if not ranks:
        for layer in config["layers"]:
            layer["mixer"].pop("decay_rank", None)
            layer["mixer"].pop("gate_rank", None)
    (directory / "config.json").write_text(json.dumps(config))
    fmt.write_file(directory / "model.safetensors", checkpoint, {})
    return directory


# ------------------------------------------------------------------------------------------------ the plain implementation
def test_norms_activations_and_unit_vectors():
    x, w = rand(3, 6), rand(6, seed=1) * 0.1
    for r in range(3):
        rms = math.sqrt(sum(float(v) ** 2 for v in x[r]) / 6 + 0.5)
        for c in range(6):
            assert abs(float(oracle.zero_centred_norm(x, w, 0.5)[r, c]) - float(x[r, c]) / rms * (1 + float(w[c]))) < 1e-12
            assert abs(float(oracle.rms_norm(x, w, 0.5)[r, c]) - float(x[r, c]) / rms * float(w[c])) < 1e-12
    z = torch.tensor([-800.0, -30.0, -1.0, 0.0, 2.0, 800.0], dtype=torch.float64)
    assert torch.allclose(oracle.softplus(z), torch.tensor([0.0, math.exp(-30), math.log1p(math.exp(-1)), math.log(2), 2 + math.log1p(math.exp(-2)), 800.0], dtype=torch.float64))
    assert abs(float(oracle.silu(torch.tensor(1.5))) - 1.5 / (1 + math.exp(-1.5))) < 1e-6
    u = oracle.unit(torch.tensor([[3e-4, 4e-4]], dtype=torch.float64))  # the constant is inside the root
    assert torch.allclose(u, torch.tensor([[3e-4, 4e-4]], dtype=torch.float64) / math.sqrt(25e-8 + 1e-6))


def test_convolution_starts_from_zeros_and_its_last_tap_is_now():
    u, w = rand(5, 2), rand(2, 3, seed=1)
    got = oracle.causal_conv(u, w)
    for t in range(5):
        for c in range(2):
            want = sum(float(w[c, j]) * float(u[t - 2 + j, c]) for j in range(3) if t - 2 + j >= 0)
            assert abs(float(got[t, c]) - want) < 1e-12


def test_delta_rule_by_hand():
    """Two tokens, two key and two value channels; the write uses the decayed state, the read-out sees the write."""
    q, k, g = (rand(2, 1, 2, seed=s) for s in (1, 2, 3))
    v, beta = rand(2, 1, 2, seed=4), torch.tensor([[0.3], [0.8]], dtype=torch.float64)
    g = torch.sigmoid(g)
    out, state = oracle.delta_rule(q, k, v, beta, g)
    S = [[0.0, 0.0], [0.0, 0.0]]
    for t in range(2):
        S = [[float(g[t, 0, d]) * S[d][c] for c in range(2)] for d in range(2)]
        for c in range(2):
            u = float(beta[t]) * (float(v[t, 0, c]) - sum(S[d][c] * float(k[t, 0, d]) for d in range(2)))
            for d in range(2):
                S[d][c] += float(k[t, 0, d]) * u
        for c in range(2):
            assert abs(float(out[t, 0, c]) - sum(S[d][c] * float(q[t, 0, d]) for d in range(2))) < 1e-12
    assert torch.allclose(state[0], torch.tensor(S, dtype=torch.float64))
    again, _ = oracle.delta_rule(q, k, v, beta, g, state)  # a state that is carried on
    longer, _ = oracle.delta_rule(*(torch.cat([x, x]) for x in (q, k, v, beta, g)))
    assert torch.allclose(longer[2:], again)


def test_decay_is_per_head_and_key_channel():
    h, a1, a2, bias, a_log = rand(3, 5), rand(2, 5, seed=1), rand(6, 2, seed=2), rand(6, seed=3), rand(2, seed=4)
    got = oracle.channel_decay(h, a1, a2, bias, a_log, 2, 3)
    for t in range(3):
        for head in range(2):
            for d in range(3):
                z = sum(float(a2[head * 3 + d, r]) * sum(float(a1[r, i]) * float(h[t, i]) for i in range(5)) for r in range(2)) + float(bias[head * 3 + d])
                assert abs(float(got[t, head, d]) - math.exp(-math.exp(float(a_log[head])) * math.log1p(math.exp(z)))) < 1e-12


def test_key_heads_are_shared_by_consecutive_value_heads():
    m, width = delta(4, 2, 8, 8, 2, 3, 3), 16
    w = {n: rand(*s, seed=i) * 0.5 for i, (n, s) in enumerate(m.tensors(width).items())}
    cfg, h = m.to_config(), rand(6, width, seed=99)
    base = oracle.channel_delta(h, cfg, w.__getitem__, 1e-5)
    alone = []  # every value head by itself, with the key head it should use
    for head in range(4):
        kv = head // 2
        rows, vrows = slice(kv * 8, kv * 8 + 8), slice(head * 8, head * 8 + 8)
        one = {"q": w["q"][rows], "q.conv": w["q.conv"][rows], "k": w["k"][rows], "k.conv": w["k.conv"][rows], "v": w["v"][vrows], "v.conv": w["v.conv"][vrows],
               "b": w["b"][head : head + 1], "A_log": w["A_log"][head : head + 1], "norm": w["norm"], "a1": w["a1"], "a2": w["a2"][vrows], "dt_bias": w["dt_bias"][vrows],
               "g1": w["g1"], "g2": w["g2"][vrows], "o": w["o"][:, vrows]}
        alone.append(oracle.channel_delta(h, {**cfg, "heads": 1, "kv_heads": 1}, one.__getitem__, 1e-5))
    assert torch.allclose(sum(alone), base)


def test_rotation_pairs_neighbours_and_starts_at_position_zero():
    x = rand(4, 1, 6)
    got = oracle.rotate_pairs(x, 4, 100.0)
    assert torch.equal(got[0], x[0]) and torch.equal(got[..., 4:], x[..., 4:])
    for p in range(4):
        for i in range(2):
            a = p * 100.0 ** (-2 * i / 4)
            u, v = float(x[p, 0, 2 * i]), float(x[p, 0, 2 * i + 1])
            assert abs(float(got[p, 0, 2 * i]) - (u * math.cos(a) - v * math.sin(a))) < 1e-12
            assert abs(float(got[p, 0, 2 * i + 1]) - (v * math.cos(a) + u * math.sin(a))) < 1e-12


def test_a_sink_takes_its_share_and_counts_once():
    scores, sink = rand(2, 3, 3), torch.tensor([0.5, -1.0], dtype=torch.float64)
    p = oracle.sink_softmax(scores, sink, torch.ones(3, 3, dtype=torch.bool).tril())
    for h in range(2):
        for i in range(3):
            total = math.exp(float(sink[h])) + sum(math.exp(float(scores[h, i, j])) for j in range(i + 1))
            for j in range(3):
                assert abs(float(p[h, i, j]) - (math.exp(float(scores[h, i, j])) / total if j <= i else 0.0)) < 1e-12


def test_latent_attention_absorbed_is_the_same():
    """Queries through the key projection against the latents themselves: what the engine's decode computes."""
    m, width, T = latent(3, 6, 4, 5, 8, 7), 12, 9
    w = {n: rand(*s, seed=i) * 0.7 for i, (n, s) in enumerate(m.tensors(width).items())}
    h = rand(T, width, seed=50)
    base = oracle.latent_attention(h, m.to_config(), w.__getitem__, 1e-5)
    q = (oracle.rms_norm(h @ w["dq"].T, w["dq.norm"], 1e-5) @ w["uq"].T).reshape(T, 3, 10)
    joint = h @ w["dkv"].T
    c = oracle.rms_norm(joint[:, :7], w["dkv.norm"], 1e-5)
    qa = torch.einsum("thd,hdl->thl", q[..., :6], w["uk"].reshape(3, 6, 7))
    qr, kr = oracle.rotate_pairs(q[..., 6:], 4, m.rot_base), oracle.rotate_pairs(joint[:, None, 7:], 4, m.rot_base)[:, 0]
    s = (torch.einsum("thl,jl->htj", qa, c) + torch.einsum("thr,jr->htj", qr, kr)) * m.scale
    p = oracle.sink_softmax(s, w["sink"], torch.ones(T, T, dtype=torch.bool).tril())
    out = torch.einsum("htl,hvl->thv", torch.einsum("htj,jl->htl", p, c), w["uv"].reshape(3, 5, 7)) * torch.sigmoid(h @ w["g"].T)[..., None]
    assert torch.allclose(out.reshape(T, -1) @ w["o"].T, base)


def test_experts_take_the_weighted_input_and_scores_are_not_renormalized():
    E, top, width, ff = 4, 2, 6, 5
    w = {"router": rand(E, width)} | {f"e{e}.{n}": rand(*s, seed=10 * e + i) for e in range(E) for i, (n, s) in enumerate(DenseSpec(ff).tensors(width).items())}
    h = rand(3, width, seed=77)
    got = oracle.routed_experts(h, {"experts": E, "top": top}, w.__getitem__)
    for t in range(3):
        s = torch.sigmoid(w["router"] @ h[t])
        want = torch.zeros(width, dtype=torch.float64)
        for e in s.argsort(descending=True)[:top].tolist():
            x = s[e] * h[t]
            z = w[f"e{e}.gate"] @ x
            want += w[f"e{e}.down"] @ (z * torch.sigmoid(z) * (w[f"e{e}.up"] @ x))
        assert torch.allclose(got[t], want)


def test_layers_that_use_other_layers_weights():
    g = geometries()["again"]
    ck, tokens = sharp_checkpoint(g, 1), tokens_for(g, 20)
    copied = dataclasses.replace(g, layers=tuple(dataclasses.replace(layer, weights_of=None) for layer in g.layers))
    names = [n for n in copied.tensor_shapes() if n.split(".")[0] in ("l2", "l3", "l4")]
    assert names and not any(n in g.tensor_shapes() for n in names)
    full = dict(ck)
    for i in (2, 3, 4):
        full |= {f"l{i}" + n[len(f"l{g.owner(i)}") :]: t for n, t in ck.items() if n.startswith(f"l{g.owner(i)}.")}
    assert g.owner(4) == 1 and torch.equal(expected(copied, full, tokens), expected(g, ck, tokens))


@pytest.mark.parametrize("mistake", ["state", "history", "decay_order", "sink", "far_key", "rotation", "weight_outside", "shared_state"])
def test_sharp_weights_show_a_small_mistake(mistake, monkeypatch):
    """What the engine tests rely on: each of these faults, planted here, moves some logits far beyond the tolerance they use."""
    g = geometries()["again" if mistake == "shared_state" else "tiny" if mistake == "weight_outside" else "tiles"]
    ck, T = sharp_checkpoint(g, 3), 150
    tokens = tokens_for(g, T, 3)
    if mistake == "far_key":
        tokens[140] = tokens[0]
    right = expected(g, ck, tokens)
    if mistake == "state":  # lost between two portions
        plain = oracle.delta_rule
        monkeypatch.setattr(oracle, "delta_rule", lambda *x: (torch.cat([plain(*(t[:100] for t in x))[0], plain(*(t[100:] for t in x))[0]]), None))
    elif mistake == "history":
        plain_conv = oracle.causal_conv
        monkeypatch.setattr(oracle, "causal_conv", lambda u, w: torch.cat([plain_conv(u[:100], w), plain_conv(u[100:], w)]))
    elif mistake == "decay_order":  # the token's decay after its write
        plain = oracle.delta_rule
        monkeypatch.setattr(oracle, "delta_rule", lambda q, k, v, beta, decay: plain(q, k, v, beta, torch.cat([torch.ones_like(decay[:1]), decay[:-1]])))
    elif mistake == "sink":
        plain_softmax = oracle.sink_softmax
        monkeypatch.setattr(oracle, "sink_softmax", lambda s, sink, visible: plain_softmax(s, sink - 1e4, visible))
    elif mistake == "far_key":
        plain_softmax = oracle.sink_softmax

        def without_first(s, sink, visible):
            visible = visible.clone()
            visible[1:, 0] = False
            return plain_softmax(s, sink, visible)

        monkeypatch.setattr(oracle, "sink_softmax", without_first)
    elif mistake == "rotation":  # one position off from the hundredth token on
        plain_rot = oracle.rotate_pairs

        def shifted(x, dims, base):
            longer = plain_rot(torch.cat([x, x[-1:]]), dims, base)
            moved = plain_rot(torch.cat([x[:1], x]), dims, base)[1:]
            return torch.cat([longer[:100], moved[100 : x.shape[0]]])

        monkeypatch.setattr(oracle, "rotate_pairs", shifted)
    elif mistake == "weight_outside":

        def outside(h, router, weight):
            scores = torch.sigmoid(h @ weight("router").T)
            value, chosen = scores.topk(router["top"], dim=-1)
            out = torch.zeros_like(h)
            for e in range(router["experts"]):
                rows, slot = (chosen == e).nonzero(as_tuple=True)
                out = out.index_add(0, rows, value[rows, slot][:, None] * oracle.gated_ff(h[rows], weight, f"e{e}."))
            return out

        monkeypatch.setattr(oracle, "routed_experts", outside)
    else:  # a layer that runs again goes on from the state its first run left
        plain, left = oracle.delta_rule, []

        def carried(*x):
            out, state = plain(*x, left[-1] if left and left[-1].shape == (x[0].shape[1], x[0].shape[2], x[2].shape[2]) else None)
            left.append(state)
            return out, state

        monkeypatch.setattr(oracle, "delta_rule", carried)
    worst = float(row_errors(expected(g, ck, tokens), right).max())
    assert worst > (0.005 if mistake == "far_key" else 0.1), worst


def test_settled_tokens_leave_no_close_call():
    g = geometries()["tiles"]
    ck = sharp_checkpoint(g, 5)
    tokens, margins = settled_tokens(g, ck, 80, 5, keep=((60, 2),)), []
    expected(g, ck, tokens, margins_out=margins)
    assert len(margins) == 2 and float(torch.stack(margins).min()) > MARGIN * 0.99 and tokens[60] == tokens[2]
    h, router = rand(2, 3), {"experts": 3, "top": 3}
    assert torch.isinf(oracle.router_margin(h, router, lambda n: rand(3, 3))).all()


# ------------------------------------------------------------------------------------------------ configuration
def test_config_round_trip_and_refusals():
    for g in geometries().values():
        assert ZikevikGeometry.from_config(json.loads(json.dumps(g.to_config()))) == g and len(g.geometry_hash) == 64
    assert len({g.geometry_hash for g in geometries().values()}) == len(geometries())
    good = tiny_zikevik().to_config()
    for change in ({"architecture": "Other"}, {"layers": []}, {"norm": {}}, {"vocab": 0}, {"embedding": {}}):
        with pytest.raises(ConfigValidationError):
            ZikevikGeometry.from_config({**good, **change})
    for layer, path, value in ((0, ("type",), "attention"), (0, ("mlp", "kind"), "sparse"), (0, ("mixer", "heads"), 5), (1, ("mixer", "rot", "dims"), 6), (1, ("mixer", "rot_dim"), 0),
                               (1, ("mlp", "router", "top"), 7), (1, ("mlp", "expert", "ff"), 0), (4, ("weights_of",), 4), (4, ("weights_of",), 9), (4, ("weights_of",), 1)):
        bad = json.loads(json.dumps(good))
        at = bad["layers"][layer]
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(ConfigValidationError):
            ZikevikGeometry.from_config(bad)


def test_ranks_come_from_the_tensors():
    g = geometries()["odd"]
    config = g.to_config()
    for layer in config["layers"]:
        layer["mixer"].pop("decay_rank", None)
        layer["mixer"].pop("gate_rank", None)
    with pytest.raises(ConfigValidationError):
        ZikevikGeometry.from_config(config)
    assert ZikevikGeometry.from_config(config, g.tensor_shapes()) == g
    again = geometries()["again"]  # a layer without tensors of its own asks the layer whose weights it uses
    config = again.to_config()
    for layer in config["layers"]:
        layer["mixer"].pop("decay_rank", None)
        layer["mixer"].pop("gate_rank", None)
    assert ZikevikGeometry.from_config(config, again.tensor_shapes()) == again


def test_every_constant_of_the_file_matters():
    """Changing any number of config.json (weights of the same shapes) changes the logits: nothing is assumed."""
    g = tiny_zikevik()
    ck, tokens = sharp_checkpoint(g, 2), tokens_for(g, 70, 2)
    base = expected(g, ck, tokens)
    for layer, key, value in ((1, "scale", 0.05), (1, "rot", {"dims": 12, "base": 300.0})):
        config = g.to_config()
        config["layers"][layer]["mixer"][key] = value
        assert float(row_errors(oracle.forward(config, ck, tokens), base).max()) > 1e-3 and ZikevikGeometry.from_config(config) != g, key
    for section, key, value in (("norm", "eps", 0.5), ("embedding", "scale", 1.0)):
        config = g.to_config()
        config[section][key] = value
        assert float(row_errors(oracle.forward(config, ck, tokens), base).max()) > 1e-3 and ZikevikGeometry.from_config(config) != g, key
    config = g.to_config()
    config["layers"][1]["mlp"]["router"]["top"] = 1
    assert float(row_errors(oracle.forward(config, ck, tokens), base).max()) > 1e-2


def test_registry():
    g, source = registry.resolve_model("random:zikevik-tiny")
    assert source == ("random", None) and registry.family_of(g) is registry.ZIKEVIK and not registry.ZIKEVIK.multi_gpu
    assert registry.family_of_config(g.to_config()) is registry.ZIKEVIK and registry.resolve_model("random:zikevik-tiny:2")[0].num_layers == 2
    assert registry.ZIKEVIK.dtypes == ("bfloat16", "float32") and not registry.NAMIZEN.matches(g.to_config())
    assert registry.ZIKEVIK.from_config(g.to_config()) == g
    big = bench_zikevik(3, width=64, heads=4, head_dim=16, ff=96, vocab=154880)
    assert profile_for(big, 256).model_id == "Zikevik"  # a vocabulary of GLM's size does not make it GLM
    assert [layer.mixer.kind for layer in big.layers] == ["channel_delta", "channel_delta", "latent_attention"]
    with pytest.raises(PlanValidationError):
        registry.ZIKEVIK.build_runner(g, world=2, device="cpu")


# ------------------------------------------------------------------------------------------------ cache and scratch sizes
def test_hybrid_cache_shapes():
    g = geometries()["odd"]
    c = HybridCacheConfig(g, 100, lanes=3, element_bytes=4)
    assert [c.is_latent(i) for i in range(4)] == [False, True, False, True]
    assert c.latent_shape(1) == (3, 100, 32 + 16) and c.latent_shape(3) == (3, 100, 96 + 16)
    assert c.state_shape(0) == (3, 3, 13, 32) and c.state_shape(2) == (3, 2, 44, 64)
    assert c.conv_shape(0) == (3, 1, 2 * 21 + 39) and c.conv_shape(2) == (3, 6, 2 * 72 + 88)
    assert c.cache_bytes_per_gpu() == sum(c.layer_bytes(i) for i in range(4))
    assert c.layer_bytes(0) == 4 * (3 * 3 * 13 * 32 + 3 * 81) and c.layer_bytes(1) == 4 * 3 * 100 * 48
    assert HybridCacheConfig(g, 200, lanes=3).layer_bytes(0) == HybridCacheConfig(g, 100, lanes=3).layer_bytes(0)  # a state does not grow with the context
    for bad in (dict(context_capacity=0), dict(context_capacity=8, lanes=9)):
        with pytest.raises(PlanValidationError):
            HybridCacheConfig(g, **bad)


def test_scratch_is_sized_for_the_widest_layer():
    from glm_tpu_b200.models.zikevik import model as zm

    g = geometries()["tiles"]
    cache = HybridCacheConfig(g, 256, lanes=2)
    decode = zm.workspace_elements(g, cache, 2, prefill=False, is_f32=False)
    prefill = zm.workspace_elements(g, cache, 64, prefill=True, is_f32=False)
    assert "keys" not in decode["model"] and prefill["model"]["keys"] == 256 * 40 * 128 and prefill["f32"]["records"] > 0
    assert "records" not in zm.workspace_elements(g, cache, 64, prefill=True, is_f32=True)["f32"]
    assert decode["model"]["qa"] == 2 * 40 * 576 and prefill["model"]["qa"] == 8 * 40 * 576
    m = g.layers[1].mixer
    assert zm.expand_heads(m, 256, 2) == 40 and zm.expand_heads(m, 1 << 22, 2) == 1
    assert zm.delta_record_bytes(delta(1, 1, 200, 8)) == 0 and zm.delta_record_bytes(delta(1, 1, 8, 12)) == 0 and zm.delta_record_bytes(delta(1, 1, 8, 8, 5)) == 0


# ------------------------------------------------------------------------------------------------ weights
def test_resident_tables_from_a_directory(tmp_path):
    g = geometries()["odd"]
    ck = sharp_checkpoint(g, 4)
    path = write_model(tmp_path / "model", g, ck, ranks=False)
    geometry, source = registry.resolve_model(str(path))
    assert geometry == g and source == ("checkpoint", path)
    tensors = registry.ZIKEVIK.load_checkpoint(path)
    assert isinstance(tensors, SourceTensors) and set(tensors) == set(ck) and all(torch.equal(tensors[n], ck[n]) for n in ck)
    w = zw.resident_weights(g, tensors, "cpu", torch.float32)
    t = w.layers[0].mixer
    C = 2 * 21 + 39
    assert t.proj.shape == (pad8(C) + 8 + 8 + 8, 104) and (t.off_b, t.off_a, t.off_g) == (pad8(C), pad8(C) + 8, pad8(C) + 16)
    assert torch.equal(t.proj[:21, :100], ck["l0.mix.q"].float()) and torch.equal(t.proj[42:C, :100], ck["l0.mix.v"].float()) and not t.proj[:, 100:].any()
    assert torch.equal(t.proj[t.off_b : t.off_b + 3, :100], ck["l0.mix.b"].float()) and torch.equal(t.proj[t.off_g : t.off_g + 7, :100], ck["l0.mix.g1"].float())
    assert torch.equal(t.conv, torch.cat([ck[f"l0.mix.{n}.conv"].float().T for n in "qkv"], 1)) and torch.equal(t.a_rate, ck["l0.mix.A_log"].float().exp())
    assert t.a2.shape == (pad8(63), 8) and torch.equal(t.a2[:63, :5], ck["l0.mix.a2"].float()) and t.out.shape == (104, 40)
    m, t = g.layers[1].mixer, w.layers[1].mixer
    assert (t.off_kv, t.off_gate, t.dimp, t.vdimp) == (40, 80, 32, 16) and t.proj.shape == (88, 104)
    uq = ck["l1.mix.uq"].float().view(5, 25, 33)
    assert torch.equal(t.uq.view(5, 32, 40)[:, :25, :33], uq) and not t.uq.view(5, 32, 40)[:, 25:].any()
    row = torch.randn(1, 48)  # a cache row: latent, padding, rotated part, padding
    row[:, 27:32] = row[:, 38:] = 0
    keys = (row @ t.expand_k.T).view(5, 32)
    assert torch.allclose(keys[:, :19], (ck["l1.mix.uk"].float() @ row[0, :27]).view(5, 19), atol=1e-5) and torch.equal(keys[:, 19:25], row[:, 32:38].expand(5, 6))
    assert not keys[:, 25:].any()
    assert torch.allclose((row[:, :32] @ t.expand_v.T).view(5, 16)[:, :11], (ck["l1.mix.uv"].float() @ row[0, :27]).view(5, 11), atol=1e-5)
    f = w.layers[1].mlp
    assert f.router.shape == (8, 104) and f.gate_up.shape == (3, 64, 104) and f.down.shape == (3, 104, 32)
    assert torch.equal(f.gate_up[2, 32 : 32 + 29, :100], ck["l1.mlp.e2.up"].float()) and torch.equal(f.down[1, :100, :29], ck["l1.mlp.e1.down"].float())
    assert w.layers[3].mlp is None and w.layers[3].norm2 is None and w.head.shape == (304, 104)
    assert zw.resident_weights(g, tensors, "cpu").embed.dtype == torch.bfloat16
    with pytest.raises(CheckpointValidationError):
        registry.ZIKEVIK.load_checkpoint(path, pins={"manifest_sha256": "ab" * 32})
    again = geometries()["again"]
    shared = zw.resident_weights(again, sharp_checkpoint(again), "cpu")
    assert shared.layers[4].mixer is shared.layers[1].mixer and shared.layers[2] is shared.layers[0]
    single = sum(t.numel() * t.element_size() for layer in (shared.layers[0], shared.layers[1], shared.layers[5]) for part in (layer, layer.mixer, layer.mlp)
                 for t in vars(part).values() if isinstance(t, torch.Tensor))
    counted = single + sum(t.numel() * t.element_size() for t in (shared.embed, shared.final_norm, shared.head))
    assert shared.bytes_resident <= counted and shared.bytes_resident > counted * 0.9  # shared tables once (values that need no padding serve twice)


def test_missing_and_misshapen_tensors_are_refused():
    g = tiny_zikevik()
    ck = zw.random_checkpoint(g)
    with pytest.raises(CheckpointValidationError, match="l2.mix.k.conv"):
        zw.resident_weights(g, {n: t for n, t in ck.items() if n != "l2.mix.k.conv"}, "cpu")
    with pytest.raises(CheckpointValidationError, match="shape"):
        zw.resident_weights(g, {**ck, "l0.mix.o": ck["l0.mix.o"][:, :-1]}, "cpu")


# ------------------------------------------------------------------------------------------------ engine, worker, command line
def greedy(g, ck, prompt, n, dtype=torch.float32):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(torch.argmax(expected(g, ck, seq, dtype=dtype)[-1])))
        if seq[-1] in g.eos_ids:
            break
    return seq[len(prompt) :]


def test_engine_generates_greedily_on_the_cpu_backend():
    g = tiny_zikevik()
    ck = zw.random_checkpoint(g, 0)
    profile = profile_for(g, 128)
    runner = OracleRunner(g, ck, context_capacity=128, lanes=2)
    prompts = [tokens_for(g, 20, 1), tokens_for(g, 5, 2)]
    requests = [rq.from_token_ids(p, request_id=f"r{i}", max_new_tokens=4 + i, context_capacity=128, profile=profile) for i, p in enumerate(prompts)]
    events: list = []
    LLMEngine(runner, profile=profile).generate_concurrent(rq.batch(requests, concurrent=True, profile=profile), events.append)
    for i, p in enumerate(prompts):
        assert [e.token_id for e in events if e.request_id == f"r{i}"] == greedy(g, ck, p, 4 + i)


def test_ask_serves_a_directory_end_to_end_on_the_cpu_backend(tmp_path):
    """The command line, the controller and a worker process with a Zikevik directory as the model."""
    g = ZikevikGeometry(vocab_size=320, hidden_size=32, norm_eps=1e-5, embedding_scale=2.0, eos_ids=(318, 319), layers=(
        LayerSpec(delta(2, 1, 8, 8, 3, 4, 4), RoutedSpec(3, 2, 24)), LayerSpec(latent(2, 8, 4, 8, 12, 16), DenseSpec(40)), LayerSpec(delta(2, 1, 8, 8, 3, 4, 4), RoutedSpec(3, 2, 24), weights_of=0)))
    ck = zw.random_checkpoint(g, 7)
    model = write_model(tmp_path / "model", g, ck, ranks=False)
    env = dict(os.environ, GLM_B200_RUN_ROOT=str(tmp_path / "runs"), GLM_B200_SITE_CONFIG=str(tmp_path / "none.toml"))
    (tmp_path / "runs").mkdir()
    done = subprocess.run([sys.executable, "-m", "glm_tpu_b200", "ask", "hi", "--model", str(model), "--backend", "oracle", "--gpus", "1", "--capacity", "128",
                           "--max-new-tokens", "3"], capture_output=True, text=True, timeout=280, env=env, cwd=ROOT)
    assert done.returncode == 0, done.stdout[-2000:] + done.stderr[-2000:]
    body = json.loads(next((tmp_path / "runs").rglob("runner.rank0.json")).read_text())
    assert body["geometry_hash"] == g.geometry_hash and body["requests"][0]["emitted"] >= 1
    prompt = json.loads(next((tmp_path / "runs").rglob("prepared-000.json")).read_text())["prompt_ids"]
    tokens = [json.loads(line)["token_id"] for line in next((tmp_path / "runs").rglob("tokens.jsonl")).read_text().splitlines()]
    assert tokens == greedy(g, ck, prompt, 3)


def test_the_family_library_is_complete(tmp_path, monkeypatch):
    """What the family launches links without the rest of the kernels, loads, and has every entry point its bindings call."""
    from glm_tpu_b200.csrc import build as builder

    if not Path(builder.NVCC).exists():
        pytest.skip("no CUDA compiler")
    builder.build()
    monkeypatch.setattr(builder, "LIB", tmp_path / "complete.so")  # as in a checkout where nothing is built
    monkeypatch.setattr(builder, "OUT_DIR", tmp_path)
    path = builder.build(component="zikevik")
    assert path == tmp_path / "libglmb200_zikevik.so"
    code = ("import sys; from glm_tpu_b200.ops import native; native.select_library(sys.argv[1]); lib = native.lib(); "
            "[getattr(lib, 'glmb_' + n) for n in ('parallel_norm', 'delta_prep', 'delta_scan', 'delta_out', 'delta_chunk', 'delta_step', 'latent_rows', 'latent_query', "
            "'latent_absorb', 'latent_value', 'latent_decode', 'chunk_attn_prefill', 'chunk_attn_decode', 'chunk_attn_any', 'router_topk', 'route_sort128', 'expert_glu', "
            "'expert_down', 'gather_routes', 'route_combine', 'glu_rows', 'gemm_f32', 'skinny_bf16', 'skinny_bf16_swiglu', 'gemm_bf16_tcgen05', 'argmax_rows_f32', "
            "'step_finalize', 'fill_random_bf16', 'peer_create')]; print(hasattr(lib, 'glmb_moe_gateup_fp8'))")
    done = subprocess.run([sys.executable, "-c", code, str(path)], capture_output=True, text=True, timeout=120, cwd=ROOT)
    assert done.returncode == 0 and done.stdout.strip() == "False", done.stderr[-2000:]
