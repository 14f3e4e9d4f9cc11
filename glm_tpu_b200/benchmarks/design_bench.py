"""Prefill and decode throughput of the one-GPU designs beside the GLM-MoE-DSA family at equal size, on one GPU.

    python bench.py --design namizen [--sizes small,medium,large] [--steps 64] [--warmup 8]
    python bench.py --design zikevik [--sizes small,medium,large,routed]
    python -m glm_tpu_b200.benchmarks.design_bench --kernels prefill [--family glm] [--size medium]

All models get the same width, head count, feed-forward sizes, vocabulary and layer count, and random weights; feed-forwards are dense except
at size `routed`, where every layer has routed experts (bf16 in Zikevik, FP8 with a shared one in GLM).  The GLM side keeps its latent
attention (rank 512) and its indexer; every third layer of Zikevik is latent attention of the same ranks, the others are delta-rule layers.
Decode is the captured step at a given depth (synthetic cache), timed with CUDA events over blocks of steps; prefill is a whole prompt
through the runner, timed the same way.  Every step streams more weight bytes than the L2 holds.  ``--kernels`` prints device time per
entry point of one eager prefill pass or decode step.
"""

from __future__ import annotations

import argparse
import json
import statistics
import sys

# width, heads, kv heads, head size, feed-forward, vocabulary, layers
SIZES = {
    "small": dict(width=2048, heads=16, kv_heads=4, head_dim=128, ff=8192, vocab=65536, layers=6),
    "medium": dict(width=4096, heads=32, kv_heads=8, head_dim=128, ff=14336, vocab=131072, layers=6),
    "large": dict(width=8192, heads=64, kv_heads=8, head_dim=128, ff=28672, vocab=131072, layers=4),
    "routed": dict(width=4096, heads=32, kv_heads=8, head_dim=128, ff=1536, experts=64, top=4, vocab=131072, layers=6),
}
DESIGNS = {"namizen": ("namizen", "glm"), "zikevik": ("zikevik", "glm")}
CHUNK = 8192
CONTEXT = 32768


def namizen_geometry(size: dict):
    from glm_tpu_b200.config.namizen import bench_namizen

    return bench_namizen(size["layers"], width=size["width"], heads=size["heads"], kv_heads=size["kv_heads"], head_dim=size["head_dim"], ff=size["ff"],
                         vocab=size["vocab"], chunk=CHUNK)


def zikevik_geometry(size: dict):
    from glm_tpu_b200.config.zikevik import RoutedSpec, bench_zikevik

    routed = RoutedSpec(size["experts"], size["top"], size["ff"]) if "experts" in size else None
    return bench_zikevik(size["layers"], width=size["width"], heads=size["heads"], head_dim=size["head_dim"], ff=size["ff"], vocab=size["vocab"],
                         routed=routed)


def geometry_of(family: str, size: dict):
    return {"namizen": namizen_geometry, "zikevik": zikevik_geometry, "glm": glm_geometry}[family](size)


def glm_geometry(size: dict):
    from glm_tpu_b200.config.model import ModelGeometry

    n = size["layers"]
    return ModelGeometry(
        vocab_size=size["vocab"], hidden_size=size["width"], num_layers=n, attention_heads=size["heads"], q_lora_rank=1536, kv_lora_rank=512,
        qk_nope_head_dim=64, qk_rope_head_dim=64, v_head_dim=size["head_dim"], dense_intermediate_size=size["ff"],
        moe_intermediate_size=size["ff"] if "experts" in size else 512, num_routed_experts=size.get("experts", 8), routed_top_k=size.get("top", 2), num_shared_experts=1, routed_scaling_factor=1.0, index_heads=32, index_head_dim=128, index_top_k=2048,
        indexer_types=tuple("full" if i % 4 == 0 else "shared" for i in range(n)), mlp_layer_types=("sparse" if "experts" in size else "dense",) * n, rope_theta=500000.0, rms_norm_eps=1e-5)


def parameters(g) -> int:
    """Weights a decode step of one lane streams (everything but the embedding table and the experts that are not chosen)."""
    if hasattr(g, "tensor_shapes"):
        total = 0
        for name, shape in g.tensor_shapes().items():
            if name == "embed" or len(shape) != 2:
                continue
            parts = name.split(".")
            if len(parts) == 4 and parts[2].startswith("e") and int(parts[2][1:]) >= g.layers[int(parts[0][1:])].mlp.top:
                continue
            total += shape[0] * shape[1]
        return total
    from glm_tpu_b200.models.glm_moe_dsa.weights import projection_shapes

    shapes = [shape for i in range(g.num_layers) for shape in projection_shapes(g, i).values()]
    return sum((g.routed_top_k if len(shape) == 3 else 1) * shape[-2] * shape[-1] for shape in shapes) + g.vocab_size * g.hidden_size


def make_runner(family: str, size: dict, lanes: int, prefill_chunk: int, graphs: bool = True):
    from glm_tpu_b200.runner.gpu_runner import build_runner

    g = geometry_of(family, size)
    return build_runner(g, device="cuda:0", seed=0, context_capacity=CONTEXT, lanes=lanes, prefill_chunk=prefill_chunk, use_graphs=graphs)


def timed(fn, repeats: int) -> list[float]:
    import torch

    out = []
    for _ in range(repeats):
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        start.record()
        fn()
        stop.record()
        torch.cuda.synchronize()
        out.append(start.elapsed_time(stop))
    return out


def measure(family: str, size: dict, *, lanes_list=(1, 8), prompt: int = 8192, prefill_chunk: int = 4096, steps: int = 64, warmup: int = 8, repeats: int = 3,
            depth: int = 8000) -> dict:
    import torch

    g = geometry_of(family, size)
    out: dict = {"parameters_streamed": parameters(g)}
    for lanes in lanes_list:
        runner = make_runner(family, size, lanes, prefill_chunk)
        if lanes == lanes_list[0]:
            ids = torch.randint(0, g.vocab_size, (prompt,), generator=torch.Generator().manual_seed(1)).tolist()
            runner.prefill(0, ids)
            ms = statistics.median(timed(lambda: runner.prefill(0, ids), repeats))
            out["prefill"] = {"prompt": prompt, "rows_per_pass": prefill_chunk, "ms": round(ms, 3), "tok_s": round(prompt / ms * 1e3)}
        for lane in range(lanes):
            runner.synthetic_context(lane, depth - 37 * lane, seed=lane)
        rec = runner.build_decode_program()
        for _ in range(max(warmup, 3)):
            runner.decode_step()
        ms = statistics.median(timed(lambda: [runner.decode_step() for _ in range(steps)], repeats)) / steps
        runner.peer.check_status()
        out[f"decode_{lanes}"] = {"lanes": lanes, "depth": depth, "ms_per_step": round(ms, 4), "tok_s": round(lanes * 1e3 / ms, 1),
                                  "launches": rec.launches, "weight_gbs": round(out["parameters_streamed"] * 2 / ms / 1e6, 1)}
        runner.close()
        del runner
        torch.cuda.empty_cache()
    return out


def run(sizes, *, steps: int, warmup: int, design: str = "namizen", sampler=None) -> dict:
    result = {}
    if sampler is not None:
        sampler.start()
    for name in sizes:
        result[name] = {"size": SIZES[name]}
        for family in DESIGNS[design]:
            result[name][family] = measure(family, SIZES[name], steps=steps, warmup=warmup)
            print(f"[{name}] {family}: {json.dumps(result[name][family])}", file=sys.stderr, flush=True)
    clocks = sampler.stop() if sampler is not None else None
    return {"sizes": result, "clocks": clocks}


def kernel_times(family: str, size: dict, what: str, lanes: int, rows: int) -> list:
    """``[(entry point, launches, total ms), ...]`` of one eager prefill pass or decode step (the second of two)."""
    import torch

    from glm_tpu_b200.ops import native

    runner = make_runner(family, size, lanes, rows, graphs=False)
    ids = torch.randint(0, size["vocab"], (CHUNK,), generator=torch.Generator().manual_seed(1)).tolist()
    if what == "decode":
        for lane in range(lanes):
            runner.synthetic_context(lane, 8000 - 37 * lane, seed=lane)
        call = runner.decode_step
        runner.build_decode_program()
    else:
        call = lambda: runner.prefill(0, ids)  # noqa: E731
    call()
    torch.cuda.synchronize()
    with native.kernel_timeline() as tl:
        call()
    totals: dict = {}
    for name, ints, ms in tl.rows():
        key = (name, tuple(i for i in ints if abs(i) < 1 << 24)[:4] if name.startswith(("gemm", "skinny")) else ())
        n, t = totals.get(key, (0, 0.0))
        totals[key] = (n + 1, t + ms)
    runner.close()
    return sorted(((name, ints, n, t) for (name, ints), (n, t) in totals.items()), key=lambda row: -row[3])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--kernels", choices=["prefill", "decode"], required=True)
    ap.add_argument("--family", choices=["namizen", "zikevik", "glm"], default="namizen")
    ap.add_argument("--size", choices=sorted(SIZES), default="medium")
    ap.add_argument("--lanes", type=int, default=1)
    ap.add_argument("--rows", type=int, default=4096)
    args = ap.parse_args(argv)
    from glm_tpu_b200.csrc.build import build

    build()
    for name, ints, n, ms in kernel_times(args.family, SIZES[args.size], args.kernels, args.lanes, args.rows):
        print(f"{ms:9.3f} ms  {n:4d} x {ms / n * 1e3:9.1f} us  {name} {ints}")
    return 0


if __name__ == "__main__":
    sys.exit(main())
