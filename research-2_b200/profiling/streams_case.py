"""Runs one kernel three times at sizes that exceed the L2 cache, for ncu to capture one launch of a case that ends by itself:

    python -m research_2_b200.profiling.streams_case --kernel join --rows 16384 &&
    ncu --set full --clock-control none -k regex:stream_join -s 1 -c 1 -o join \
        python -m research_2_b200.profiling.streams_case --kernel join --rows 16384

--kernel join: several residual streams take a sublayer's output (kernel stream_join). chunks: decay attention over prompts (kernels
decay_chunk_sums, decay_chunk_states, decay_chunk_outputs; --entries of --rows rows). step: its decode step (kernel decay_step; --entries
requests). router: corrected softmax scores with identity outputs (kernel route_scored_rows from 512 rows on, else route_scored). experts:
the first product of experts without gates, gelu and routing weights in its epilogue. With --time the case is timed inside a CUDA graph
of 20 launches and microseconds per launch are printed.
"""
import argparse

import torch

from ..kernels import ops
from .kernel_cases import time_in_graph


def main() -> int:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--kernel", default="join", choices=("join", "chunks", "step", "router", "experts"))
    ap.add_argument("--rows", type=int, default=16384)
    ap.add_argument("--entries", type=int, default=16)
    ap.add_argument("--width", type=int, default=768)
    ap.add_argument("--streams", type=int, default=4)
    ap.add_argument("--heads", type=int, default=6)
    ap.add_argument("--dim", type=int, default=64)
    ap.add_argument("--time", action="store_true")
    args = ap.parse_args()
    dev, d, s, h, dk = "cuda:0", args.width, args.streams, args.heads, args.dim
    if args.kernel == "join":
        x, y = torch.randn(args.rows, s, d, device=dev), torch.randn(args.rows, d, device=dev)
        read, mix, gain = torch.full((s,), 1.0 / s, device=dev), torch.eye(s, device=dev), torch.ones(d, device=dev)
        fn = lambda: ops.stream_join(x, read, gain, 1e-5, torch.bfloat16, y=y, mix=mix, join=read)  # noqa: E731
    elif args.kernel in ("chunks", "step"):
        rows = 1 if args.kernel == "step" else args.rows
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)  # noqa: E731
        arrays = (i32([i * rows for i in range(args.entries + 1)]), i32(list(range(args.entries))), i32([0] * args.entries))
        qkv = torch.randn(args.entries * rows, 3 * h * dk, device=dev).bfloat16()
        state, decay = torch.zeros(args.entries, h * dk * dk, device=dev), torch.full((h,), 0.97, device=dev)
        q, k, v = qkv.split(h * dk, dim=1)
        positions = torch.zeros(args.entries * rows, dtype=torch.int32, device=dev)
        fn = lambda: ops.retention_scan(q, k, v, decay, 1.0, None, 0, positions, state, *arrays, h, dk, dk, silu=True,  # noqa: E731
                                        n_tiles=args.entries * -(-rows // 64))
    else:
        hrow = torch.randn(args.rows, d, device=dev).bfloat16()
        router, correction = torch.randn(10, d, device=dev) * 0.02, torch.randn(10, device=dev) * 0.1
        pick = lambda: ops.route_scored(hrow, router, correction, 3, 2, 1, scoring="softmax", group_mark="best", n_identity=2)  # noqa: E731
        route, w_up = pick()[0], (torch.randn(8 * d, d, device=dev) * 0.02).bfloat16()
        fn = pick if args.kernel == "router" else lambda: ops.routed_linear(hrow, w_up, "gelu", route, d)  # noqa: E731
    if args.time:
        print(f"{time_in_graph(fn):.1f} us a launch")
        return 0
    for _ in range(3):
        fn()
    torch.cuda.synchronize()
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
