"""Runs the recurrence of the gated delta rule (or, with --time-mix, of time mixing with a decay per channel) of given sizes three
times, for ncu to capture one launch of a case that ends by itself:

    python -m research_2_b200.profiling.state_scan_case --entries 16 --rows 256 &&
    ncu --set full --clock-control none -k regex:state_scan -s 1 -c 1 -o scan \
        python -m research_2_b200.profiling.state_scan_case --entries 16 --rows 256

(--rows 1: a decode step, kernel state_step). With --prepare the launch in front of the recurrence runs instead (kernels
delta_prepare, time_mix_prepare). With --time the case is timed inside a CUDA graph of 20 launches and microseconds per launch are
printed.
"""
import argparse

import torch

from ..kernels import ops
from .kernel_cases import time_in_graph


def main() -> int:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--heads", type=int, default=12)
    ap.add_argument("--groups", type=int, default=6, help="delta rule: heads of queries and keys")
    ap.add_argument("--dim", type=int, default=64)
    ap.add_argument("--vdim", type=int, default=64)
    ap.add_argument("--width", type=int, default=768)
    ap.add_argument("--entries", type=int, default=16)
    ap.add_argument("--rows", type=int, default=256, help="rows of every entry (1: a decode step)")
    ap.add_argument("--time-mix", action="store_true")
    ap.add_argument("--prepare", action="store_true")
    ap.add_argument("--time", action="store_true")
    args = ap.parse_args()
    dev, h, g, dk = "cuda:0", args.heads, args.groups, args.dim
    dv = dk if args.time_mix else args.vdim
    t, d = args.entries * args.rows, args.width
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)  # noqa: E731
    arrays = (i32([i * args.rows for i in range(args.entries + 1)]), i32(list(range(args.entries))), i32([0] * args.entries))
    row_entry = i32([e for e in range(args.entries) for _ in range(args.rows)])
    hrow = torch.randn(t, d, device=dev).bfloat16()
    off = h * ops.scan_state_floats(dk, dv)
    if args.time_mix:
        rank, n = 64, h * dk
        state = torch.zeros(args.entries, -(-(off + d) // 4) * 4, device=dev)
        w1, w2t = (torch.randn(rank, d, device=dev) * 0.02).bfloat16(), (torch.randn(rank, n, device=dev) * 0.1).bfloat16()
        mu, w0, bonus = torch.rand(5, d, device=dev), torch.zeros(n, device=dev), torch.zeros(n, device=dev)
        prepare = lambda: ops.time_mix_prepare(hrow, mu, w1, w2t, w0, state, off, row_entry, *arrays)  # noqa: E731
        rkv, decay = torch.randn(t, 3 * n, device=dev).bfloat16(), prepare()[1]
        scan = lambda: ops.time_mix_scan(rkv[:, :n], rkv[:, n: 2 * n], rkv[:, 2 * n:], decay, bonus, state, *arrays, h, dk, row_in=hrow, row_state_off=off)  # noqa: E731
    else:
        taps, channels = 4, 2 * g * dk + h * dv
        state = torch.zeros(args.entries, -(-(off + (taps - 1) * channels) // 4) * 4, device=dev)
        raw, conv = torch.randn(t, channels, device=dev).bfloat16(), torch.randn(channels, taps, device=dev) * 0.3
        w_gates, per_head = (torch.randn(2 * h, d, device=dev) * 0.02).bfloat16(), torch.zeros(h, device=dev)
        prepare = lambda: ops.delta_prepare(raw, hrow, conv, w_gates, per_head, per_head, dk ** -0.5, 1e-6, h, g, dk, dv, state, off, row_entry, *arrays)  # noqa: E731
        qk, v, numbers = prepare()
        scan = lambda: ops.delta_scan(qk, v, numbers, dk, state, *arrays, conv_in=raw, conv_taps=taps, conv_state_off=off)  # noqa: E731
    fn = prepare if args.prepare else scan
    if args.time:
        print(f"{time_in_graph(fn):.1f} us a launch")
        return 0
    for _ in range(3):
        fn()
    torch.cuda.synchronize()
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
