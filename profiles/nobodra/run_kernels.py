"""Profiling driver: the Nobodra kernels alone on a small case (a few hundred MB on the device), so that a profiler
capture ends by itself.  Usage:

    python profiles/nobodra/run_kernels.py [--tokens 4096] [--width 2048]

Runs, once each after a warm-up: the delta-rule scan with one decay per head over a prompt, the output norm + sum with and
without the experts' weighted sum, the same with the router for one token, and a product that forms its input row."""
import argparse
import sys
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parents[2]
sys.path.insert(0, str(ROOT))

from cold_compress_b200 import seq_ops  # noqa: E402


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--tokens", type=int, default=4096)
    ap.add_argument("--width", type=int, default=2048)
    a = ap.parse_args()
    dev = torch.device("cuda", 0)
    P, E, H, D, top, n = a.tokens, a.width, a.width // 256, 128, 4, 16
    gen = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, device=dev, generator=gen)
    q, k, v, beta, decay = rnd(P, H * D), rnd(P, H * D), rnd(P, H * D), rnd(P, H), rnd(P, H)
    zero, state, o = torch.zeros(H, device=dev), torch.zeros(H, D, D, device=dev), torch.empty(P, H * D, device=dev)
    x, y, rows = rnd(P, E), rnd(P, E), rnd(P * top, E)
    w, act = torch.zeros(E, device=dev), torch.empty(P, E, device=dev, dtype=torch.bfloat16)
    wts = torch.full((P, top), 0.25, device=dev)
    slot = torch.randperm(P * top, device=dev, generator=gen).to(torch.int32)
    router, bias = rnd(n, E).to(torch.bfloat16), torch.zeros(n, device=dev)
    ids, w1 = torch.empty(1, top, dtype=torch.int32, device=dev), torch.empty(1, top, device=dev)
    big, out, total = rnd(3 * E, E).to(torch.bfloat16), torch.empty(1, 3 * E, device=dev), torch.empty(1, E, device=dev)
    for _ in range(2):
        seq_ops.delta_scan(q, k, v, beta, decay, zero, zero, state, o, H, H, D, D, D ** -0.5)
        seq_ops.post_norm(x, y, w, 1e-5, 1.0, x_act=act)
        seq_ops.post_norm(x, rows, w, 1e-5, 1.0, wts=wts, slot=slot, x_act=act)
        seq_ops.post_norm_route(x[:1], y[:1], w, 1e-5, 1.0, router, bias, ids, w1, x_act=act[:1])
        seq_ops.gemv_multi([(None, big, out)], pre=seq_ops.output_norm_row(x[:1], rows[:top], w, 1e-5, 1.0, total, wts=wts[:1]))
    torch.cuda.synchronize()
    print("ok")


if __name__ == "__main__":
    main()
