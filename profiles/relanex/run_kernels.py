"""Profiling driver: the Relanex kernels alone on a small case (a few hundred MB on the device), so that a profiler capture
ends by itself.  Usage:

    python profiles/relanex/run_kernels.py [--tokens 4096] [--width 2048]

Runs, twice each: the matrix memory over a prompt (four chunk launches) and for one token, the sum between two bounded norms
over a prompt, and a one-token product with that sum as its way out."""
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
    P, E, H, D = a.tokens, a.width, a.width // 256, 128
    gen = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, device=dev, generator=gen)
    n = H * D
    row, ib, fb = rnd(P, 3 * n + 2 * H), torch.zeros(H, device=dev), torch.full((H,), 3.0, device=dev)
    state, aux, o = torch.zeros(H, D, D, device=dev), torch.zeros(H, D + 2, device=dev), torch.empty(P, n, device=dev)
    x, y, h = rnd(P, E), rnd(P, E), torch.empty(P, E, device=dev, dtype=torch.bfloat16)
    norms = [(torch.full((1,), 0.7, device=dev), torch.ones(E, device=dev), torch.zeros(E, device=dev)) for _ in range(2)]
    big, inp = rnd(E, 4 * E).to(torch.bfloat16), rnd(1, 4 * E).to(torch.bfloat16)
    post = seq_ops.bounded_way_out(x[:1], norms[0], 0.5, x[:1], norms[1], h[:1])

    def memory(t):
        r = row[:t]
        seq_ops.mlstm(r[:, :n], r[:, n:2 * n], r[:, 2 * n:3 * n], r[:, 3 * n:3 * n + H], r[:, 3 * n + H:], ib, fb, 15.0, D ** -0.5, state, aux, o[:t], H, D, D)

    for _ in range(2):
        memory(P)
        memory(1)
        seq_ops.bounded_sum(x, y, norms[0], 0.5, None, x, norms[1], h)
        seq_ops.gemv_multi([(inp, big, None)], post=post)
    torch.cuda.synchronize()
    print("ok")


if __name__ == "__main__":
    main()
