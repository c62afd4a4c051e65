"""GPU parity of the fused row-parallel linear + all-reduce (reference layers/linear.py:133-153:
`F.linear(x, W_shard)` then `dist.all_reduce(y)`), csrc/gemm_reduce.cu through the C ABI `cvllm_gemm_allreduce`.

On one GPU a world of ONE rank runs (its own reduce-scatter rounds and all-gather stores included) against a torch fp32
GEMM within bf16 rounding.  Ranks whose kernels wait on one another are never launched side by side on one GPU: the
multi-rank protocol is tested with one process per GPU where two GPUs are there."""
import json
import socket
import subprocess
import sys
from pathlib import Path

import pytest
import torch

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent


def _option(name, value):
    from compactor_vllm import _native as N
    N.check(N.lib().cvllm_set_test_option(name.encode(), float(value)), name)


@pytest.fixture
def options():
    yield _option
    _option("grs_pairs", 0)
    _option("grs_rows_per_round", 0)


def _shards(m, n, k_total, world, dtype, seed):
    dev = torch.device("cuda", 0)
    g = torch.Generator(device=dev).manual_seed(seed)
    x = (torch.randn((m, k_total), generator=g, device=dev) * 0.5).to(dtype)
    w = (torch.randn((n, k_total), generator=g, device=dev) * 0.05).to(dtype)
    per = k_total // world
    return x, w, [(x[:, r * per:(r + 1) * per], w[:, r * per:(r + 1) * per]) for r in range(world)]


def _run_alone(m, n, shard, calls=1):
    """y of a world of one rank after `calls` back-to-back calls (the flags must carry over)."""
    from compactor_vllm.layers.linear import PeerGemmAllReduce
    (rank,), free = PeerGemmAllReduce.virtual_ranks(1, m, n, torch.device("cuda", 0))
    try:
        for _ in range(calls):
            out = rank.linear(*shard)
        return out.clone()
    finally:
        free()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float16])
@pytest.mark.parametrize("m,n,k", [(256, 256, 64), (1000, 512, 192), (4096, 8192, 1024), (300, 264, 72)])
def test_world1_matches_fp32_gemm(options, dtype, m, n, k):
    x, w, shards = _shards(m, n, k, 1, dtype, seed=m + n + k)
    y = _run_alone(m, n, shards[0], calls=3)
    ref = x.float() @ w.float().t()
    err = (y.float() - ref).abs()
    bound = ref.abs() * 2.0 ** (-8 if dtype == torch.bfloat16 else -11) + 1e-3
    assert bool((err <= bound).all()), float((err - bound).max())
    # and the library GEMM rounds the same fp32 sums to (nearly always) the same 16-bit values
    lib = torch.mm(x, w.t())
    assert float((y != lib).float().mean()) < 2e-2


def test_rounds_and_changing_shapes_share_one_buffer(options):
    """Several reduce rounds (rows_per_round 256), then smaller M on the same buffers: the counters are reset per call
    and the layout depends on the call's M only."""
    from compactor_vllm.layers.linear import PeerGemmAllReduce
    dev, dtype, n, k = torch.device("cuda", 0), torch.bfloat16, 512, 256
    options("grs_rows_per_round", 256)
    (rank,), free = PeerGemmAllReduce.virtual_ranks(1, 4096, n, dev)
    try:
        for m in (4096, 640, 4096, 1):
            x, w, shards = _shards(m, n, k, 1, dtype, seed=m)
            y = rank.linear(*shards[0]).clone()
            ref = x.float() @ w.float().t()
            assert float((y.float() - ref).abs().max()) <= float(ref.abs().max()) * 2.0 ** -6 + 1e-3
    finally:
        free()


def test_refuses_unaligned_shapes(options):
    from compactor_vllm import _native as N
    from compactor_vllm.layers.linear import PeerGemmAllReduce
    dev = torch.device("cuda", 0)
    ranks, free = PeerGemmAllReduce.virtual_ranks(1, 256, 256, dev)
    try:
        x = torch.zeros((256, 60), dtype=torch.bfloat16, device=dev)
        w = torch.zeros((256, 60), dtype=torch.bfloat16, device=dev)
        assert not ranks[0].supports(x, w)
        with pytest.raises((AssertionError, N.NativeLibraryError)):
            ranks[0].linear(x, w)
    finally:
        free()


@pytest.mark.skipif(torch.cuda.device_count() < 2, reason="needs two GPUs (NVLink peer memory between processes)")
@pytest.mark.parametrize("rows", [4096, 1000])
def test_two_processes_two_gpus(rows):
    """One process per GPU, buffers shared by cudaIpc handles: every rank holds the same bits, and they are the fp32
    rank-order sum of the ranks' own cuBLAS partials (tools/gemm_reduce_bench.py does the checks on the devices)."""
    with socket.socket() as sk:
        sk.bind(("127.0.0.1", 0))
        port = sk.getsockname()[1]
    cmd = [sys.executable, "-m", "torch.distributed.run", "--nnodes=1", "--nproc-per-node", "2", "--master-addr",
           "127.0.0.1", "--master-port", str(port), str(ROOT / "tools" / "gemm_reduce_bench.py"), str(rows)]
    run = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    line = [ln for ln in run.stdout.splitlines() if ln.startswith("{")][-1]
    res = json.loads(line)
    assert res["identical_on_all_ranks"] is True
    assert res["frac_equal_rank_order_sum_of_cublas_partials"] == 1.0
    assert res["max_abs_diff_vs_nccl"] <= res["max_abs"] * 2.0 ** -7
