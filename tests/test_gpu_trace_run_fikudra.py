"""bin/trace_run end to end on a Fikudra model from files: a config.json and a model.safetensors written by the test
(every tensor name of the design: both mixers, a layer that reads another layer's keys, routed experts with and without a
shared one, a layer without a feed-forward, a decay projection whose inner size only the checkpoint gives), a schedule on
standard input with portions beside single tokens and requests that end and give their pages and state slots to later
ones, logits compared with the CPU oracle."""
import json
import os
import subprocess
from pathlib import Path

import numpy as np
import pytest
import torch

from fikudra_common import attn, clean, gla, model_cfg, moe, random_checkpoint, write_checkpoint

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent


def default_config():
    return model_cfg([
        (gla(2, 14, 10, 12.0, 7), moe(4, 2, 10, 12, 2, 1, 2.0)),
        (attn(3, 1, 12, 8, rot=10, base=90.0, factor=3.0, scale=0.4), moe(3, 1, 14, 0, 0, scale=0.8)),
        (gla(1, 18, 6, 5.0, 3), None),
        (attn(3, 1, 12, 8, rot=10, base=90.0, factor=3.0, scale=0.6, kv_from=1), moe(6, 3, 8, 10, 3, 2, 1.3)),
    ], vocab=50, width=36, eps=1e-6, streams=2, scale=7.0, buckets=41, mul_prev=13, mul_cur=5)


@pytest.mark.parametrize("dtype,tol", [("float32", 3e-5), ("bfloat16", 8e-2)])
def test_trace_run_replays_a_schedule_from_files(tmp_path, dtype, tol):
    from oracle import fikudra as O

    cfg = default_config()
    tensors = random_checkpoint(cfg, seed=3)
    write_checkpoint(tmp_path / "model", cfg, tensors)
    c = clean(cfg)
    g = torch.Generator().manual_seed(5)
    reqs = {k: torch.randint(0, 50, (n,), generator=g).tolist() for k, n in (("a", 40), ("b", 17), ("c", 5), ("d", 70), ("e", 1))}
    want = {k: O.forward(c, tensors, v) for k, v in reqs.items()}
    # pool: 3 pages of 64 tokens; a, b, c live together, then d (2 pages) beside b after a and c have ended, then e
    plan = [[("a", 16), ("b", 2)], [("a", 1), ("b", 1)], [("a", 23), ("c", 5)], [("b", 1)], [("b", 13), ("d", 33)],
            [("d", 1)], [("d", 36), ("e", 1)]]
    at = {k: 0 for k in reqs}
    lines, expect = [], []
    for n, step in enumerate(plan):
        entries, end, rows = [], [], []
        for k, cnt in step:
            lo, hi = at[k], at[k] + cnt
            entries.append({"id": "req-" + k, "tokens": reqs[k][lo:hi], "want": list(range(cnt))})
            rows.append(want[k][lo:hi])
            at[k] = hi
            if hi == len(reqs[k]):
                end.append("req-" + k)
        lines.append(json.dumps({"step": n, "entries": entries, "end": end}))
        expect.append(torch.cat(rows))
    assert all(at[k] == len(v) for k, v in reqs.items())
    out = tmp_path / "out"
    env = dict(os.environ, HOME=str(tmp_path), TMPDIR=str(tmp_path))
    res = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "model"), "--dtype", dtype, "--out",
                          str(out), "--max-tokens", "192"], input="\n".join(lines) + "\n", capture_output=True, text=True,
                         env=env, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done ")] == [f"done {n}" for n in range(len(plan))]
    scale = torch.cat(list(want.values())).std()
    errs = []
    for n, exp in enumerate(expect):
        got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(exp.shape)).double()
        d = (got - exp) - (got - exp).mean(-1, keepdim=True)
        errs.append(d.pow(2).mean(-1).sqrt() / scale)
    errs = torch.cat(errs)
    # bfloat16: a token whose routing is a close call may take another expert than in exact arithmetic
    assert (errs > tol).sum() <= (0 if dtype == "float32" else 8) and errs.median() < tol / 3
