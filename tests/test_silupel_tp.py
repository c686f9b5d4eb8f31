"""Silupel with tensor-parallel ranks on gloo: two ranks reproduce the plain restatement."""
import os
import socket

import pytest
import torch
import torch.multiprocessing as mp

import silupel_plain as plain
from test_silupel import chunked, close, config, dense, latent, mingru, run_portions, tokens, weights, write

CFG = config([mingru(56, dense(40)), chunked(4, 2, 24, 40, 19, 16, 0.3, 4.0, dense(72)), latent(2, 16, 8, 24, 40, 24, 0.3),
              chunked(2, 1, 16, 8, 70, 8, 0.2, 30.0)], vocab=102, loop=(1, 3, 2))


def _free_port():
    s = socket.socket()
    s.bind(("127.0.0.1", 0))
    p = s.getsockname()[1]
    s.close()
    return p


def _worker(rank, world, port, path):
    from lightllm_b200.engine.trace import TraceReplayer
    from lightllm_b200.parallel import dist as pdist

    torch.set_num_threads(2)
    ps = pdist.init_distributed(world, rank, host="127.0.0.1", port=port, backend="gloo", device=torch.device("cpu"))
    rep = TraceReplayer.open(path, "float32", 256, pstate=ps)
    toks = tokens(90, 3, 102)
    got = torch.cat([run_portions(rep, "a", toks, [90]), run_portions(rep, "b", toks, [40, 7, 1])])
    outs = rep.llm.generate([toks[:20]], {"max_new_tokens": 12, "do_sample": False})
    torch.save((got, outs[0]["token_ids"]), os.path.join(path, f"out{rank}.pt"))
    pdist.destroy()


@pytest.mark.timeout(600)
def test_two_ranks(tmp_path):
    t = weights(CFG, 6)
    path = write(tmp_path, CFG, t)
    mp.spawn(_worker, args=(2, _free_port(), path), nprocs=2, join=True)
    toks = tokens(90, 3, 102)
    want = plain.forward(t, CFG, toks)
    (g0, ids0), (g1, ids1) = (torch.load(os.path.join(path, f"out{r}.pt")) for r in range(2))
    close(g0, torch.cat([want, want]), ("cpu", "float32"))
    assert torch.equal(g0, g1) and ids0 == ids1
    lg = plain.forward(t, CFG, toks[:20] + ids0)[19:-1]
    assert (lg.max(-1)[0] - lg.gather(1, torch.tensor(ids0)[:, None])[:, 0]).max() < 1e-3
