"""The HTTP server with a Silupel folder (config.json and safetensors, no tokenizer), on the CPU: launcher, router, rank
process, prefix cache with state snapshots; greedy tokens against the plain restatement."""
import os
import signal
import subprocess
import sys
import time

import pytest
import requests
import torch

import silupel_plain as plain
from test_silupel import MIXED, ROOT, tokens, weights, write
from test_silupel_tp import _free_port


@pytest.mark.timeout(600)
def test_server_generates(tmp_path):
    t = weights(MIXED, 2)
    path, port = write(tmp_path / "m", MIXED, t), _free_port()
    log = open(tmp_path / "server.log", "w")
    proc = subprocess.Popen([sys.executable, "-m", "lightllm_b200.server.api_server", "--model_dir", path, "--port",
                             str(port), "--data_type", "fp32", "--max_total_token_num", "2048", "--running_max_req_size",
                             "4", "--max_req_total_len", "256", "--linear_att_hash_page_size", "32"], env=dict(os.environ, LLB_FORCE_CPU="1", PYTHONPATH=ROOT),
                            stdout=log, stderr=subprocess.STDOUT, cwd=ROOT, start_new_session=True)
    try:
        url, t0 = f"http://127.0.0.1:{port}", time.time()
        while True:
            assert proc.poll() is None and time.time() - t0 < 240, open(tmp_path / "server.log").read()[-3000:]
            try:
                if requests.get(url + "/liveness", timeout=2).status_code == 200:
                    break
            except requests.RequestException:
                time.sleep(1)
        prompt = tokens(70, 4)
        body = {"inputs": prompt, "parameters": {"max_new_tokens": 20, "do_sample": False, "return_details": True}}
        for i in range(2):
            r = requests.post(url + "/generate", json=body, timeout=60).json()
            ids = [x["id"] for x in r["tokens"]]
            lg = plain.forward(t, MIXED, prompt + ids)[69:-1]
            assert len(ids) == 20
            assert (lg.max(-1)[0] - lg.gather(1, torch.tensor(ids)[:, None])[:, 0]).max() < 1e-3
        assert r["tokens"][0]["prompt_cache_len"] > 0
    finally:
        os.killpg(proc.pid, signal.SIGTERM)
        try:
            proc.wait(timeout=20)
        except subprocess.TimeoutExpired:
            os.killpg(proc.pid, signal.SIGKILL)
