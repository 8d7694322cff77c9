"""``bin/trace_run``: token ids replayed through the engine step by step, logits to files (CPU form of the operators; the GPU
run of the same schedule is marked)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import fetelorn_oracle as O
import lufivik_oracle as LO
import ruburax_oracle as RO
import sotazen_oracle as SO
import test_lufivik as L
import test_ruburax as R
import test_sotazen as S
from test_fetelorn import bf16_exact, build, config, parallel, retention, toks
from b200fw.model import ModelConfig, ParallelTransformerModel, registry

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CFG = config(36, 51, [parallel(2, 1, 16, 8, 20, 12, 2, 1, 16, 24, 5, ff=16), retention(2, 8, 16, 4, ff=16)])

SOTAZEN = S.config(36, 51, [S.latent(2, 16, 8, 12, 24, ff=16), S.lightning(2, 8, 16, ff=None), S.differential(2, 1, 16, 8, 19, 4, ff=16)])
RUBURAX = R.config(36, 51, [R.rglru(24, 2, 3, ff=R.dense(16)), R.attention(2, 1, 16, 8, R.rot(8, 400.0, (4.0, 1.0, 2.0, 20))),
                            R.parallel(R.att(2, 1, 8, 8, R.rot(8)), 2, 8, 12, 6.0, 0.7, 1.2, ff=R.moe(6, 2, 12, (3, 2), 8)),
                            R.attention(4, 1, 16, 8, R.rot(8, 400.0, (4.0, 1.0, 2.0, 20)), kv_from=1, ff=R.dense(16))])
# every expert is chosen: no position rests on a close choice
LUFIVIK = L.config(36, 51, [L.latent(2, 16, 8, 12, 20, 24, 11, L.moe(6, 6, 12)), L.latent(3, 8, 4, 10, 12, 16, 7), L.latent(1, 8, 8, 8, 8, 8, 30, L.moe(5, 5, 8))],
                   loop=(1, 3, 2))
MODELS = {"Fetelorn": (CFG, O, build), "Sotazen": (SOTAZEN, SO, S.build), "Ruburax": (RUBURAX, RO, R.build), "Lufivik": (LUFIVIK, LO, L.build)}


def replay(model_dir, out, steps, max_tokens, device, dtype="float32"):
    p = subprocess.Popen([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(model_dir), "--dtype", dtype,
                          "--out", str(out), "--max-tokens", str(max_tokens), "--device", device],
                         stdin=subprocess.PIPE, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True)
    done = []
    for s in steps:
        p.stdin.write(json.dumps(s) + "\n")
        p.stdin.flush()
        while True:
            line = p.stdout.readline()
            if not line:
                return p.wait(), done, p.stderr.read()
            if line.startswith("done "):
                done.append(int(line.split()[1]))
                break
    p.stdin.close()
    return p.wait(), done, p.stderr.read()


def schedule(seqs, cuts_by_seq):
    """Steps in which sequence i runs its k-th portion at step k + i (later ones join, earlier ones end)."""
    steps, at = [], [0] * len(seqs)
    n = max(len(c) + i for i, c in enumerate(cuts_by_seq))
    for k in range(n):
        entries, end = [], []
        for i, cuts in enumerate(cuts_by_seq):
            if 0 <= k - i < len(cuts):
                c = cuts[k - i]
                entries.append({"id": f"s{i}", "tokens": seqs[i][at[i]:at[i] + c], "want": list(range(0, c, 2))})
                at[i] += c
                if at[i] == len(seqs[i]):
                    end.append(f"s{i}")
        if k == 1:
            for e in entries:
                e["want"] = []
        steps.append({"step": 10 + k, "entries": entries, "end": end})
    return steps


@pytest.mark.parametrize("device,dtype", [("cpu", "float32"), pytest.param("cuda", "float32", marks=pytest.mark.gpu),
                                          pytest.param("cuda", "bfloat16", marks=pytest.mark.gpu)])
@pytest.mark.parametrize("design", list(MODELS))
def test_replay(tmp_path, design, device, dtype):
    cfg, oracle, make = MODELS[design]
    w = bf16_exact(oracle.random_weights(cfg, 4))
    registry.save_checkpoint(make(cfg, w, ("cpu", torch.float32)), str(tmp_path / "m"))
    lens = [33, 18, 25, 40, 9]
    seqs = [toks(n, 51, n) for n in lens]
    cuts = [[20, 1, 12], [17, 1], [2, 3, 20], [39, 1], [9]]
    steps = schedule(seqs, cuts)
    # three requests are live at a time at most: the pool is made for that, not for all five
    rc, done, err = replay(tmp_path / "m", tmp_path / "o", steps, 192, device, dtype)
    assert rc == 0 and done == [s["step"] for s in steps], err[-2000:]
    want = [oracle.forward(cfg, w, s).float().numpy() for s in seqs]
    at = {}
    for s in steps:
        rows = []
        for e in s["entries"]:
            i, a = int(e["id"][1:]), at.get(e["id"], 0)
            rows += [want[i][a + k] for k in e["want"]]
            at[e["id"]] = a + len(e["tokens"])
        path = tmp_path / "o" / f"{s['step']}.f32"
        assert path.exists() == bool(rows)
        if rows:
            got = np.fromfile(path, dtype="<f4").reshape(len(rows), 51)
            np.testing.assert_allclose(got, np.stack(rows), atol=2e-3 if dtype == "float32" else 0.4)


def test_replay_dense_model(tmp_path):
    mc = ModelConfig(vocab_size=64, hidden_size=32, num_layers=2, num_heads=4, num_kv_heads=2, head_dim=8, intermediate_size=48,
                     max_position_embeddings=256, tie_word_embeddings=True)
    m = ParallelTransformerModel(mc)
    m.init_weights(0, std=0.3)
    registry.save_checkpoint(m, str(tmp_path / "m"))
    seq = toks(30, 64)
    steps = schedule([seq], [[11, 1, 2, 16]])
    for s in steps:
        s["entries"][0]["want"] = list(range(len(s["entries"][0]["tokens"])))
    rc, done, err = replay(tmp_path / "m", tmp_path / "o", steps, 32, "cpu")
    assert rc == 0, err[-2000:]
    got = np.concatenate([np.fromfile(tmp_path / "o" / f"{s['step']}.f32", dtype="<f4").reshape(-1, 64) for s in steps])
    with torch.no_grad():
        np.testing.assert_allclose(got, m(torch.tensor([seq]))[0].numpy(), atol=1e-3)


def test_replay_reports_what_does_not_fit(tmp_path):
    w = bf16_exact(O.random_weights(CFG, 4))
    registry.save_checkpoint(build(CFG, w, ("cpu", torch.float32)), str(tmp_path / "m"))
    rc, done, err = replay(tmp_path / "m", tmp_path / "o",
                           [{"step": 0, "entries": [{"id": "a", "tokens": toks(40, 51), "want": []}], "end": []}], 32, "cpu")
    assert rc not in (0, 3) and done == [] and "exhausted" in err
    (tmp_path / "m" / "config.json").write_text(json.dumps({"architecture": "Unheard"}))
    rc, _, err = replay(tmp_path / "m", tmp_path / "o", [], 32, "cpu")
    assert rc not in (0, 3) and "unknown architecture" in err
