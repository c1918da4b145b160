"""The gated layer-list engine (Sefalorn) against the plain implementation, through prompts, portions, decoding, batches and
the backend (B200).  fp32 engines are held to 1e-4 of the logits' spread, which no wrong key, window or state passes; bf16
engines to their rounding."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from conftest import ROOT, pkg
from gated_cases import CASES, all_chosen, config, engine, light, moe, par, prompt, row_error, run_cuts, weights
from oracle import sefalorn_ref as ref

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
TOL = {F32: 1e-4, BF: 6e-2}


def blocks(n, start=0):
    return list(range(start, start + -(-n // 16)))


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", sorted(CASES))
def test_prompt_portions_and_decoding_equal_the_plain_implementation(ops, name, dtype):
    cfg = CASES[name] if dtype == F32 else all_chosen(CASES[name])
    t = weights(cfg, seed=1, gain=2.0 if dtype == F32 else 1.0)
    toks = prompt(cfg, 170)
    want, _ = ref.forward(cfg, t, toks)
    eng = engine(cfg, t, dtype)
    tol = TOL[dtype]
    for slot, cuts in enumerate(([170], [100, 2, 3, 2, 31, 32], [15] + [1] * 20 + [2, 70] + [1] * 63, [1] * 170,
                                 [33, 47, 1, 1, 2, 86], [64, 64, 42])):
        assert sum(cuts) == 170
        assert row_error(run_cuts(eng, toks, cuts, blocks(170, 3), slot), want) < tol, cuts
    # chunks inside one prompt pass
    _, lg = eng.prefill(toks, blocks(170, 20), chunk=23, want=[169, 5, 22, 23], slot=2)
    assert row_error(lg, want[[169, 5, 22, 23]]) < tol
    with pytest.raises(ValueError):
        eng.prefill(toks, blocks(170), slot=eng.num_slots)


def test_logits_hardly_depend_on_the_cut_in_bf16(ops):
    """Portions and decoding differ from one prompt pass by rounding alone, far less than bf16 differs from the equations."""
    cfg = all_chosen(CASES["wide"])
    eng = engine(cfg, weights(cfg, seed=2, gain=1.0), BF)
    toks = prompt(cfg, 300)
    whole = run_cuts(eng, toks, [300], blocks(300))
    for cuts in ([64, 236], [100] + [1] * 40 + [160], [16] * 18 + [12], [129, 2, 169]):
        assert row_error(run_cuts(eng, toks, cuts, blocks(300, 20), 1), whole) < 4e-2


def test_long_decoding_over_windows_and_states(ops):
    """Hundreds of decoded tokens: windows pass over decoded tokens, the states carry the prompt along."""
    cfg = config([par((4, 2, 64, 64, 0.2, 40), (2, 2, 32, 32, 3), moe(4, 2, 64)), light(2, 32, 32, (0.9, 0.9995), moe(4, 2, 64)),
                  par((4, 4, 32, 32, 0.3, 33), (4, 2, 32, 16, 4))], width=128)
    t = weights(cfg, seed=5, gain=2.0)
    for n in t:  # slow decays: what the first tokens wrote is still there at the end
        if n.endswith("A_log"):
            t[n] = torch.full_like(t[n], -5.0)
    toks = prompt(cfg, 380)
    want, _ = ref.forward(cfg, t, toks)
    eng = engine(cfg, t)
    assert row_error(run_cuts(eng, toks, [30] + [1] * 350, blocks(380, 1)), want) < TOL[F32]
    other, _ = ref.forward(cfg, t, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    assert row_error(other[-1:], want[-1:]) > 100 * TOL[F32]


@pytest.mark.parametrize("dtype", [F32, BF])
def test_batches_of_unequal_requests_on_reused_pages_and_slots(ops, dtype):
    """Rows of a step at different positions equal each request alone; pages and state slots given back are taken up by
    others, and what is left in them does not show."""
    cfg = CASES["odd"] if dtype == F32 else all_chosen(CASES["odd"])
    t = weights(cfg, seed=7, gain=1.0)
    eng = engine(cfg, t, dtype, num_blocks=21, max_batch=4, num_slots=4)
    be = pkg("backend").B200Backend(eng, max_new_tokens=2)
    seqs = [prompt(cfg, n, seed=n) for n in (1, 17, 48, 90)]
    extra = [prompt(cfg, 40, seed=200 + i) for i in range(4)]
    want = [ref.forward(cfg, t, s + e)[0] for s, e in zip(seqs, extra)]
    for order in ([0, 1, 2, 3], [3, 1, 0, 2]):  # the second round runs on the first one's pages and slots, in another order
        batch, rows = None, []
        for i in order:
            kv, _, n = be.prefill(seqs[i])
            batch = be.splice_into_batched(batch, kv, n)
            rows.append(i)
        with pytest.raises(MemoryError):
            be.prefill([1])
        done = {i: 0 for i in rows}
        for step in range(36):
            if step == 12:  # one request ends in the middle, the others move up
                rows.pop(1)
                batch = be.remove_row_from_cache(batch, 1)
            tok = torch.tensor([[extra[i][done[i]]] for i in rows])
            _, batch = be.decode_step_batched(tok, batch)
            lg = eng.last_logits[: len(rows)].float().cpu()
            for r, i in enumerate(rows):
                at = len(seqs[i]) + done[i]
                assert row_error(lg[r:r + 1], want[i][at:at + 1]) < 2 * TOL[dtype], (step, i)
                done[i] += 1
        while batch.rows:
            be.remove_row_from_cache(batch, 0)
        assert len(be._alloc.free) == 21 and len(be._slots.free) == 4


def test_a_decode_step_can_be_repeated(ops):
    """Running the same step again (as the warm-up of a CUDA graph does) leaves every state as one run leaves it."""
    cfg = CASES["wide"]
    t = weights(cfg, seed=3)
    toks = prompt(cfg, 60)
    want, _ = ref.forward(cfg, t, toks)
    eng = engine(cfg, t)
    eng.prefill(toks[:50], blocks(60), slot=0)
    eng.block_table[0, :4] = torch.tensor(blocks(60), dtype=torch.int32)
    for at in range(50, 60):
        for _ in range(3):
            eng.ctx_lens[0] = at
            eng.tokens[0] = toks[at]
            eng.step(1)
        assert row_error(eng.last_logits[:1], want[at:at + 1]) < TOL[F32]


@pytest.mark.parametrize("dtype", [F32, BF])
def test_merged_pass(ops, dtype):
    """A decode step that carries a prompt chunk (long and short ones) equals the plain implementation for both."""
    cfg = CASES["plain"] if dtype == F32 else all_chosen(CASES["plain"])
    t = weights(cfg, seed=9, gain=1.0)
    eng = engine(cfg, t, dtype)
    be = pkg("backend").B200Backend(eng, max_new_tokens=4)
    olds = [prompt(cfg, n, seed=n) for n in (20, 70)]
    new = prompt(cfg, 120, seed=3)
    forced = [prompt(cfg, 2, seed=50 + i) for i in range(4)] + [prompt(cfg, 3, seed=77)]
    batch = None
    for s in olds:
        kv, _, n = be.prefill(s)
        batch = be.splice_into_batched(batch, kv, n)
    partial, at = None, 0
    for step, n in enumerate((50, 2, 40, 28)):
        tok = torch.tensor(forced[step]).view(-1, 1)
        _, batch, partial, last, _ = be.decode_step_with_prefill_chunk(tok, batch, new[at:at + n], partial)
        at += n
    batch = be.splice_into_batched(batch, partial, at)
    be.decode_step_batched(torch.tensor(forced[4]).view(-1, 1), batch)
    lg = eng.last_logits[:3].float().cpu()
    eng.check_status("merged")
    full = [s + [f[i] for f in forced] for i, s in enumerate(olds)] + [new + [forced[4][2]]]
    for i, s in enumerate(full):
        want, _ = ref.forward(cfg, t, s)
        assert row_error(lg[i:i + 1], want[-1:]) < TOL[dtype], i
    if dtype == F32:
        assert last == int(ref.forward(cfg, t, new)[0][-1].argmax())


def test_greedy_generation_through_the_backend(ops, tmp_path):
    """load_model on a folder, then generate / generate_batch: token by token what the plain implementation picks (the
    logits' factor is negative in this configuration)."""
    cfg = CASES["odd"]
    t = weights(cfg, seed=11)
    pkg("checkpoint").write_safetensors(str(tmp_path / "model.safetensors"), t)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    be = pkg("backend").B200Backend(max_new_tokens=24)
    be.load_model(str(tmp_path), num_blocks=48, max_batch=3, max_pages_per_seq=16, dtype=F32)
    prompts = [prompt(cfg, n, seed=n) for n in (5, 33, 64)]

    def greedy(p, n):
        s = list(p)
        for _ in range(n):
            s.append(int(ref.forward(cfg, t, s)[0][-1].argmax()))
        return s[len(p):]

    want = [greedy(p, 8) for p in prompts]
    assert be.generate(prompts[1], 8) == want[1]
    assert be.generate_batch(prompts, [8, 4, 7]) == [want[0], want[1][:4], want[2][:7]]
    be._eos_ids = {want[0][6]}
    assert be.generate(prompts[0], 8) == want[0][:want[0].index(want[0][6])]
    assert len(be._alloc.free) == 48 and len(be._slots.free) == be.engine.num_slots


def test_graphs_equal_eager_steps_and_leave_other_states_alone(ops):
    cfg = CASES["plain"]
    t = weights(cfg, seed=13)
    toks = [prompt(cfg, n, seed=n) for n in (15, 33, 47)]
    outs = []
    for graphs in (True, False):
        eng = engine(cfg, t, BF, num_blocks=16, max_batch=4, max_pages=4, use_graphs=graphs, num_slots=6)
        for i, s in enumerate(toks):
            eng.prefill(s, blocks(64, 4 * i + 1), slot=2 * i)
            eng.block_table[i] = torch.tensor(blocks(64, 4 * i + 1), dtype=torch.int32)
            eng.ctx_lens[i] = len(s)
            eng.state_slots[i] = 2 * i
        eng.tokens[:3] = torch.tensor([3, 4, 5])
        before = [p.clone() for p in eng.states + eng.rings if p is not None]
        lg = []
        for _ in range(3):
            nxt = eng.step(3).clone()
            lg.append(eng.last_logits[:3].clone())
            eng.tokens[:3] = nxt
        eng.check_status("graphs")
        outs.append(torch.stack(lg))
        for a, b in zip(before, [p for p in eng.states + eng.rings if p is not None]):
            changed = set((a != b).flatten(1).any(1).nonzero().flatten().tolist())
            assert changed - {6} == {0, 2, 4}, changed  # the rows' own slots and the padding rows'
    assert torch.equal(outs[0], outs[1])


def test_random_weight_engine_of_a_built_in_kind(ops):
    lay = pkg("layered")
    cfg = lay.gated_config("small", 512, 256, "plp", 8, 4, 64, 32, 4, 64, 4, 8, 2, 128)
    eng = lay.LayeredEngine(cfg, 32, 4, 8)
    be = pkg("backend").B200Backend(eng, max_new_tokens=16)
    out = be.generate_batch([[1, 2, 3], list(range(40))], [8, 8])
    assert [len(o) for o in out] == [8, 8] and out == be.generate_batch([[1, 2, 3], list(range(40))], [8, 8])
    assert eng.kv_bytes_per_token() == 2 * (2 * 2 * 4 * 64)
    assert eng.state_bytes_per_sequence() == 3 * 2 * 4 * 64 * 64 * 4 + 2 * 4 * 3 * 4 * 64 * 2


def test_trace_runner_replays_a_trace(ops, tmp_path):
    """bin/trace_run as a process: portions, decode steps, two requests one after the other."""
    cfg = CASES["plain"]
    t = weights(cfg, seed=17)
    model, out = tmp_path / "m", tmp_path / "o"
    model.mkdir(), out.mkdir()
    pkg("checkpoint").write_safetensors(str(model / "model.safetensors"), t)
    (model / "config.json").write_text(json.dumps(cfg))
    a, b = prompt(cfg, 40, seed=1), prompt(cfg, 21, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [29, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[31:32], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[32:], "want": [7]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b[:1], "want": [0]}], "end": []},
             {"step": 5, "entries": [{"id": "b", "tokens": b[1:], "want": [0, 19]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "40"], input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True,
                       timeout=280)
    assert r.returncode == 0, r.stderr[-2000:]
    wa, wb = ref.forward(cfg, t, a)[0], ref.forward(cfg, t, b)[0]
    want = {0: wa[[29, 3]], 2: wa[[31]], 3: wa[[39]], 4: wb[[0]], 5: wb[[1, 20]]}
    assert sorted(os.listdir(out)) == sorted(f"{i}.f32" for i in want)
    for i, w in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert row_error(got, w) < TOL[F32], i
