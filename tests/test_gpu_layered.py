"""The layer-list engine against the plain implementation, through prompts, portions, decoding, batches and the backend
(B200).  fp32 engines are held to 1e-4 of the logits' spread, which no wrong key, window or state passes; bf16 engines
to their rounding."""
import pytest
import torch

from conftest import pkg
from layered_cases import CASES, att, config, engine, lat, prompt, row_error, weights
from oracle import layered_ref as ref

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
TOL = {F32: 1e-4, BF: 6e-2}


def blocks(n, start=0):
    return list(range(start, start + -(-n // 16)))


def run_cuts(eng, tokens, cuts, block_ids):
    """Logits of every position, the sequence fed in portions of the given sizes; size 1 is a decode step (row 0) once the
    sequence has begun."""
    out, at = [], 0
    for n in cuts:
        if n == 1 and at:
            eng.block_table[0].zero_()
            eng.block_table[0, : len(block_ids)] = torch.tensor(block_ids, dtype=torch.int32)
            eng.ctx_lens[0] = at
            eng.tokens[0] = tokens[at]
            eng.step(1)
            out.append(eng.last_logits[:1].float().cpu())
        else:
            _, lg = eng.prefill(tokens[: at + n], block_ids, cached_tokens=at, want=list(range(at, at + n)))
            out.append(lg.float().cpu())
        at += n
    eng.check_status("test")
    return torch.cat(out)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", sorted(CASES))
def test_prompt_portions_and_decoding_equal_the_plain_implementation(ops, name, dtype):
    cfg = CASES[name]
    t = weights(cfg, seed=1, gain=2.0 if dtype == F32 else 1.0)
    toks = prompt(cfg, 170)
    want, _ = ref.layered_forward(cfg, t, toks)
    eng = engine(cfg, t, dtype)
    tol = TOL[dtype]
    for cuts in ([170], [100, 2, 3, 2, 31, 32], [15] + [1] * 20 + [2, 70] + [1] * 63, [1] * 170,
                 [33, 47, 1, 1, 2, 86]):
        assert sum(cuts) == 170
        assert row_error(run_cuts(eng, toks, cuts, blocks(170, 3)), want) < tol, cuts
    # chunks inside one prompt pass
    _, lg = eng.prefill(toks, blocks(170, 20), chunk=23, want=[169, 5, 22, 23])
    assert row_error(lg, want[[169, 5, 22, 23]]) < tol
    with pytest.raises(ValueError):
        eng.prefill(toks, blocks(170), cached_tokens=16, want=[15])


def test_logits_hardly_depend_on_the_cut_in_bf16(ops):
    """Portions, decoding and batches differ from one prompt pass by rounding alone, far less than bf16 differs from the
    equations."""
    cfg = CASES["plain"]
    eng = engine(cfg, weights(cfg, seed=2), BF)
    toks = prompt(cfg, 130)
    whole = run_cuts(eng, toks, [130], blocks(130))
    for cuts in ([64, 66], [100] + [1] * 30, [16] * 8 + [2]):
        assert row_error(run_cuts(eng, toks, cuts, blocks(130, 20)), whole) < 4e-2


def test_long_decoding_over_far_keys(ops):
    """Hundreds of decoded tokens: chunks pass over decoded tokens, a latent layer keeps reaching back to the prompt."""
    cfg = config([att(4, 2, 64, 64, 0.2, 40, 128), lat(4, 64, 64, 64, 0.4, 128), att(4, 4, 32, 32, 0.3, 33, 64)], width=128, groups=2, taps=3)
    t = weights(cfg, seed=5, gain=4.0)
    toks = prompt(cfg, 380)
    want, _ = ref.layered_forward(cfg, t, toks)
    eng = engine(cfg, t)
    got = run_cuts(eng, toks, [30] + [1] * 350, blocks(380, 1))
    assert row_error(got, want) < TOL[F32]
    # a change of one early token reaches the last position through the latent layer (so the comparison can see it)
    other, _ = ref.layered_forward(cfg, t, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
    assert row_error(other[-1:], want[-1:]) > 100 * TOL[F32]


@pytest.mark.parametrize("dtype", [F32, BF])
def test_batches_of_unequal_requests_and_reused_pages(ops, dtype):
    """Rows of a step at different positions equal each request alone; pages given back are taken up by others, and what
    is left in them (K/V, latents, convolution history) does not show."""
    cfg = CASES["odd"]
    t = weights(cfg, seed=7, gain=1.0)
    eng = engine(cfg, t, dtype, num_blocks=21, max_batch=4)
    be = pkg("backend").B200Backend(eng, max_new_tokens=2)
    seqs = [prompt(cfg, n, seed=n) for n in (1, 17, 48, 90)]
    extra = [prompt(cfg, 40, seed=200 + i) for i in range(4)]
    want = [ref.layered_forward(cfg, t, s + e)[0] for s, e in zip(seqs, extra)]
    for round_ in range(2):  # the second round runs on the first one's pages, in another order
        order = [0, 1, 2, 3] if round_ == 0 else [3, 1, 0, 2]
        batch, rows = None, []
        for i in order:
            kv, _, n = be.prefill(seqs[i])
            batch = be.splice_into_batched(batch, kv, n)
            rows.append(i)
        done = {i: 0 for i in rows}
        for step in range(36):
            if step == 12:  # one request ends in the middle, the others move up
                gone = rows.pop(1)
                batch = be.remove_row_from_cache(batch, 1)
            tok = torch.tensor([[extra[i][done[i]]] for i in rows])
            _, batch = be.decode_step_batched(tok, batch)
            lg = eng.last_logits[: len(rows)].float().cpu()
            for r, i in enumerate(rows):
                at = len(seqs[i]) + done[i]
                assert row_error(lg[r:r + 1], want[i][at:at + 1]) < 2 * TOL[dtype], (round_, step, i)
                done[i] += 1
        while batch.rows:
            be.remove_row_from_cache(batch, 0)
        assert len(be._alloc.free) == 21


def test_a_decode_step_can_be_repeated(ops):
    """Running the same step again (as the warm-up of a CUDA graph does) leaves every page as one run leaves it."""
    cfg = CASES["wide"]
    t = weights(cfg, seed=3)
    toks = prompt(cfg, 60)
    want, _ = ref.layered_forward(cfg, t, toks)
    eng = engine(cfg, t)
    eng.prefill(toks[:50], blocks(60))
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
    cfg = CASES["plain"]
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
        nxt, batch, partial, last, _ = be.decode_step_with_prefill_chunk(tok, batch, new[at:at + n], partial)
        at += n
    batch = be.splice_into_batched(batch, partial, at)
    be.decode_step_batched(torch.tensor(forced[4]).view(-1, 1), batch)
    lg = eng.last_logits[:3].float().cpu()
    eng.check_status("merged")
    full = [s + [f[i] for f in forced] for i, s in enumerate(olds)] + [new + [forced[4][2]]]
    for i, s in enumerate(full):
        want, _ = ref.layered_forward(cfg, t, s)
        assert row_error(lg[i:i + 1], want[-1:]) < TOL[dtype], i
    if dtype == F32:
        assert last == int(ref.layered_forward(cfg, t, new)[0][-1].argmax())


def test_greedy_generation_through_the_backend(ops, tmp_path):
    """load_model on a folder, then generate / generate_batch: token by token what the plain implementation picks."""
    import json
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
            s.append(int(ref.layered_forward(cfg, t, s)[0][-1].argmax()))
        return s[len(p):]

    want = [greedy(p, 10) for p in prompts]
    assert be.generate(prompts[1], 10) == want[1]
    assert be.generate_batch(prompts, [10, 4, 7]) == [want[0], want[1][:4], want[2][:7]]
    be._eos_ids = {want[0][6]}
    stop = want[0].index(want[0][6])
    assert be.generate(prompts[0], 10) == want[0][:stop]
    assert len(be._alloc.free) == 48


def test_graphs_equal_eager_steps_and_leave_other_pages_alone(ops):
    cfg = CASES["plain"]
    t = weights(cfg, seed=13)
    toks = [prompt(cfg, n, seed=n) for n in (15, 33, 47)]
    outs = []
    for graphs in (True, False):
        eng = engine(cfg, t, BF, num_blocks=16, max_batch=4, max_pages=4, use_graphs=graphs)
        for i, s in enumerate(toks):
            eng.prefill(s, blocks(64, 4 * i + 1))
            eng.block_table[i] = torch.tensor(blocks(64, 4 * i + 1), dtype=torch.int32)
            eng.ctx_lens[i] = len(s)
        eng.tokens[:3] = torch.tensor([3, 4, 5])
        before = [p.clone() for p in eng.k_pools if p is not None] + [h.clone() for h in eng.hist]
        lg = []
        for _ in range(3):
            nxt = eng.step(3).clone()
            lg.append(eng.last_logits[:3].clone())
            eng.tokens[:3] = nxt
        eng.check_status("graphs")
        outs.append(torch.stack(lg))
        for a, b in zip(before, [p for p in eng.k_pools if p is not None] + eng.hist):
            changed = (a != b).flatten(1).any(1).nonzero().flatten().tolist()
            assert set(changed) <= {1, 2, 7, 11, 12, 16}, changed  # the rows' own pages and the scratch page
    assert torch.equal(outs[0], outs[1])


def test_random_weight_engine_of_a_built_in_kind(ops):
    lay = pkg("layered")
    cfg = lay.uniform_config("small", 512, 256, 1, 4, "aal", 8, 4, 64, 64, 4, 128, 256, 7.0)
    eng = lay.LayeredEngine(cfg, 32, 4, 8)
    be = pkg("backend").B200Backend(eng, max_new_tokens=16)
    out = be.generate_batch([[1, 2, 3], list(range(40))], [8, 8])
    assert [len(o) for o in out] == [8, 8] and out == be.generate_batch([[1, 2, 3], list(range(40))], [8, 8])
    assert eng.kv_bytes_per_token() == 2 * (2 * 2 * 4 * 64 + 128 + 3 * 4 * 256 // 16)


def test_trace_runner_replays_a_trace(ops, tmp_path):
    """bin/trace_run as a process: portions, decode steps, two requests one after the other."""
    import json
    import os
    import subprocess
    import numpy as np
    from conftest import ROOT
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
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(6)]
    wa, wb = ref.layered_forward(cfg, t, a)[0], ref.layered_forward(cfg, t, b)[0]
    want = {0: wa[[29, 3]], 2: wa[[31]], 3: wa[[39]], 4: wb[[0]], 5: wb[[1, 20]]}
    assert sorted(os.listdir(out)) == sorted(f"{i}.f32" for i in want)
    for i, w in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert row_error(got, w) < TOL[F32], i
