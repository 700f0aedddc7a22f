"""Dinutar on the GPU against the plain implementation (tests/plain/dinutar_plain.py): every mechanism's kernels alone,
then whole models through the step function, the cache and state manager, the generation loop, the command line and
replay, in both precisions.

Schedules: whole prompts; a prompt, then token by token across page and tile borders; decoding from the first token;
prompts in portions down to two tokens; steps cut into chunks; batches of unequal requests; slots, pages and state used
again; long decoding.  Mechanisms: the embedding with its second table (rows picked by the previous token, which comes
from the step or from state), the norm after the sum, the stretched rotation with its magnitude on queries, keys and the
shared key part, the retention by single tokens, by tiles and by the walk over tokens with keys far away that decide a
read-out, the latent attention with a score that towers at the first key, at page borders and at the query itself and a
larger one right after the query, layers that read another layer's rows, the squared-relu product in all its kernels.
"""
from __future__ import annotations

import json
import os
import subprocess
import sys
import tempfile

import numpy as np
import pytest
import torch

from tests import dinutar_cases as cases
from tests.plain import dinutar_plain as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DTYPES = ["float32", "bfloat16"]
WHOLE = ["a", "b", "c", "d"]
ALONE = ["retention", "latent_attention"]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name: str, seed: int = 11):
        key = (name, seed)
        if key not in made:
            cfg = cases.CONFIGS[name]()
            w = cases.random_weights(cfg, seed)
            made[key] = (cases.write_folder(cfg, w, str(tmp_path_factory.mktemp(f"dinutar-{name}-{seed}"))), cfg, w)
        return made[key]
    return get


_plain_logits = {}


def plain_logits(cfg, w, ids):
    key = (id(w), tuple(ids))
    if key not in _plain_logits:
        _plain_logits[key] = (w, plain.forward(cfg, w, ids))       # w is kept: its id stays taken
    return _plain_logits[key][1]


def make_stepper(folder, dtype, max_tokens=64 * 60, chunk_tokens=2048, n_slots=None):
    from cpmcu_b200.cache import Cache
    from cpmcu_b200.engine.step import Stepper
    from cpmcu_b200.loading import load_model

    _, _, model = load_model(folder, dtype)
    cache = Cache(model.cache_needs(), max_tokens=max_tokens, dtype=DT[dtype], device="cuda:0", n_slots=n_slots,
                  max_step_tokens=chunk_tokens)
    return Stepper(model, cache, chunk_tokens=chunk_tokens)


def run_portions(stepper, requests, portions):
    """Feeds request r its tokens in portions[r] (sizes that add up to its length), step k taking the k-th portion of
    every request that still has one, all as one batch.  Returns the logits of every position per request."""
    from cpmcu_b200.engine.step import SequenceStep

    slots = stepper.open(len(requests))
    at = [0] * len(requests)
    out = [[] for _ in requests]
    for k in range(max(len(p) for p in portions)):
        batch, who = [], []
        for r, ids in enumerate(requests):
            if k < len(portions[r]):
                n = portions[r][k]
                batch.append(SequenceStep(slots[r], ids[at[r]:at[r] + n], list(range(n))))
                who.append((r, n))
                at[r] += n
        logits = stepper.step(batch)
        o = 0
        for r, n in who:
            out[r].append(logits[o:o + n].clone())
            o += n
        for r, _ in who:
            if at[r] == len(requests[r]) and slots[r] is not None:
                stepper.close(slots[r])
                slots[r] = None
    stepper.ops.raise_on_kernel_error()
    stepper.cache.check_consistent()
    return [torch.cat(x) for x in out]


def check(got, want, dtype, what=""):
    e = cases.row_errors(got, want)
    worst = int(e.argmax())
    assert float(e.max()) <= cases.TOL[dtype], f"{what}: row {worst} differs by {float(e.max()):.3e} (allowed {cases.TOL[dtype]})"
    if e.numel() >= 20:
        assert float(e.median()) <= cases.MEDIAN_TOL[dtype], f"{what}: the median row differs by {float(e.median()):.3e}"


def run_and_check(stepper, cfg, w, requests, portions, dtype, what):
    got = run_portions(stepper, requests, portions)
    for r, ids in enumerate(requests):
        check(got[r], plain_logits(cfg, w, ids), dtype, f"{what}, request {r}")


# ---------------------------------------------------------------------------
# whole models, and models of one mechanism alone
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", WHOLE + ALONE)
def test_whole_prompt_and_first_tokens(folders, name, dtype):
    folder, cfg, w = folders(name)
    st = make_stepper(folder, dtype)
    for n in (200, 1, 2, 15, 16, 64, 67):
        ids = cases.random_ids(cfg["vocab"], n, 40 + n)
        run_and_check(st, cfg, w, [ids], [[n]], dtype, f"whole prompt of {n}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", WHOLE + ALONE)
def test_prompt_then_token_by_token_across_pages(folders, name, dtype):
    folder, cfg, w = folders(name)
    ids = cases.random_ids(cfg["vocab"], 200, 3)
    run_and_check(make_stepper(folder, dtype), cfg, w, [ids], [[45] + [1] * 155], dtype, "prompt then decode")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", WHOLE)
def test_token_by_token_from_the_first_token(folders, name, dtype):
    folder, cfg, w = folders(name)
    ids = cases.random_ids(cfg["vocab"], 80, 4)
    run_and_check(make_stepper(folder, dtype), cfg, w, [ids], [[1] * 80], dtype, "decode from the start")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,cuts", [("a", [2] * 40 + [70]), ("a", [63, 1, 64, 2, 20]), ("c", [33, 32, 31, 3, 51]), ("d", [64, 64, 22]),
                                       ("c", [149, 1]), ("d", [1, 2, 147]), ("b", [20, 19, 2, 36, 73]), ("d", [65, 2, 16, 67]),
                                       ("retention", [15, 16, 17, 2, 100]), ("latent_attention", [65, 2, 83])])
def test_portions_of_a_prompt(folders, dtype, name, cuts):
    folder, cfg, w = folders(name)
    ids = cases.random_ids(cfg["vocab"], 150, 6)
    run_and_check(make_stepper(folder, dtype), cfg, w, [ids], [cuts], dtype, f"portions {cuts[:4]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", WHOLE)
def test_step_function_cuts_long_steps_into_chunks(folders, name, dtype):
    folder, cfg, w = folders(name)
    reqs = [cases.random_ids(cfg["vocab"], n, 70 + n) for n in (130, 50, 3)]
    st = make_stepper(folder, dtype, chunk_tokens=48)
    run_and_check(st, cfg, w, reqs, [[130], [50], [3]], dtype, "chunks of 48")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", WHOLE + ALONE)
def test_batches_of_unequal_requests(folders, name, dtype):
    """Among them a request of one token and one whose first portion is a page: the first tokens of sequences stand in the
    middle of the batch, where a lost previous token or a state of the neighbour would show."""
    folder, cfg, w = folders(name)
    reqs = [cases.random_ids(cfg["vocab"], n, 90 + n) for n in (100, 31, 66, 5, 1, 140)]
    portions = [[70] + [1] * 30, [21] + [1] * 10, [64, 2], [2] + [1] * 3, [1], [129, 11]]
    run_and_check(make_stepper(folder, dtype), cfg, w, reqs, portions, dtype, "batch")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_batch_of_many_requests(folders, dtype):
    """More sequences than the products' smallest row counts take, decoded together and leaving one by one."""
    folder, cfg, w = folders("a")
    lengths = [3 + 2 * (i % 9) for i in range(40)]
    reqs = [cases.random_ids(cfg["vocab"], n, 300 + i) for i, n in enumerate(lengths)]
    run_and_check(make_stepper(folder, dtype, max_tokens=64 * 100), cfg, w, reqs, [[2] + [1] * (n - 2) for n in lengths], dtype, "many")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "d"])
def test_slots_pages_and_state_are_used_again(folders, name, dtype):
    """A cache of two slots and few pages serves nine requests one after another and in pairs: every slot, every page,
    every matrix state and every previous token are used again with what the last sequence left in them."""
    folder, cfg, w = folders(name)
    st = make_stepper(folder, dtype, max_tokens=64 * 6, n_slots=2)
    for round_no in range(3):
        reqs = [cases.random_ids(cfg["vocab"], n, 100 + 7 * round_no + n) for n in (130, 9, 70)]
        run_and_check(st, cfg, w, reqs[:2], [[100] + [1] * 30, [9]], dtype, "reused slots")
        run_and_check(st, cfg, w, reqs[2:], [[3, 67]], dtype, "reused slots")
        assert st.cache.slots.n_held == 0 and all(g.pages.n_held == 0 for g in st.cache.groups)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["b", "c"])
def test_long_decoding(folders, name, dtype):
    folder, cfg, w = folders(name)
    ids = cases.random_ids(cfg["vocab"], 330, 5)
    run_and_check(make_stepper(folder, dtype, max_tokens=64 * 8), cfg, w, [ids], [[10] + [1] * 320], dtype, "long decode")


@pytest.mark.parametrize("dtype", DTYPES)
def test_logits_do_not_depend_on_the_cut_the_batch_or_the_slots(folders, dtype):
    """The engine against itself, closer than against the plain implementation: one request whole, in portions, decoded,
    beside others, and in a slot and pages that others have used."""
    folder, cfg, w = folders("a")
    ids = cases.random_ids(cfg["vocab"], 150, 8)
    others = [cases.random_ids(cfg["vocab"], n, 20 + n) for n in (33, 100)]
    st = make_stepper(folder, dtype, max_tokens=64 * 10, n_slots=3)
    whole = run_portions(st, [ids], [[150]])[0]
    for reqs, portions in (([ids], [[70, 2, 78]]), ([ids], [[149, 1]]), ([others[0], ids], [[33], [150]]),
                           ([others[1], ids, others[0]], [[64] + [1] * 36, [120] + [1] * 30, [1] * 33])):
        got = run_portions(st, reqs, portions)[reqs.index(ids)]
        e = cases.row_errors(got, whole)
        assert float(e.max()) <= (2e-5 if dtype == "float32" else cases.TOL[dtype]), (portions, float(e.max()))
        assert float(e.median()) <= (5e-6 if dtype == "float32" else 1e-2)


# ---------------------------------------------------------------------------
# through the library's own entry points
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("graph", [False, True])
@pytest.mark.parametrize("name", ["a", "c"])
def test_greedy_generation_through_llm(folders, name, graph):
    """fp32: the tokens of the plain implementation for a batch of unequal prompts (a comparison stops where the two
    best logits nearly tie), twice in a row so that slots and state are used again; prompts go through chunks of 16
    tokens, which the graph variant records and replays, and decoding through the decode runner."""
    from cpmcu_b200 import LLM

    folder, cfg, w = folders(name)
    llm = LLM(folder, dtype="float32", cuda_graph=graph, max_tokens=64 * 16, chunk_length=16)
    prompts = [cases.random_ids(cfg["vocab"], n, 60 + n) for n in (41, 1, 3, 70)]
    want = [plain.greedy(cfg, w, p, 10) for p in prompts]
    for _ in range(2):
        res = llm.generate_batch(prompts, generation_length=10)
        compared = 0
        for r, (tokens, gaps) in zip(res, want):
            firm = next((i for i, g in enumerate(gaps) if g < 1e-3), len(tokens))
            assert r.tokens[:firm] == tokens[:firm]
            compared += firm
        assert compared >= 25


@pytest.mark.parametrize("graph", [False, True])
def test_bfloat16_generation(folders, graph):
    """The tokens of the plain implementation up to the first choice between two logits closer than rounding moves them."""
    from cpmcu_b200 import LLM

    folder, cfg, w = folders("d")
    prompts = [cases.random_ids(cfg["vocab"], n, 80 + n) for n in (33, 90, 64, 2, 17)]
    llm = LLM(folder, dtype="bfloat16", cuda_graph=graph, max_tokens=64 * 16, chunk_length=32)
    compared = 0
    for prompt, r in zip(prompts, llm.generate_batch(prompts, generation_length=10)):
        tokens, gaps = plain.greedy(cfg, w, prompt, 10)
        firm = next((i for i, g in enumerate(gaps) if g < 0.6), len(tokens))
        assert r.tokens[:firm] == tokens[:firm]
        compared += firm
    assert compared >= 15


def test_command_line_and_replay(folders, tmp_path):
    folder, cfg, w = folders("c")
    ids = cases.random_ids(cfg["vocab"], 30, 9)
    env = dict(os.environ, PYTHONPATH=ROOT)
    p = subprocess.run([sys.executable, "-m", "cpmcu_b200.cli", "--model-path", folder, "--dtype", "float32",
                        "--prompt-ids", ",".join(map(str, ids)), "--num-generate", "6", "--max-tokens", "512"],
                       capture_output=True, text=True, env=env, cwd=ROOT, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    tokens, gaps = plain.greedy(cfg, w, ids, 6)
    firm = next((i for i, g in enumerate(gaps) if g < 1e-3), 6)
    assert firm >= 1 and " ".join(map(str, tokens[:firm])) in p.stdout.replace(",", " ").replace("  ", " ")
    out = tmp_path / "out"
    steps = [{"step": 0, "entries": [{"id": "r", "tokens": ids[:17], "want": [0, 16]}], "end": []},
             {"step": 1, "entries": [{"id": "r", "tokens": ids[17:29], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "r", "tokens": ids[29:], "want": [0]}], "end": ["r"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, env=env, cwd=ROOT, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = plain.forward(cfg, w, ids)
    got0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4")).view(2, -1)
    got2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4")).view(1, -1)
    assert not (out / "1.f32").exists()
    check(got0, want[[0, 16]], "float32", "replay")
    check(got2, want[[29]], "float32", "replay")


# ---------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------

def _ctx(q_lens, starts, slots):
    """A step's description on the device for sequences that bring ``q_lens`` tokens from positions ``starts``."""
    from cpmcu_b200.parts.base import QUERY_TILE_TOKENS, StepContext

    i32 = dict(dtype=torch.int32, device="cuda")
    pos = torch.cat([torch.arange(s, s + n) for n, s in zip(q_lens, starts)]).to(**i32)
    seq = torch.cat([torch.full((n,), i) for i, n in enumerate(q_lens)]).to(**i32)
    cu = torch.tensor([0] + list(np.cumsum(q_lens)), **i32)
    kv = [s + n for n, s in zip(q_lens, starts)]
    ctx = StepContext(n_tokens=sum(q_lens), n_seqs=len(q_lens), is_decode=all(n == 1 for n in q_lens), captured=False,
                      q_lens=list(q_lens), kv_lens=kv, slots=list(slots), max_q_len=max(q_lens), max_kv_len=max(kv),
                      token_ids=torch.zeros(sum(q_lens), **i32), positions=pos, token_seq=seq, cu_q=cu,
                      kv_len_dev=torch.tensor(kv, **i32), slot_dev=torch.tensor(list(slots), **i32))
    ts = [i for i, n in enumerate(q_lens) for _ in range(0, n, QUERY_TILE_TOKENS)]
    trow = [r for n in q_lens for r in range(0, n, QUERY_TILE_TOKENS)]
    ctx.q_tiles = (torch.tensor(ts, **i32), torch.tensor(trow, **i32), len(ts))
    return ctx


def _close(got, want, dtype, tol32=3e-5, tol16=2e-2):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape, (got.shape, want.shape)
    err = float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))
    assert err <= (tol32 if dtype == "float32" else tol16), err


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,n,scaled", [(64, 5, True), (100, 70, True), (99, 3, True), (2048, 17, True), (4100, 2, True), (128, 9, False)])
def test_norm_after_the_sum(dtype, hidden, n, scaled):
    from cpmcu_b200.ops.ops import Ops

    ops = Ops(DT[dtype])
    g = torch.Generator().manual_seed(hidden)
    x, a = torch.randn(n, hidden, generator=g) * 2, (torch.randn(n, hidden, generator=g) * 3).to(DT[dtype])
    x[0] *= 1e-3
    a[0] *= 1e-3                                                 # a row where eps counts
    ls = torch.randn(hidden, generator=g) if scaled else torch.ones(hidden)
    wn = 1 + 0.3 * torch.randn(hidden, generator=g)
    w = {"ls1": ls.double(), "norm1": wn.double()}
    want = plain.joined(x.double(), a.double(), w, "", 1, 2.75, 1e-5)
    xd = x.cuda()
    y = ops.post_norm(xd, a.cuda(), 2.75, ls.cuda() if scaled else None, wn.cuda(), 1e-5)
    for row in range(n):
        _close(xd[row], want[row], "float32", tol32=3e-6)        # the stream is 32-bit in both precisions
    _close(y, want, dtype, tol32=3e-6, tol16=5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,bigram,scale,norm", [(96, (101, 37, 11), 0.7, True), (100, (1, 2_000_000_011, 1_999_999_973), 1.5, True),
                                                      (99, (40, 1, 0), 1.0, True), (64, None, 0.3, True), (64, (7, 3, 5), 2.0, False)])
def test_embedding_with_a_table_of_token_pairs(dtype, hidden, bigram, scale, norm):
    """Three sequences whose tokens come in portions (single tokens, two, many); the previous tokens start as rubbish in
    their slots, so a first token that read them would show."""
    from cpmcu_b200.ops.ops import Ops

    ops = Ops(DT[dtype])
    g = torch.Generator().manual_seed(hidden)
    V, eps = 61, 1e-4
    table = torch.randn(V, hidden, generator=g).to(DT[dtype])
    cfg = {"embedding": {"scale": scale}, "norm": {"eps": eps}}
    w = {"embed": table.double(), "embed.norm": (1 + 0.3 * torch.randn(hidden, generator=g)).double()}
    second, mul_prev, mul_cur = None, 0, 0
    if bigram:
        buckets, mul_prev, mul_cur = bigram
        second = torch.randn(buckets + 1, hidden, generator=g).to(DT[dtype])
        cfg["embedding"]["bigram"] = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
        w["bigram"] = second.double()
    seqs = [cases.random_ids(V, n, n) for n in (40, 1, 17)]
    wants = []
    for ids in seqs:
        if norm:
            wants.append(plain.embedding(cfg, w, ids))
        else:
            wants.append(w["embed"][ids] * scale + (w["bigram"][plain.bigram_rows(ids, cfg["embedding"]["bigram"])] if bigram else 0))
    state = torch.full((5,), 33, dtype=torch.int32, device="cuda")
    slots, done = [4, 0, 2], [0, 0, 0]
    got = [[], [], []]
    for step in ([20, 1, 2], [1, 0, 1], [2, 0, 14], [17, 0, 0]):
        live = [i for i in range(3) if step[i]]
        ctx = _ctx([step[i] for i in live], [done[i] for i in live], [slots[i] for i in live])
        ctx.token_ids = torch.tensor([t for i in live for t in seqs[i][done[i]:done[i] + step[i]]], dtype=torch.int32, device="cuda")
        x, y = ops.embed_norm(ctx, table.cuda(), scale, second.cuda() if bigram else None, mul_prev, mul_cur, state,
                              w["embed.norm"].float().cuda() if norm else None, eps)
        assert torch.equal(y.float(), x.to(DT[dtype]).float())
        at = 0
        for i in live:
            got[i].append(x[at:at + step[i]])
            at += step[i]
            done[i] += step[i]
    for i in range(3):
        _close(torch.cat(got[i]), wants[i], "float32", tol32=3e-6)
    if bigram:
        assert state.tolist() == [seqs[1][-1], 33, seqs[2][-1], 33, seqs[0][-1]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim,dr,R,scaling", [(3, 16, 8, 24, (4.0, 64, 16.0, 1.0)), (5, 13, 6, 19, (1.5, 10, 3.0, 2.0)), (2, 32, 0, 40, None),
                                                (18, 64, 64, 512, None), (1, 128, 32, 96, (16.0, 4096, 32.0, 1.0))])
def test_latent_preparation_turns_queries_and_the_shared_key_part(dtype, H, dim, dr, R, scaling):
    """Prepared queries and cached rows of two sequences (one of them after a history) against the plain rotation with its
    magnitude and the plain norm; then the forms for queries with a latent, with a magnitude."""
    from cpmcu_b200.cache import Cache
    from cpmcu_b200.ops.ops import Ops
    from cpmcu_b200.parts.base import CacheNeeds
    from cpmcu_b200.parts.position import YarnRotary

    ops = Ops(DT[dtype])
    g = torch.Generator().manual_seed(R)
    eps, base = 1e-4, 3000.0
    rot, params = {"dims": dr, "base": base}, {}
    if scaling:
        rot["scaling"] = params = dict(zip(("factor", "original", "fast", "slow"), scaling))
    inv, mag, _ = YarnRotary(ops, max(dr, 2), base, dr, **params).rotary() if dr else (None, 1.0, 0)
    assert (mag != 1.0) == bool(scaling)
    lens, starts = [70, 5], [0, 130]
    n, cols = sum(lens), H * (dim + dr)
    proj = torch.randn(n, cols + R + dr, generator=g)
    gkv = 1 + 0.3 * torch.randn(R, generator=g)
    cache = Cache([CacheNeeds(kv_heads=1, head_dim=R + dr, values=False)], max_tokens=64 * 8, dtype=DT[dtype], device="cuda:0", n_slots=3)
    cache.open_sequence()
    slots = [cache.open_sequence(), cache.open_sequence()]
    for s, a, b in zip(slots, starts, lens):
        cache.reserve(s, a + b)
    cache.sync()
    lane = cache.lane(0)
    ctx = _ctx(lens, starts, slots)
    q = ops.latent_prepare(ctx, proj.cuda(), gkv.cuda(), lane, H, dim, R, dr, inv, eps, magnitude=mag)
    alone = ops.latent_prepare(ctx, proj[:, :cols].contiguous().cuda(), None, lane, H, dim, R, dr, inv, eps, write_cache=False, magnitude=mag)
    assert torch.equal(q, alone)                                 # a layer without rows of its own
    if dr:
        turned = ops.rotate_heads(ctx, proj[:, :cols].contiguous().cuda(), H, dim, dr, inv, magnitude=mag)
        _close(turned, q.cpu(), dtype, tol32=1e-6, tol16=1e-2)
    at = 0
    for s, start, m in zip(slots, starts, lens):
        rows = torch.zeros(start + m, cols + R + dr, dtype=torch.float64)
        rows[start:] = proj[at:at + m].double()
        heads = rows[:, :cols].view(-1, H, dim + dr)
        want_q = torch.cat([heads[..., :dim], plain.rotate_half(heads[..., dim:], rot if dr else None)], -1)[start:]
        _close(q[at:at + m].view(m, H, -1), want_q, dtype, tol32=3e-5, tol16=1e-2)
        w = {"dkv": torch.eye(R + dr, dtype=torch.float64), "dkv.norm": gkv.double()}
        c, k = plain.latent_rows(rows[:, cols:], w, "", {"kv_rank": R, "rot_dim": dr, "rot": rot if dr else None}, eps)
        pages = lane.page_table[s].tolist()
        stored = torch.stack([lane.k[pages[p // 64], 0, p % 64] for p in range(start, start + m)])
        _close(stored, torch.cat([c, k], -1)[start:], dtype, tol32=3e-5, tol16=1e-2)
        at += m
    before = lane.k.clone()
    wide = torch.cat([proj[:, :24], proj[:, cols:]], 1).contiguous().cuda()       # a query latent of 24 values in front
    ops.latent_norm_store(ctx, wide, torch.ones(24, device="cuda"), gkv.cuda(), lane, 24, R, eps, rot_dim=dr, inv_freq=inv, magnitude=mag)
    _close(lane.k, before.cpu(), dtype, tol32=1e-6, tol16=1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,row", [(3, 40), (18, 64), (5, 512), (4, 576), (1, 26)])
def test_latent_attention_with_towering_scores(dtype, H, row):
    """Cached rows and queries in latent space with scores that tower at the first key, on both sides of page borders and at
    the query itself, and larger ones right after the query (unseen); a prompt, then single tokens, by every kernel that
    takes the size; in a slot and pages that are not the first."""
    from cpmcu_b200.cache import Cache
    from cpmcu_b200.ops.ops import Ops
    from cpmcu_b200.parts.base import CacheNeeds

    ops = Ops(DT[dtype])
    g = torch.Generator().manual_seed(row)
    T, spike, scale = 200, row - 1, 0.2
    q = torch.randn(T, H, row, generator=g) * 0.3
    c = torch.randn(T, row, generator=g) * 0.3
    seen = [(199, 0), (198, 63), (190, 64), (180, 127), (170, 128), (150, 150), (129, 64), (128, 127), (65, 0), (64, 64), (63, 63), (1, 0), (0, 0)]
    marked = {a for a, _ in seen} | {b for _, b in seen}
    q[:, :, spike] = 0.0
    c[:, spike] = 0.0
    for i, (qi, kj) in enumerate(seen):
        q[qi] = 0.0                                              # the row looks along one direction of its own
        d = i % (row - 1)
        q[qi, :, d] = 8.0
        c[:, d] = 0.05 * c[:, d]
    for i, (qi, kj) in enumerate(seen):
        d = i % (row - 1)
        c[kj, d] = 9.0
        if qi + 1 < T:
            c[qi + 1, d] = 20.0
    rnd = lambda t: t.to(DT[dtype]).double()
    qq, cc = rnd(q), rnd(c)
    want = torch.stack([plain.causal_softmax((qq[:, h] @ cc.T) * scale) @ cc for h in range(H)], 1)
    cache = Cache([CacheNeeds(kv_heads=1, head_dim=row, values=False)], max_tokens=64 * 8, dtype=DT[dtype], device="cuda:0", n_slots=3)
    other = cache.open_sequence()
    cache.reserve(other, 70)
    slot = cache.open_sequence()
    cache.reserve(slot, T)
    cache.sync()
    lane = cache.lane(0)
    pages = lane.page_table[slot].tolist()
    for p in range(T):
        lane.k[pages[p // 64], 0, p % 64] = c[p].to(DT[dtype]).cuda()
    qd = qq.float().cuda()
    ways = [dict(tensor_cores=False)] + ([dict(tensor_cores=True), dict(tensor_cores=True, n_splits=3)]
                                         if ops.latent_attention_on_tensor_cores(row) else [])
    assert (len(ways) == 3) == (dtype == "bfloat16" and row % 16 == 0)
    for way in ways:
        got = ops.latent_attention(_ctx([T], [0], [slot]), qd, lane, scale, **way)
        _close(got, want, dtype)
        for qi, _ in seen:
            _close(got[qi], want[qi], dtype)
            one = ops.latent_attention(_ctx([1], [qi], [slot]), qd[qi:qi + 1].contiguous(), lane, scale, **way)
            _close(one[0], want[qi], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["rotated", "plain"])
def test_latent_layers_where_one_part_of_the_score_decides(folders, dtype, which):
    """The latent layers alone, with the rotated part of queries and keys (or the plain part) scaled up so that it decides
    the softmax: a rotation that paired other channels, a lost magnitude, a key part without its position or a reader's
    query against the wrong rows would move nearly all of a token's weight.  A prompt, then single tokens."""
    _, cfg, w = folders("latent_attention")
    w = {k: v.clone() for k, v in w.items()}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        H, d, dr, R = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
        q = w[p + "q"].float().view(H, d + dr, -1)
        if which == "rotated" and dr:
            q[:, d:] *= 3.0
            if p + "dkv" in w:
                w[p + "dkv"] = torch.cat([w[p + "dkv"][:R], (w[p + "dkv"][R:].float() * 2.0).bfloat16()])
        elif which == "plain":
            q[:, :d] *= 3.0
            w[p + "uk"] = (w[p + "uk"].float() * 2.0).bfloat16()
        w[p + "q"] = q.reshape(H * (d + dr), -1).bfloat16()
    folder = cases.write_folder(cfg, w, tempfile.mkdtemp(prefix=f"dinutar-latent-{which}-"))
    ids = cases.random_ids(cfg["vocab"], 160, 8)
    got = run_portions(make_stepper(folder, dtype), [ids], [[60, 2, 18] + [1] * 80])[0]
    e = cases.row_errors(got, plain.forward(cfg, w, ids))
    assert float(e.max()) <= {"float32": 3e-4, "bfloat16": 0.5}[dtype], float(e.max())
    assert float(e.median()) <= {"float32": 2e-5, "bfloat16": 5e-2}[dtype], float(e.median())


def _retention_data(H, d, dv, T, decay, rot, seed):
    """Projections [q | k | v | gate] in which the queries of some late tokens look along a direction that only one far
    key has: what it stored must still be there, decayed by the distance, and nothing else."""
    g = torch.Generator().manual_seed(seed)
    q, k = torch.randn(T, H, d, generator=g) * 0.5, torch.randn(T, H, d, generator=g) * 0.5
    v, gate = torch.randn(T, H, dv, generator=g), torch.randn(T, H, dv, generator=g) * 2
    far = [(T - 1, 0), (T - 2, 63), (T - 3, 64), (T - 9, T - 20)]
    if d > len(far) + rot:                                       # channels that are not turned
        for i, (a, b) in enumerate(far):
            c = d - 1 - i
            q[:, :, c] = 0.0
            k[:, :, c] = 0.0
            q[a] = 0.0
            q[a, :, c] = 30.0
            k[b, :, c] = 20.0
    return q, k, v, gate, [a for a, _ in far]


RETENTION_SIZES = [
    # H, d, dv, rot
    (3, 16, 40, 8), (6, 40, 8, 32), (2, 70, 20, 0), (2, 64, 64, 32), (1, 128, 128, 64), (1, 200, 136, 64), (5, 12, 7, 6), (1, 256, 256, 128),
    (2, 9, 33, 2), (1, 1, 1, 0),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,dv,rot", RETENTION_SIZES)
def test_retention_by_tokens_by_tiles_and_by_the_walk(dtype, H, d, dv, rot):
    """Three sequences at once in slots whose state starts as rubbish (a sequence's first token ignores it), their tokens in
    portions: whole prompts, pieces that end inside tiles, single tokens; far keys that decide a read-out; the step's, the
    tiles' and the walk's kernels, in 32-bit whatever the compute type (outputs in it)."""
    from cpmcu_b200.ops.ops import Ops

    ops = Ops(DT[dtype])
    decays = torch.tensor([[0.5, 0.97, 0.9995, 0.9, 0.99, 0.999][i % 6] for i in range(H)]) if H > 1 else torch.tensor([0.995])
    eps, kf, mag, base = 1e-5, d ** -0.5, 1.25, 500.0
    inv = (base ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))).float()
    lens = [210, 1, 130]
    data = [_retention_data(H, d, dv, n, decays, rot, 7 * n + d) if n > 100 else
            tuple(torch.randn(n, H, x, generator=torch.Generator().manual_seed(5)) for x in (d, d, dv, dv)) + ([],) for n in lens]
    wants, finals = [], []
    for q, k, v, gate, _ in data:
        turn = lambda t: torch.cat([plain.rotate_half(t.double()[..., :rot], {"dims": rot, "base": base}) * mag, t.double()[..., rot:]], -1) \
            if rot else t.double()
        o, S = plain.retention_recurrence(turn(q), turn(k) * kf, v.double(), decays.double())
        wants.append((plain.rms_norm(o, None, eps) * plain.silu(gate.double())).reshape(len(q), -1))
        finals.append(S)
    projs = [torch.cat([t.reshape(t.shape[0], -1) for t in x[:4]], 1) for x in data]
    powers = (decays.double()[:, None] ** torch.arange(65, dtype=torch.float64)).float().cuda()
    slots = [3, 0, 4]

    def by_tiles(ctx, proj, state):
        ops.rotate_scale(ctx, proj, 2 * H, d, inv.cuda() if rot else None, rot, mag, first_scaled=H, factor=kf)
        return ops.retention_tiles(ctx, proj[:, :H * d], proj[:, H * d:2 * H * d], proj[:, 2 * H * d:2 * H * d + H * dv],
                                   proj[:, 2 * H * d + H * dv:], powers, state, H, d, dv, eps)

    def by_tiles_raw(ctx, proj, state):
        ops.rotate_scale(ctx, proj, 2 * H, d, inv.cuda() if rot else None, rot, mag, first_scaled=H, factor=kf)
        o = ops.retention_tiles(ctx, proj[:, :H * d], proj[:, H * d:2 * H * d], proj[:, 2 * H * d:2 * H * d + H * dv], None, powers, state,
                                H, d, dv)
        return ops.gated_head_norm(o, proj[:, 2 * H * d + H * dv:], None, eps)

    def by_walk(ctx, proj, state):
        ops.rotate_scale(ctx, proj, 2 * H, d, inv.cuda() if rot else None, rot, mag, first_scaled=H, factor=kf)
        decay = decays.cuda().unsqueeze(0).expand(ctx.n_tokens, H)
        o = ops.linear_recurrence(ctx, proj[:, :H * d], proj[:, H * d:2 * H * d], proj[:, 2 * H * d:2 * H * d + H * dv], decay, None, state,
                                  H, H, d, dv, 1.0)
        return ops.gated_head_norm(o, proj[:, 2 * H * d + H * dv:], None, eps)

    def by_step(ctx, proj, state):
        return ops.retention_step(ctx, proj, decays.cuda(), state, H, d, dv, inv.cuda() if rot else None, rot, mag, False, kf, eps)

    whole = [[210, 1, 130]]
    pieces = [[70, 1, 64], [2, 0, 2], [138, 0, 63], [0, 0, 1]]
    ending = [[150, 1, 0], [0, 0, 90]] + [[1, 0, 1]] * 40 + [[1, 0, 0]] * 20
    for plan, kernels in ((whole, (by_tiles, by_tiles_raw, by_walk)), (pieces, (by_tiles, by_walk)), (ending, (None,))):
        for kernel in kernels:
            state = torch.randn(5, H, d, dv, generator=torch.Generator().manual_seed(1)).cuda()
            rubbish = state[1].clone()
            done, got = [0, 0, 0], [[], [], []]
            for step in plan:
                live = [i for i in range(3) if step[i]]
                ctx = _ctx([step[i] for i in live], [done[i] for i in live], [slots[i] for i in live])
                proj = torch.cat([projs[i][done[i]:done[i] + step[i]] for i in live]).cuda()
                fn = kernel or (by_step if ctx.is_decode else by_tiles)
                o = fn(ctx, proj, state)
                at = 0
                for i in live:
                    got[i].append(o[at:at + step[i]])
                    at += step[i]
                    done[i] += step[i]
            assert done == lens
            for i in range(3):
                out = torch.cat(got[i])
                _close(out, wants[i], dtype, tol32=5e-5, tol16=1e-2)
                for row in data[i][4]:
                    _close(out[row], wants[i][row], dtype, tol32=2e-4, tol16=1e-2)
                _close(state[slots[i]], finals[i], "float32", tol32=2e-5)
            assert torch.equal(state[1], rubbish)                # a slot that took no part


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,K,N", [(1, 64, 40), (8, 96, 33), (16, 128, 256), (9, 100, 20), (40, 96, 64), (300, 128, 192), (300, 192, 264),
                                   (2048, 256, 1032), (130, 72, 7)])
def test_squared_relu_product(dtype, M, K, N):
    """Every kernel that applies the activation: weight-streaming, tcgen05 and library product with a kernel behind it."""
    from cpmcu_b200.ops.ops import Ops

    ops = Ops(DT[dtype])
    g = torch.Generator().manual_seed(M + K)
    a, w = torch.randn(M, K, generator=g).to(DT[dtype]), (torch.randn(N, K, generator=g) * K ** -0.5).to(DT[dtype])
    want = torch.relu(a.double() @ w.double().T) ** 2
    got = ops.relu2_linear(a.cuda(), w.cuda())
    assert float(got.min()) >= 0
    _close(got, want, dtype, tol32=1e-5, tol16=1.5e-2)
    if dtype == "bfloat16" and K % 64 == 0 and N % 8 == 0:
        for pair in (False, True):
            forced = ops.linear_tcgen05(a.cuda(), w.cuda(), pair=pair, epilogue=ops.RELU2_EPILOGUE)
            _close(forced, want, dtype, tol16=1.5e-2)
        ops.raise_on_kernel_error()
