"""Layer-stack models on the GPU against the plain oracles (tests/roluzen_oracle.py, tovalix_oracle.py, zikezen_oracle.py, zigipel_oracle.py): whole
prompts, portions, mixed batches, decoding, slots and pages that are used again, greedy generation through the engine. Mechanism tests are in
test_stack_kernels_gpu.py and test_gated_linear_gpu.py."""
import functools

import pytest
import torch

from tests import stack_cases as C

pytestmark = pytest.mark.gpu
TOL = {torch.float32: 1e-5, torch.bfloat16: 1.5e-2}       # relative rms error of the logits against the oracle, all rows
NOISY = {"looped": 2.0}     # models whose longer chain of sublayers amplifies rounding: factor of the bf16 tolerance


class Ids:
    def encode(self, s):
        return [3 + (ord(c) % 50) for c in s]

    def decode(self, ids):
        return " ".join(str(int(i)) for i in ids)

    def bos_id(self):
        return 1

    def eos_id(self):
        return -1

    def pad_id(self):
        return 0


@functools.lru_cache(None)
def case(name, dtype, tmp=None):
    import tempfile

    from tunix_b200.models.automodel import AutoModel
    from tunix_b200.models.hf_config import config_from_hf
    cfg = C.CASES[name]
    w = C.weights(cfg, seed=len(name))
    src = C.write(tempfile.mkdtemp(), cfg, w)
    model, _ = AutoModel.from_pretrained(src, model_source="local", model_path=src, config=config_from_hf(src, dtype=dtype),
                                         device="cuda")
    return cfg, w, model


@functools.lru_cache(None)
def oracle(name, toks):
    cfg, w = C.CASES[name], C.weights(C.CASES[name], seed=len(name))
    return C.oracle(cfg).forward(cfg, w, list(toks))


def engine(model, pages=16, slots=3, page=64, ctx=None, **kw):
    from tunix_b200.common.configs import CacheConfig
    from tunix_b200.generate.engine import PagedEngine
    c = model.config
    return PagedEngine(model, Ids(), CacheConfig(ctx or pages * page, c.num_layers, c.num_kv_heads, c.head_dim), page_size=page,
                       max_running_requests=slots, num_pages=pages, **kw)


def session(model, **kw):
    from tunix_b200.generate.engine import StepSession
    return StepSession(engine(model, **kw))


def error(got, want):
    d = got.double().cpu() - want
    return (d.pow(2).mean().sqrt() / want.pow(2).mean().sqrt()).item()


def close(got, want, dtype):
    """All rows together within the tolerance (if they are enough for an average), and no single row far off (a random model
    amplifies rounding at some)."""
    print(f"rms {error(got, want):.2e}, worst row {worst_row(got, want):.2e}")
    return (got.shape[0] < 4 or error(got, want) < TOL[dtype]) and worst_row(got, want) < 8 * TOL[dtype]


def worst_row(got, want):
    d = (got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    return d.max().item()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_whole_prompt_and_layers(name, dtype):
    from tunix_b200.generate.engine import PagePool
    from tunix_b200.ops.ragged import RaggedBatch
    cfg, w, model = case(name, dtype)
    toks = C.tokens(cfg, 150)
    want, layers = C.oracle(cfg).forward(cfg, w, toks, want_layers=True)
    pool = PagePool(model.config, 4, 64, 2, 4, "cuda", dtype, prefix_caching=False)
    pool.open(1, toks, 0)
    pool.sync_table()
    sums = []
    ex = model.executor()
    ex.refresh()
    h = ex.forward(RaggedBatch.build([(1, 0, toks)], "cuda"), pool, sums)
    # the last pass is closed by the final norm's kernel, so every pass has left its sum
    assert len(sums) == len(model.config.runs())
    for s, ref in zip(sums, layers):
        assert close(s, ref, dtype)
    logits, cap = ex.logits(h), model.config.final_logit_softcap
    if cap:
        logits = cap * torch.tanh(logits / cap)
    assert close(logits, want, dtype)
    z, _ = model(torch.tensor([toks]))
    assert torch.allclose(z[0].float(), logits, atol=1e-4 if dtype == torch.float32 else 0.15)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_portions_and_decoding_agree_with_the_oracle(name, dtype):
    """The same sequence token by token, in twos, in growing portions and in one piece with a decoded tail."""
    cfg, _, model = case(name, dtype)
    n = 140
    toks = C.tokens(cfg, n, 1)
    want = oracle(name, tuple(toks))
    ses = session(model, pages=4, slots=1)
    for cuts in ([1] * n, [2] * 70, [3, 64, 1, 2, 5, 31, 30, 4], [65, 1, 1, 1, 63, 9], [100] + [1] * 40):
        at, rows = 0, []
        for c in cuts:
            rows.append(ses.step([("r", toks[at:at + c], range(c))], end=["r"] if at + c == n else ()))
            at += c
        assert at == n
        assert close(torch.cat(rows), want, dtype), cuts


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["mixed", "wide", "shared", "tiles", "uneven", "looped", "ragged", "blocks", "pairs", "crooked", "slabs"])
def test_mixed_batches_and_reused_slots(name, dtype):
    """Unequal requests: portions beside decoded tokens, requests that sit out steps, ends in between; six requests share
    three slots and a pool that holds two of the longest, so that pages and slots change owners."""
    cfg, _, model = case(name, dtype)
    lens = [130, 5, 77, 64, 129, 1]
    seqs = [C.tokens(cfg, n, 10 + i) for i, n in enumerate(lens)]
    wants = [oracle(name, tuple(s)) for s in seqs]
    ses = session(model, pages=7, slots=3)
    gen = torch.Generator().manual_seed(4)
    at, live, nxt, got = [0] * 6, [], 0, [[] for _ in seqs]
    while live or nxt < 6:
        while nxt < 6 and len(live) < 3 and sum(-(-lens[i] // 64) for i in live) + -(-lens[nxt] // 64) <= 7:
            live.append(nxt)
            nxt += 1
        entries, order, end = [], [], []
        for i in live:
            if len(live) > 1 and torch.rand((), generator=gen) < 0.25:
                continue                                                # sits this step out
            size = [1, 1, 2, 7, 64, 40][int(torch.randint(0, 6, (), generator=gen))]
            part = seqs[i][at[i]:at[i] + size]
            entries.append((i, part, range(len(part))))
            order.append((i, len(part)))
            at[i] += len(part)
            if at[i] == lens[i]:
                end.append(i)
        z, o = ses.step(entries, end), 0
        for i, k in order:
            got[i].append(z[o:o + k])
            o += k
        live = [i for i in live if i not in end]
    for i, want in enumerate(wants):
        assert close(torch.cat(got[i]), want, dtype), i


@pytest.mark.parametrize("name", ["wide", "tiles", "blocks", "slabs"])
def test_a_batch_equals_each_request_alone_in_bf16(name):
    """bf16 results do not depend on the company beyond rounding: compared with the single request, not with the oracle."""
    cfg, _, model = case(name, torch.bfloat16)
    seqs = [C.tokens(cfg, n, 30 + n) for n in (33, 190, 70)]
    ses = session(model, pages=8, slots=3)
    together = ses.step([(i, s, range(len(s))) for i, s in enumerate(seqs)])
    step = ses.step([(i, [7 + i], [0]) for i in range(3)], end=[0, 1, 2])
    o = 0
    for i, s in enumerate(seqs):
        alone = ses.step([("x", s, range(len(s)))])
        after = ses.step([("x", [7 + i], [0])], end=["x"])
        assert error(together[o:o + len(s)], alone.double().cpu()) < 1e-2
        assert error(step[i:i + 1], after.double().cpu()) < 2e-2
        o += len(s)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["mixed", "shared", "tiles", "looped", "blocks", "pairs", "slabs"])
def test_long_decoding(name, dtype):
    """Several hundred decoded tokens: states, rings, windows and chunks that have turned over many times."""
    cfg, _, model = case(name, dtype)
    toks = C.tokens(cfg, 460, 2)
    want = oracle(name, tuple(toks))
    ses = session(model, pages=8, slots=2)
    ses.step([("r", toks[:30], [])])
    rows = [ses.step([("r", [t], [0])]) for t in toks[30:]]
    assert close(torch.cat(rows), want[30:], dtype)


def test_step_session_errors():
    cfg, _, model = case("mixed", torch.float32)
    ses = session(model, pages=2, slots=1)
    ses.step([("a", [1, 2], [1])])
    with pytest.raises(RuntimeError, match="slots"):
        ses.step([("b", [1], [0])])
    with pytest.raises(KeyError):
        ses.end("b")
    assert ses.step([("a", [3], [])], end=["a"]).shape == (0, cfg["vocab"])
    with pytest.raises(ValueError, match="page table"):
        ses.step([("c", [1] * 200, [])])
    assert ses.step([("d", [1], [0])]).shape == (1, cfg["vocab"])       # the slot was not lost


# ------------------------------------------------------------------------------------------------ generation
def greedy_reference(name, prompt, steps):
    """Greedy continuation by the oracle; stops being followed where the two best logits are close."""
    cfg, w = C.CASES[name], C.weights(C.CASES[name], seed=len(name))
    toks, margins = list(prompt), []
    for _ in range(steps):
        z = C.oracle(cfg).forward(cfg, w, toks)[-1]
        top = z.topk(2).values
        margins.append((top[0] - top[1]).item() / z.std().item())
        toks.append(int(z.argmax()))
    return toks[len(prompt):], margins


@pytest.mark.parametrize("graph", [True, False])
@pytest.mark.parametrize("name", ["mixed", "shared", "uneven", "looped", "ragged", "pairs", "crooked"])
def test_greedy_generation_matches_the_oracle(name, graph):
    """Through the engine's entry point and scheduler in 32-bit: four prompts over two slots and a pool that forces
    pre-emption, decode step captured in a graph or not; logits of the oracle decide."""
    cfg, _, model = case(name, torch.float32)
    prompts = [C.tokens(cfg, n, 50 + n) for n in (14, 33, 20, 7)]
    steps = 12
    eng = engine(model, pages=5, slots=2, page=16, ctx=64, use_cuda_graph=graph, check_every=4)
    out = eng(prompt_token_ids=prompts, max_generation_steps=steps, max_prompt_length=40, temperature=0.0, eos_tokens=[-1],
              return_logprobs=True)
    for p, got, lps in zip(prompts, out.tokens, out.logprobs):
        want, margins = greedy_reference(name, p, steps)
        for a, b, mg, lp in zip(got.tolist(), want, margins, lps):
            if a != b:
                assert mg < 1e-3, (a, b, mg)
                break
            assert lp <= 0.0


@pytest.mark.parametrize("name", ["wide", "tiles", "blocks", "pairs", "slabs"])
def test_generation_is_the_same_under_portions_preemption_and_graphs(name):
    """bf16 and the tensor-core kernels: sampled tokens of one engine against engines with other schedules."""
    cfg, _, model = case(name, torch.bfloat16)
    prompts = [C.tokens(cfg, n, 70 + n) for n in (120, 3, 64, 65, 31)]

    def gen(**kw):
        eng = engine(model, **kw)
        out = eng(prompt_token_ids=prompts, max_generation_steps=24, max_prompt_length=128, temperature=0.0, eos_tokens=[-1],
                  return_logprobs=True)
        return out, eng
    base, _ = gen(pages=20, slots=5, ctx=192)
    for kw in (dict(pages=20, slots=5, ctx=192, use_cuda_graph=False), dict(pages=20, slots=2, ctx=192),
               dict(pages=20, slots=5, ctx=192, prefill_chunk=17), dict(pages=6, slots=5, ctx=192, check_every=4)):
        out, eng = gen(**kw)
        for a, b, la, lb in zip(base.tokens, out.tokens, base.logprobs, out.logprobs):
            same = (a == b).tolist()
            k = same.index(False) if False in same else len(same)
            # identical until a near tie (rounding differs between schedules); log-probs agree along the common part
            assert max((abs(x - y) for x, y in zip(la[:k], lb[:k])), default=0.0) < 0.12, kw
            if k < len(same):
                assert abs(la[k] - lb[k]) < 0.3, kw


@pytest.mark.parametrize("name", ["wide", "tiles", "blocks", "slabs"])
def test_stop_tokens_and_sampling_run_through_the_engine(name):
    cfg, _, model = case(name, torch.bfloat16)
    eng = engine(model, pages=12, slots=4, ctx=192)
    prompts = [C.tokens(cfg, 9, 90 + i) for i in range(4)]
    kw = dict(prompt_token_ids=prompts, max_generation_steps=16, max_prompt_length=16, temperature=0.8, top_p=0.9, top_k=40, seed=5)
    a, b = eng(**kw, eos_tokens=[-1]), eng(**kw, eos_tokens=[-1])
    assert all((x == y).all() for x, y in zip(a.tokens, b.tokens))
    stop = int(a.tokens[0][3])
    c = eng(**kw, eos_tokens=[stop])
    first = a.tokens[0].tolist().index(stop)
    assert c.tokens[0].tolist() == a.tokens[0].tolist()[:first + 1]


@pytest.mark.parametrize("name", ["wide", "tiles", "blocks", "slabs"])
def test_engine_server_serves_the_model(name):
    from tunix_b200.generate.engine import EngineServer
    cfg, _, model = case(name, torch.bfloat16)
    prompts = [C.tokens(cfg, n, 120 + n) for n in (5, 40, 12)]
    with EngineServer(engine(model, pages=12, slots=2, ctx=192, check_every=4), max_new_tokens=8, max_prompt_length=64,
                      temperature=0.0, eos_tokens=[-1]) as srv:
        futs = [srv.submit(p) for p in prompts]
        first = [f.result(120)[0].tolist() for f in futs]
        srv.pause()
        srv.resume()
        assert [srv.generate(p)[0].tolist() for p in prompts][0][:1] == first[0][:1]
    assert all(len(t) == 8 for t in first)


@pytest.mark.parametrize("name", ["wide", "tiles", "blocks", "slabs"])
def test_scoring_with_padding_matches_unpadded_rows(name):
    cfg, _, model = case(name, torch.float32)
    rows = [C.tokens(cfg, n, 140 + n) for n in (6, 19)]
    T = 24
    toks, seg = torch.zeros(2, T, dtype=torch.long), torch.zeros(2, T, dtype=torch.int32)
    toks[0, T - 6:], seg[0, T - 6:] = torch.tensor(rows[0]), 1          # left padding, as prompts have
    toks[1, :19], seg[1, :19] = torch.tensor(rows[1]), 1                # right padding, as completions have
    z, _ = model(toks, segment_ids=seg)
    assert close(z[0, T - 6:], oracle(name, tuple(rows[0])), torch.float32)
    assert close(z[1, :19], oracle(name, tuple(rows[1])), torch.float32)


@pytest.mark.parametrize("name", ["mixed", "shared", "looped", "pairs"])
def test_trace_runner_replays_steps(name, tmp_path):
    import json
    import os
    import subprocess
    import sys

    import numpy as np
    cfg = C.CASES[name]
    w = C.weights(cfg, seed=3)
    src = C.write(tmp_path / "model", cfg, w)
    toks = C.tokens(cfg, 70, 5)
    want = C.oracle(cfg).forward(cfg, w, toks)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[40:41], "want": []}, {"id": "b", "tokens": toks[:9], "want": [8]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[41:], "want": [28]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", src, "--dtype", "float32", "--out",
                          str(tmp_path), "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps),
                         capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    assert [x for x in out.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    for step, rows in ((0, [0, 39]), (1, [8]), (2, [69])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{step}.f32", "<f4")).view(len(rows), -1)
        assert close(got, want[rows], torch.float32)


def test_log_probabilities_of_scaled_logits():
    """Scoring uses the scaled logits, as generation does."""
    cfg, _, model = case("pairs", torch.float32)
    toks = C.tokens(cfg, 30, 170)
    want = torch.log_softmax(oracle("pairs", tuple(toks)) / 0.7, -1)
    hidden, _ = model(torch.tensor([toks]), skip_lm_head=True)
    targets = torch.tensor([toks[1:] + [0]], device="cuda")
    got = model.token_logprobs(hidden, targets, temperature=0.7)
    got = (got[0] if isinstance(got, tuple) else got).view(-1)
    assert torch.allclose(got.double().cpu(), want[torch.arange(30), targets[0].cpu()], atol=2e-4)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["pairs", "slabs"])
def test_portions_expand_and_single_tokens_absorb(name, dtype):
    """Cuts on both sides of the length from which a portion's keys are expanded, behind prefixes longer than every window, beside
    requests that do the other; every row against the oracle."""
    from tunix_b200.ops.ragged import EXPAND_MIN, RaggedBatch
    cfg, _, model = case(name, dtype)
    windows = [L["mixer"]["mask"]["size"] for L in cfg["layers"] if L["type"] == "latent_attention"]
    lens = [300, 290, 40]
    seqs = [C.tokens(cfg, n, 180 + i) for i, n in enumerate(lens)]
    wants = [oracle(name, tuple(s)) for s in seqs]
    ses = session(model, pages=12, slots=3)
    at, got = [0, 0, 0], [[], [], []]
    cuts = [(128, 1, 15), (EXPAND_MIN - 1, 127, 1), (EXPAND_MIN, 2, 16), (1, EXPAND_MIN + 9, 0), (2, 64, 1), (65, 1, 2), (1, 1, 1),
            (72, 69, 4)]
    kinds = set()
    for step in cuts:
        entries = [(i, seqs[i][at[i]:at[i] + k], range(k)) for i, k in enumerate(step) if k]
        for w in windows:
            plan = RaggedBatch.build([(0, at[i], t) for i, t, _ in entries], "cuda").latent_plan(w)
            kinds.add((plan.blocks is not None, plan.rows is None or len(plan.rows) > 0))
        z, o = ses.step(entries), 0
        for i, t, _ in entries:
            got[i].append(z[o:o + len(t)])
            at[i], o = at[i] + len(t), o + len(t)
    assert at == lens and {(True, True), (False, True)} <= kinds
    for i, want in enumerate(wants):
        assert close(torch.cat(got[i]), want, dtype), i


def test_sequences_longer_than_the_learned_positions_are_refused():
    cfg, _, model = case("looped", torch.bfloat16)
    ses = session(model, pages=10, slots=1)
    toks = C.tokens(cfg, cfg["max_positions"], 160)
    z = ses.step([("a", toks[:500], [499])])
    assert ses.step([("a", toks[500:], [11])]).isfinite().all() and z.isfinite().all()
    with pytest.raises(ValueError, match="positions"):
        ses.step([("a", [1], [0])])
    eng = engine(model, pages=10, slots=1)
    with pytest.raises(ValueError, match="positions"):
        eng(prompt_token_ids=[toks[:500]], max_generation_steps=20, max_prompt_length=512, eos_tokens=[-1])
