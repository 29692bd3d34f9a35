"""Zuvasun through the engine against the plain implementation (tests/plain/zuvasun_plain.py, float64 on the CPU): whole
prompts, portions, token by token, batches, pages and slots used again, one key that decides near and far and at a window's
edge, entries read by another layer, graphs replayed, generation."""
import copy

import pytest
import torch

from tests import zuvasun_util as zu

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["MIXED", "ODD", "WIDE"])
def test_whole_prompt_and_portions_match_the_plain_model(name, dtype):
    cfg = getattr(zu, name)
    model, tensors = zu.build(cfg, seed=3, dtype=dtype)
    ids = zu.ids_for(cfg, 75, seed=1)
    want = zu.plain_logits(cfg, tensors, ids)
    drv = zu.driver(model, dtype)
    zu.assert_close(zu.run_in_portions(drv, "a", ids, [len(ids)]), want, dtype)
    zu.assert_close(zu.run_in_portions(drv, "a", ids, [33, 2, 1, 17, 1]), want, dtype)
    assert drv.executor.cache.all_free()


def one_mechanism(which: str) -> dict:
    """One layer (a reader: two) of MIXED alone, with or without its feed-forward."""
    at = {"latent": 0, "attention": 1, "untempered": 3, "routed": 1}.get(which)
    if at is not None:
        layer = copy.deepcopy(zu.MIXED["layers"][at])
        if which != "routed":
            layer["mlp"] = None
        return zu.config([layer])
    layers = copy.deepcopy([zu.MIXED["layers"][0], zu.MIXED["layers"][2]])
    layers[0]["mlp"] = None
    layers[1]["mixer"]["kv_from"] = 0
    return zu.config(layers)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["latent", "attention", "untempered", "routed", "reader"])
def test_each_mechanism_in_a_layer_of_its_own(which, dtype):
    cfg = one_mechanism(which)
    model, tensors = zu.build(cfg, seed=21, dtype=dtype, sigma=0.25)
    ids = zu.ids_for(cfg, 90, seed=8)
    want = zu.plain_logits(cfg, tensors, ids)
    drv = zu.driver(model, dtype)
    zu.assert_close(zu.run_in_portions(drv, "a", ids, [90]), want, dtype, which)
    zu.assert_close(zu.run_in_portions(drv, "a", ids, [40, 1, 1, 7, 2]), want, dtype, which)


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_any_size_and_single_tokens_give_the_whole_prompts_logits(dtype):
    cfg = zu.MIXED
    model, tensors = zu.build(cfg, seed=4, dtype=dtype)
    ids = zu.ids_for(cfg, 101, seed=2)
    want = zu.plain_logits(cfg, tensors, ids)
    drv = zu.driver(model, dtype)
    for portions in ([1], [2], [3, 2, 33, 31, 1, 16, 2], [32, 32, 5, 1], [47, 1, 1, 2], [24, 24, 10, 10, 1]):
        got = zu.run_in_portions(drv, "a", ids, portions)
        zu.assert_close(got, want, dtype, portions)
    assert drv.executor.cache.all_free()


@pytest.mark.parametrize("eager", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_that_cross_tiles_of_the_tensor_core_attention(dtype, eager):
    """300 tokens whole, in portions whose tiles of queries begin anywhere among the keys' tiles and the windows' edges, beside
    another request, and decoded; launched and replayed."""
    cfg = zu.TENSOR
    model, tensors = zu.build(cfg, seed=15, dtype=dtype)
    ids, other = zu.ids_for(cfg, 300, seed=5), zu.ids_for(cfg, 90, seed=6)
    want, want_other = zu.plain_logits(cfg, tensors, ids), zu.plain_logits(cfg, tensors, other)
    drv = zu.driver(model, dtype, pool_tokens=448, eager=eager)
    zu.assert_close(zu.run_in_portions(drv, "a", ids, [300]), want, dtype)
    zu.assert_close(zu.run_in_portions(drv, "a", ids, [130, 70, 1, 2, 65, 1]), want, dtype)
    got_a = [drv.step([("a", ids[:200], list(range(200)))])]
    out = drv.step([("a", ids[200:], list(range(100))), ("b", other, list(range(90)))], end=["a", "b"])
    zu.assert_close(torch.cat([got_a[0], out[:100]]), want, dtype)
    zu.assert_close(out[100:], want_other, dtype)


@pytest.mark.parametrize("name", ["WIDE", "TENSOR"])
def test_the_logits_do_not_depend_on_the_cut_beyond_rounding(name):
    """float32: token by token, in twos and whole agree far inside the tolerance against the plain model."""
    cfg = getattr(zu, name)
    model, _ = zu.build(cfg, seed=14, dtype="float32")
    ids = zu.ids_for(cfg, 80, seed=3)
    drv = zu.driver(model, "float32")
    whole = zu.run_in_portions(drv, "a", ids, [80])
    for portions in ([1], [2], [17, 3], [33, 33, 1]):
        assert zu.relative_error(zu.run_in_portions(drv, "a", ids, portions), whole) < 3e-6, portions


@pytest.mark.parametrize("eager", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_match_each_alone(dtype, eager):
    """Three requests of different lengths, portions of some beside single tokens of others; launched kernel by kernel and
    replayed from the graphs of the steps' shapes."""
    cfg = zu.MIXED
    model, tensors = zu.build(cfg, seed=5, dtype=dtype)
    ids = {"a": zu.ids_for(cfg, 70, 11), "b": zu.ids_for(cfg, 19, 12), "c": zu.ids_for(cfg, 41, 13)}
    want = {r: zu.plain_logits(cfg, tensors, t) for r, t in ids.items()}
    drv = zu.driver(model, dtype, eager=eager)
    plan = {"a": [33, 1, 1, 2, 30, 1, 1, 1], "b": [2, 1, 1, 1, 14], "c": [1, 1, 17, 2, 20]}
    pos = {r: 0 for r in ids}
    got = {r: [] for r in ids}
    k = 0
    while any(pos[r] < len(ids[r]) for r in ids):
        entries, owners, end = [], [], []
        for r in ids:
            if pos[r] >= len(ids[r]) or (r == "b" and k == 2):          # b sits one step out
                continue
            n = min(plan[r][min(k, len(plan[r]) - 1)], len(ids[r]) - pos[r])
            entries.append((r, ids[r][pos[r]:pos[r] + n], list(range(n))))
            owners.append((r, n))
            pos[r] += n
            if pos[r] == len(ids[r]):
                end.append(r)
        out = drv.step(entries, end=end)
        at = 0
        for r, n in owners:
            got[r].append(out[at:at + n])
            at += n
        k += 1
    for r in ids:
        zu.assert_close(torch.cat(got[r]), want[r], dtype, r)
    if not eager:
        assert drv.executor.n_shaped_steps > 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_are_used_again(dtype):
    """A pool of 6 pages for five requests one after and beside another: every page serves several requests, in the groups of
    both kinds (every key; a window, as wide as the widest reader's)."""
    cfg = zu.MIXED
    model, tensors = zu.build(cfg, seed=6, dtype=dtype)
    drv = zu.driver(model, dtype, pool_tokens=96, page_size=16, max_num_seqs=2)
    assert sorted(g.window for g in drv.executor.group_specs) == [0, 41]
    lengths = [40, 50, 33, 17, 48]
    all_ids = [zu.ids_for(cfg, n, 20 + i) for i, n in enumerate(lengths)]
    want = [zu.plain_logits(cfg, tensors, t) for t in all_ids]
    zu.assert_close(zu.run_in_portions(drv, 0, all_ids[0], [13, 27]), want[0], dtype)
    for a, b in ((1, 2), (3, 4)):
        ga, gb = [], []
        pa = pb = 0
        while pa < lengths[a] or pb < lengths[b]:
            entries = []
            na = min(11, lengths[a] - pa)
            nb = min(20 if pb == 0 else 1, lengths[b] - pb)
            if na:
                entries.append((a, all_ids[a][pa:pa + na], list(range(na))))
            if nb:
                entries.append((b, all_ids[b][pb:pb + nb], list(range(nb))))
            pa, pb = pa + na, pb + nb
            out = drv.step(entries, end=[r for r, p, n in ((a, pa, na), (b, pb, nb)) if n and p == lengths[r]])
            if na:
                ga.append(out[:na])
            if nb:
                gb.append(out[na:na + nb])
        zu.assert_close(torch.cat(ga), want[a], dtype, a)
        zu.assert_close(torch.cat(gb), want[b], dtype, b)
    assert drv.executor.cache.all_free()


def with_window(cfg, tensors, ids, size):
    other = copy.deepcopy(cfg)
    other["layers"][-1]["mixer"]["mask"] = {"size": size}
    return zu.plain_logits(other, tensors, ids)


def without_needle(ids):
    return [zu.FILLER_ID if t == zu.NEEDLE_ID else t for t in ids]


# (tokens, the needle's place, tokens a page): the probe is the last token and sees the NEEDLE_WINDOW = 40 positions up to itself
EDGES = [
    (300, 260, 16),     # the oldest key of the window: just inside
    (300, 259, 16),     # the key before it: just outside
    (300, 298, 16),     # the newest but one
    (300, 0, 16),       # far away
    (289, 249, 32),     # just inside, the window's edge inside a page
    (289, 248, 32),     # just outside
    (273, 233, 16),     # the probe opens a page; just inside
    (272, 232, 16),     # the probe closes a page; just inside
    (272, 231, 16),     # just outside, the last key of the page before the window's first
    (41, 0, 16),        # the first key of all, just outside
    (40, 0, 16),        # and just inside
    (30, 0, 16),        # a prompt shorter than the window
]


@pytest.mark.parametrize("name", ["NEAR", "BORROWED"])
@pytest.mark.parametrize("n,needle_at,page", EDGES)
def test_one_key_decides_inside_the_window_and_not_outside(name, n, needle_at, page):
    """The last token's query finds the latent of one token only (`plant_latent`).  Where that token lies in the probe's window,
    the probe's logits follow its value; where it lies outside (one position is enough), they must not: the plain model with a
    wider window then differs by hundreds of tolerances, as it does without the needle when the needle is inside.  Whole, in
    portions cut at and beside the needle and the window's edge, and with the probe decoded alone after single tokens.  In
    BORROWED the entries are another layer's, whose own window (7) has long passed the needle."""
    cfg = getattr(zu, name)
    model, tensors = zu.build(cfg, seed=7, dtype="float32", sigma=0.3, prepare=zu.plant_latent)
    ids = zu.needle_ids(cfg, n, needle_at, 31)
    want = zu.plain_logits(cfg, tensors, ids)
    inside = (n - 1) - needle_at < zu.NEEDLE_WINDOW
    other = zu.plain_logits(cfg, tensors, without_needle(ids)) if inside else with_window(cfg, tensors, ids, 4096)
    assert zu.relative_error(other[-1:], want[-1:]) > 100 * zu.TOL["float32"]
    drv = zu.driver(model, "float32", pool_tokens=320, page_size=page)
    edge = max(n - zu.NEEDLE_WINDOW, 0)
    cuts = {(n,), (max(needle_at, 1), 1, 2, n), (needle_at + 1, 1, n), (max(n - 45, 1),) + (1,) * 45}
    if edge > 1:
        cuts |= {(edge, n), (edge - 1, 2, n), (edge + 1, n)}
    for portions in sorted(cuts):
        got = zu.run_in_portions(drv, "a", ids, list(portions))
        assert zu.relative_error(got, want) < zu.TOL["float32"], portions
    assert drv.executor.cache.all_free()


@pytest.mark.parametrize("n,needle_at,page", [(300, 0, 16), (300, 15, 16), (300, 16, 16), (300, 298, 16), (289, 255, 32), (257, 128, 16), (2, 0, 16)])
def test_a_far_key_is_found_by_the_attention_over_every_key(n, needle_at, page):
    """FAR: one key among hundreds decides, wherever it lies; its value is the key as projected, not as normed."""
    cfg = zu.FAR
    model, tensors = zu.build(cfg, seed=7, dtype="float32", sigma=0.3, prepare=zu.plant_far)
    ids = zu.needle_ids(cfg, n, needle_at, 31)
    want = zu.plain_logits(cfg, tensors, ids)
    assert zu.relative_error(zu.plain_logits(cfg, tensors, without_needle(ids))[-1:], want[-1:]) > 100 * zu.TOL["float32"]
    drv = zu.driver(model, "float32", pool_tokens=320, page_size=page)
    for portions in ((n,), (max(needle_at, 1), 1, 2, n), (needle_at + 1, 1, n), (max(n - 30, 1),) + (1,) * 30):
        got = zu.run_in_portions(drv, "a", ids, list(portions))
        assert zu.relative_error(got, want) < zu.TOL["float32"], portions


@pytest.mark.parametrize("eager", [True, False])
@pytest.mark.parametrize("name,prepare,places", [("FAR", "plant_far", (3, 77)), ("NEAR", "plant_latent", (260, 259)), ("BORROWED", "plant_latent", (260, 259))])
def test_the_needle_in_the_bfloat16_engine_and_beside_other_requests(name, prepare, places, eager):
    """The tensor-core kernels of the bfloat16 engine take these layers' widths: two requests in one step, the needle just inside
    the probe's window in one and just outside in the other (FAR: far away in both); launched and replayed."""
    cfg = getattr(zu, name)
    model, tensors = zu.build(cfg, seed=7, dtype="bfloat16", sigma=0.3, prepare=getattr(zu, prepare))
    n = 300
    ids = [zu.needle_ids(cfg, n, at, 31 + i) for i, at in enumerate(places)]
    want = [zu.plain_logits(cfg, tensors, t) for t in ids]
    if name == "FAR":
        cost = min(zu.relative_error(zu.plain_logits(cfg, tensors, without_needle(t))[-1:], w[-1:]) for t, w in zip(ids, want))
    else:
        cost = min(zu.relative_error(with_window(cfg, tensors, ids[1], 4096)[-1:], want[1][-1:]),
                   zu.relative_error(with_window(cfg, tensors, ids[0], 39)[-1:], want[0][-1:]))
    assert cost > 5 * zu.TOL["bfloat16"]
    drv = zu.driver(model, "bfloat16", pool_tokens=640, eager=eager)
    for first in (n, 290, 250):
        out = drv.step([("a", ids[0][:first], list(range(first))), ("b", ids[1][:first], list(range(first)))], end=["a", "b"] if first == n else [])
        got = [[out[:first]], [out[first:]]]
        for t in range(first, n):
            out = drv.step([("a", ids[0][t:t + 1], [0]), ("b", ids[1][t:t + 1], [0])], end=["a", "b"] if t == n - 1 else [])
            got[0].append(out[:1])
            got[1].append(out[1:])
        for g, w in zip(got, want):
            zu.assert_close(torch.cat(g), w, "bfloat16", first)
            assert zu.relative_error(torch.cat(g)[-1:], w[-1:]) < zu.TOL["bfloat16"]


def test_the_temperature_steps_where_the_position_says():
    """A large coefficient, steps every 6 positions: one position off would show by many tolerances around every step."""
    cfg = zu.config([zu.attention(2, 1, 16, 0.5, None, q_temp=(2.0, 6))])
    model, tensors = zu.build(cfg, seed=12, dtype="float32", sigma=0.4)
    ids = zu.ids_for(cfg, 40, seed=9)
    want = zu.plain_logits(cfg, tensors, ids)
    shifted = copy.deepcopy(cfg)
    shifted["layers"][0]["mixer"]["q_temp"]["every"] = 5.999
    flat = copy.deepcopy(cfg)
    flat["layers"][0]["mixer"].pop("q_temp")
    differs = zu.row_errors(zu.plain_logits(flat, tensors, ids), want)
    assert float(differs[:5].max()) == 0.0 and float(differs[5:].median()) > 100 * zu.TOL["float32"]
    drv = zu.driver(model, "float32")
    for portions in ([40], [5, 1, 1, 5, 7], [1]):
        assert zu.relative_error(zu.run_in_portions(drv, "a", ids, portions), want) < zu.TOL["float32"], portions


def test_the_correction_chooses_and_the_score_weighs():
    """Corrections far above the scores force the choice; without them, or with them in the weights, the logits differ."""
    cfg = zu.config([zu.attention(2, 1, 8, 0.3, zu.moe(6, 2, 24, 1.5))])

    def prepare(cfg, tensors):
        tensors["l0.mlp.correction"].copy_(torch.tensor([0.0, 2.0, 0.0, 0.0, 3.0, 0.0]))
        tensors["l0.mlp.router"].mul_(4.0)

    model, tensors = zu.build(cfg, seed=12, dtype="float32", sigma=0.3, prepare=prepare)
    ids = zu.ids_for(cfg, 30, seed=9)
    want = zu.plain_logits(cfg, tensors, ids)
    flat = dict(tensors)
    flat["l0.mlp.correction"] = torch.zeros(6)
    assert float(zu.row_errors(zu.plain_logits(cfg, flat, ids), want).median()) > 100 * zu.TOL["float32"]
    drv = zu.driver(model, "float32")
    assert zu.relative_error(zu.run_in_portions(drv, "a", ids, [29, 1]), want) < zu.TOL["float32"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """A hundred tokens of prompt and 300 decoded ones: windows pass over decoded tokens many times, key parts grow."""
    cfg = zu.TENSOR
    model, tensors = zu.build(cfg, seed=8, dtype=dtype)
    ids = zu.ids_for(cfg, 400, 41)
    want = zu.plain_logits(cfg, tensors, ids)
    drv = zu.driver(model, dtype, pool_tokens=448, eager=False)
    zu.assert_close(zu.run_in_portions(drv, "a", ids, [100] + [1] * 300), want, dtype)


@pytest.mark.parametrize("name", ["MIXED", "ODD", "WIDE"])
def test_the_first_tokens_of_a_sequence(name):
    cfg = getattr(zu, name)
    model, tensors = zu.build(cfg, seed=9, dtype="float32")
    drv = zu.driver(model, "float32")
    for n in (1, 2, 3, 6):
        ids = zu.ids_for(cfg, n, 50 + n)
        for portions in ([1], [n]):
            got = zu.run_in_portions(drv, "a", ids, portions)
            assert zu.relative_error(got, zu.plain_logits(cfg, tensors, ids)) < zu.TOL["float32"], (n, portions)


@pytest.mark.parametrize("dtype", DTYPES)
def test_replayed_steps_give_the_bits_of_launched_ones(dtype):
    """Decode steps through the sampling graphs and shaped steps against the same steps launched kernel by kernel."""
    from llmgen_b200.engine.executor import StepEntry
    cfg = zu.TENSOR
    model, _ = zu.build(cfg, seed=16, dtype=dtype)
    ids = zu.ids_for(cfg, 150, 3)
    seen = []
    for eager in (True, False):
        drv = zu.driver(model, dtype, pool_tokens=448, eager=eager)
        logits = drv.step([("a", ids, list(range(0, 150, 7)))])
        ex, tok, toks = drv.executor, ids[-1], []
        for p in range(150, 170):
            assert ex.reserve("a", p, p + 1)
            tok = ex.step([StepEntry("a", [tok], p, [0])], sample=True, return_logits=False).token_ids[0]
            toks.append(tok)
        seen.append((logits.clone().cpu(), toks))
        ex.release("a")
    assert seen[0][1] == seen[1][1]
    assert float((seen[0][0] - seen[1][0]).abs().max()) <= 1e-5 * float(seen[0][0].abs().max())


@pytest.mark.parametrize("eager", [True, False])
def test_greedy_generation_through_the_engine_and_its_scheduler(eager):
    """`LLM.generate` (scheduler, chunked prompts, decode graphs, sampling kernel) against greedy decoding with the plain
    model."""
    from llmgen_b200.engine.api import LLM
    from llmgen_b200.sampling.params import SamplingParams
    cfg = zu.MIXED
    model, tensors = zu.build(cfg, seed=10, dtype="float32")
    prompts = [zu.ids_for(cfg, n, 60 + n) for n in (9, 21, 4)]
    new = 10
    ref = []
    for p in prompts:
        seq = list(p)
        for _ in range(new):
            seq.append(int(zu.plain_logits(cfg, tensors, seq)[-1].argmax()))
        ref.append(seq[len(p):])
    llm = LLM(model, dtype="float32", max_model_len=64, max_num_seqs=2, max_batched_tokens=64, pass_tokens=64, block_size=16,
              kv_blocks=8, policy="chunked", chunk=8, eager=eager, capture_at_start=False)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=new, ignore_eos=True))
    assert [o["token_ids"] for o in outs] == ref
    assert llm.executor.cache.all_free()
    if not eager:
        assert llm.executor.n_graph_steps > 0


def test_a_model_folder_through_the_replay_program_and_the_command_line(tmp_path):
    """A Zuvasun folder written by the random-weights mode: `bin/trace_run` replays a trace of five requests on four slots and a
    pool smaller than their sum (float32 logits against the plain model), `python -m llmgen_b200 chat` generates the plain
    model's greedy tokens, and `info` describes the folder."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np
    from safetensors.torch import load_file

    from llmgen_b200.engine.api import write_random_model
    from tests.util import ROOT
    cfg = zu.MIXED
    folder = write_random_model(str(tmp_path / "model"), cfg, seed=13, sigma=0.1, sigma_norm=0.2)
    tensors = load_file(os.path.join(folder, "model.safetensors"))
    lengths = [70, 40, 23, 64, 51]
    ids = [zu.ids_for(cfg, n, 70 + i) for i, n in enumerate(lengths)]
    want = [zu.plain_logits(cfg, tensors, t) for t in ids]
    steps, pos, live, waiting = [], [0] * 5, [0, 1, 2, 3], [4]
    portions = [17, 2, 1, 30, 1, 1, 64]
    k = 0
    while live:
        entries, ended = [], []
        for r in live:
            n = min(portions[(k + r) % len(portions)], lengths[r] - pos[r])
            entries.append((r, pos[r], pos[r] + n))
            pos[r] += n
            if pos[r] == lengths[r]:
                ended.append(r)
        steps.append((entries, ended))
        live = [r for r in live if r not in ended]
        if ended and waiting:
            live.append(waiting.pop(0))
        k += 1
    lines = [json.dumps({"step": i, "entries": [{"id": f"r{r}", "tokens": ids[r][lo:hi], "want": list(range(hi - lo))} for r, lo, hi in entries],
                         "end": [f"r{r}" for r in ended]}) for i, (entries, ended) in enumerate(steps)]
    out_dir = str(tmp_path / "out")
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", out_dir,
                           "--max-tokens", "256"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    for i, (entries, _) in enumerate(steps):
        got = torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{i}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]))
        ref = torch.cat([want[r][lo:hi] for r, lo, hi in entries])
        assert zu.relative_error(got, ref) < zu.TOL["float32"], i
    prompt, new = ids[2][:9], 8
    seq = list(prompt)
    for _ in range(new):
        seq.append(int(zu.plain_logits(cfg, tensors, seq)[-1].argmax()))
    proc = subprocess.run([sys.executable, "-m", "llmgen_b200", "chat", ",".join(map(str, prompt)), str(new), "--model", folder, "--dtype", "float32",
                           "--max-model-len", "64", "--max-num-seqs", "2", "--max-batched-tokens", "64", "--kv-blocks", "8"],
                          capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert proc.returncode == 0, proc.stderr[-2000:]
    printed = [l.split() for l in proc.stdout.splitlines() if l.split() and all(t.lstrip("-").isdigit() for t in l.split())]
    assert printed and [int(t) for t in printed[-1]] == seq[len(prompt):], proc.stdout[-2000:]
    from llmgen_b200.info import describe
    text = describe(folder)
    assert "latent attention" in text and "reads cache 0" in text and "the keys are the values" in text and "every declared tensor is there" in text
