"""Kugisun through the engine against the plain implementation (tests/plain/kugisun_plain.py, float64 on the CPU): whole prompts,
portions, token by token, batches, pages and state slots used again, graphs replayed, generation."""
import copy

import pytest
import torch

from tests import kugisun_util as ku

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["MIXED", "WIDE", "ODD", "PLAIN"])
def test_whole_prompt_and_portions_match_the_plain_model(name, dtype):
    cfg = getattr(ku, name)
    model, tensors = ku.build(cfg, seed=3, dtype=dtype)
    ids = ku.ids_for(cfg, 75, seed=1)
    want = ku.plain_logits(cfg, tensors, ids)
    drv = ku.driver(model, dtype, pool_tokens=128)
    ku.assert_close(ku.run_in_portions(drv, "a", ids, [len(ids)]), want, dtype)
    ku.assert_close(ku.run_in_portions(drv, "a", ids, [33, 2, 1, 17, 1]), want, dtype)


def one_mechanism(which: str) -> dict:
    """One layer of MIXED alone, or its mixer with one branch silenced (a scale of zero)."""
    if which in ("dense", "routed"):
        layer = copy.deepcopy(ku.MIXED["layers"][0 if which == "dense" else 1])
        return ku.config([layer])
    layer = copy.deepcopy(ku.MIXED["layers"][0])
    layer["mlp"] = None
    layer["mixer"]["left_scale"], layer["mixer"]["right_scale"] = {"left": (1.3, 0.0), "right": (0.0, 0.8), "both": (-0.5, 0.9)}[which]
    return ku.config([layer], streams={"left": 4, "right": None, "both": 2}[which])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["left", "right", "both", "dense", "routed"])
def test_each_mechanism_in_a_layer_of_its_own(which, dtype):
    cfg = one_mechanism(which)
    model, tensors = ku.build(cfg, seed=7, dtype=dtype)
    ids = ku.ids_for(cfg, 90, seed=8)
    want = ku.plain_logits(cfg, tensors, ids)
    drv = ku.driver(model, dtype)
    ku.assert_close(ku.run_in_portions(drv, "a", ids, [90]), want, dtype, which)
    ku.assert_close(ku.run_in_portions(drv, "a", ids, [40, 1, 1, 7, 2]), want, dtype, which)


def silenced(cfg, tensors, ids, name):
    """The plain model's last logits with one tensor (or all that end with `name`) set to zero."""
    other = {n: (torch.zeros_like(t) if n.endswith(name) else t) for n, t in tensors.items()}
    return ku.plain_logits(cfg, other, ids)[-1:]


@pytest.mark.parametrize("name", [".q.b", ".v.b", ".q.norm", ".dt_bias", ".A_log", "right.b", "right.g", ".k.conv", ".correction", ".sg", "pos", "norm2", "hc1.mix"])
def test_every_tensor_counts(name):
    """Without it the plain model's last logits move far beyond the tolerance: a kernel that left it out would fail the tests
    of this file."""
    _, _, tensors = ku.draw(ku.MIXED, 3, 0.1, 0.2)
    for n, t in tensors.items():
        if n.endswith(".router"):
            t.mul_(4.0)
    ids = ku.ids_for(ku.MIXED, 24, seed=4)
    want = ku.plain_logits(ku.MIXED, tensors, ids)[-1:]
    assert ku.relative_error(silenced(ku.MIXED, tensors, ids, name), want) > 20 * ku.TOL["float32"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_of_any_size_and_single_tokens_give_the_whole_prompts_logits(dtype):
    cfg = ku.MIXED
    model, tensors = ku.build(cfg, seed=4, dtype=dtype)
    ids = ku.ids_for(cfg, 101, seed=2)
    want = ku.plain_logits(cfg, tensors, ids)
    drv = ku.driver(model, dtype)
    for portions in ([1], [2], [3, 2, 33, 31, 1, 16, 2], [32, 32, 5, 1], [47, 1, 1, 2], [17, 15, 16, 14, 1]):
        ku.assert_close(ku.run_in_portions(drv, "a", ids, portions), want, dtype, portions)
    assert drv.executor.cache.all_free()


@pytest.mark.parametrize("eager", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_that_cross_chunks_of_the_memory_and_tiles_of_the_attention(dtype, eager):
    """400 tokens whole, in portions that end inside, at and beside a chunk of 64 tokens, and beside another request; launched
    and replayed.  Steps of 256 rows and more run chunk by chunk, the others token by token."""
    cfg = ku.TENSOR
    model, tensors = ku.build(cfg, seed=15, dtype=dtype)
    ids, other = ku.ids_for(cfg, 400, seed=5), ku.ids_for(cfg, 150, seed=6)
    want, want_other = ku.plain_logits(cfg, tensors, ids), ku.plain_logits(cfg, tensors, other)
    drv = ku.driver(model, dtype, pool_tokens=640, eager=eager)
    ku.assert_close(ku.run_in_portions(drv, "a", ids, [400]), want, dtype)
    ku.assert_close(ku.run_in_portions(drv, "a", ids, [257, 1, 2, 63, 77]), want, dtype)
    ku.assert_close(ku.run_in_portions(drv, "a", ids, [10, 320, 70]), want, dtype)
    first = drv.step([("a", ids[:191], list(range(191))), ("b", other[:65], list(range(65)))])
    out = drv.step([("a", ids[191:], list(range(209))), ("b", other[65:], list(range(85)))], end=["a", "b"])
    ku.assert_close(torch.cat([first[:191], out[:209]]), want, dtype)
    ku.assert_close(torch.cat([first[191:], out[209:]]), want_other, dtype)


def test_the_logits_do_not_depend_on_the_cut_beyond_rounding():
    """float32: token by token, in twos and whole agree far inside the tolerance against the plain model."""
    for cfg, n in ((ku.WIDE, 80), (ku.TENSOR, 300)):
        model, _ = ku.build(cfg, seed=14, dtype="float32")
        ids = ku.ids_for(cfg, n, seed=3)
        drv = ku.driver(model, "float32", pool_tokens=128 if n < 128 else 512)
        whole = ku.run_in_portions(drv, "a", ids, [n])
        for portions in ([1], [2], [17, 3], [33, 33, 1]):
            assert ku.relative_error(ku.run_in_portions(drv, "a", ids, portions), whole) < 6e-6, portions


@pytest.mark.parametrize("eager", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch_match_each_alone(dtype, eager):
    """Three requests of different lengths, portions of some beside single tokens of others; launched kernel by kernel and
    replayed from the graphs of the steps' shapes."""
    cfg = ku.MIXED
    model, tensors = ku.build(cfg, seed=5, dtype=dtype)
    ids = {"a": ku.ids_for(cfg, 70, 11), "b": ku.ids_for(cfg, 19, 12), "c": ku.ids_for(cfg, 41, 13)}
    want = {r: ku.plain_logits(cfg, tensors, t) for r, t in ids.items()}
    drv = ku.driver(model, dtype, eager=eager)
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
        ku.assert_close(torch.cat(got[r]), want[r], dtype, r)
    if not eager:
        assert drv.executor.n_shaped_steps > 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_state_slots_are_used_again(dtype):
    """A pool of 6 pages and 2 state slots, five requests one after and beside another: every page and slot serves several
    requests, and a request that starts in a used slot starts from empty states and no token before its first."""
    cfg = ku.MIXED
    model, tensors = ku.build(cfg, seed=6, dtype=dtype)
    drv = ku.driver(model, dtype, pool_tokens=96, page_size=16, max_num_seqs=2)
    lengths = [40, 50, 33, 17, 48]
    all_ids = [ku.ids_for(cfg, n, 20 + i) for i, n in enumerate(lengths)]
    want = [ku.plain_logits(cfg, tensors, t) for t in all_ids]
    slots_seen = set()
    ku.assert_close(ku.run_in_portions(drv, 0, all_ids[0], [13, 27]), want[0], dtype)
    for a, b in ((1, 2), (3, 4)):
        got = {a: [], b: []}
        pos = {a: 0, b: 0}
        while any(pos[r] < lengths[r] for r in (a, b)):
            entries, sizes = [], []
            for r, n in ((a, 11), (b, 20 if pos[b] == 0 else 1)):
                n = min(n, lengths[r] - pos[r])
                if n:
                    entries.append((r, all_ids[r][pos[r]:pos[r] + n], list(range(n))))
                    sizes.append((r, n))
                    pos[r] += n
            out = drv.step(entries, end=[])
            slots_seen |= {drv.executor.cache.state.slot(r) for r, _, _ in entries}
            at = 0
            for r, n in sizes:
                got[r].append(out[at:at + n])
                at += n
                if pos[r] == lengths[r]:
                    drv.executor.release(r)
                    del drv.positions[r]
        for r in (a, b):
            ku.assert_close(torch.cat(got[r]), want[r], dtype, r)
    assert slots_seen == {0, 1}
    assert drv.executor.cache.all_free()


# (tokens, the needle's place, page size): the probe is the last token and sees every position up to itself
PLACES = [(300, 0, 16), (300, 298, 16), (300, 255, 16), (300, 256, 16), (289, 31, 32), (289, 32, 32), (273, 271, 16), (65, 63, 16), (65, 0, 64)]


@pytest.mark.parametrize("n,needle_at,page", PLACES)
def test_one_key_decides_however_far_away(n, needle_at, page):
    """The last token's query finds the key of one token only (`plant_needle`): the first, one beside a page's border, the
    newest but one.  Without it the plain model's logits differ by hundreds of tolerances.  Whole, in portions cut at and
    beside the needle, and with the probe decoded alone after single tokens."""
    cfg = ku.NEEDLE
    model, tensors = ku.build(cfg, seed=7, dtype="float32", sigma=0.3, prepare=ku.plant_needle)
    ids = ku.needle_ids(cfg, n, needle_at, 31)
    want = ku.plain_logits(cfg, tensors, ids)
    without = list(ids)
    without[needle_at] = ku.FILLER_ID
    assert ku.relative_error(ku.plain_logits(cfg, tensors, without)[-1:], want[-1:]) > 100 * ku.TOL["float32"]
    drv = ku.driver(model, "float32", pool_tokens=320, page_size=page)
    for portions in ((n,), (max(needle_at, 1), 1, 2, n), (needle_at + 1, 1, n), (max(n - 10, 1),) + (1,) * 10, (n - 1, 1)):
        got = ku.run_in_portions(drv, "a", ids, list(portions))
        assert ku.relative_error(got, want) < ku.TOL["float32"], portions
    assert drv.executor.cache.all_free()


@pytest.mark.parametrize("eager", [True, False])
def test_the_needle_in_the_bfloat16_engine_and_beside_other_requests(eager):
    cfg = copy.deepcopy(ku.NEEDLE)
    cfg["layers"][0]["mixer"]["left"]["vdim"] = 64           # the tensor-core attention takes these widths
    model, tensors = ku.build(cfg, seed=7, dtype="bfloat16", sigma=0.3, prepare=ku.plant_needle)
    n = 300
    ids = [ku.needle_ids(cfg, n, 1, 31), ku.needle_ids(cfg, n, 257, 32)]
    want = [ku.plain_logits(cfg, tensors, t) for t in ids]
    for t, at, w in zip(ids, (1, 257), want):
        without = list(t)
        without[at] = ku.FILLER_ID
        assert ku.relative_error(ku.plain_logits(cfg, tensors, without)[-1:], w[-1:]) > 5 * ku.TOL["bfloat16"]
    drv = ku.driver(model, "bfloat16", pool_tokens=640, eager=eager)
    for first in (n, 290):
        a = [drv.step([("a", ids[0][:first], list(range(first))), ("b", ids[1][:first], list(range(first)))], end=["a", "b"] if first == n else [])]
        for t in range(first, n):
            a.append(drv.step([("a", ids[0][t:t + 1], [0]), ("b", ids[1][t:t + 1], [0])], end=["a", "b"] if t == n - 1 else []))
        got = [torch.cat([a[0][:first]] + [x[:1] for x in a[1:]]), torch.cat([a[0][first:]] + [x[1:] for x in a[1:]])]
        for g, w in zip(got, want):
            ku.assert_close(g, w, "bfloat16", first)
            assert ku.relative_error(g[-1:], w[-1:]) < ku.TOL["bfloat16"]


def test_a_memory_that_forgets_little_is_carried_through_portions_and_long_decoding():
    cfg = ku.KEEPING
    model, tensors = ku.build(cfg, seed=8, dtype="float32", prepare=ku.keep_long)
    ids = ku.ids_for(cfg, 400, 41)
    want = ku.plain_logits(cfg, tensors, ids)
    drv = ku.driver(model, "float32", pool_tokens=448)
    for portions in ([400], [31, 33, 32, 1, 2, 64, 1], [300, 100], [100] + [1] * 300):
        got = ku.run_in_portions(drv, "a", ids, portions)
        assert ku.relative_error(got, want) < ku.TOL["float32"], portions[:3]
    # a state lost where a portion was cut would show at the next token (the positions' table is shifted along with the cut)
    for cut in (31, 100, 398):
        moved = dict(tensors, pos=tensors["pos"].roll(-cut, 0))
        restarted = ku.plain_logits(cfg, moved, ids[cut:cut + 2])
        assert ku.relative_error(restarted[:1], want[cut:cut + 1]) > 100 * ku.TOL["float32"], cut
    # and the first token still counts at the end: without it the last logits differ
    shifted = ku.plain_logits(cfg, dict(tensors, pos=tensors["pos"].roll(-1, 0)), ids[1:])
    assert ku.relative_error(shifted[-1:], want[-1:]) > 5 * ku.TOL["float32"]


@pytest.mark.parametrize("name", ["MIXED", "ODD", "PLAIN"])
def test_the_first_tokens_of_a_sequence(name):
    """One, two and three tokens: zeros before the start of a convolution, a memory that starts from nothing, a lone key."""
    cfg = getattr(ku, name)
    model, tensors = ku.build(cfg, seed=9, dtype="float32")
    drv = ku.driver(model, "float32", pool_tokens=128)
    for n in (1, 2, 3, 9):
        ids = ku.ids_for(cfg, n, 50 + n)
        for portions in ([1], [n]):
            got = ku.run_in_portions(drv, "a", ids, portions)
            assert ku.relative_error(got, ku.plain_logits(cfg, tensors, ids)) < ku.TOL["float32"], (n, portions)


def test_positions_end_with_their_table():
    """A sequence as long as the table of positions runs; a longer one is refused when the engine is built."""
    from llmgen_b200.engine.executor import EngineLimits, Executor, StepError
    cfg = ku.config([ku.layer(ku.left(2, 1, 8, 8, 0.3), ku.right(1, 1, 8, 8, 2), None)], width=16, vocab=31, streams=2, max_positions=40)
    model, tensors = ku.build(cfg, seed=2)
    ids = ku.ids_for(cfg, 40, 3)
    drv = ku.driver(model, "float32", pool_tokens=64)
    assert ku.relative_error(ku.run_in_portions(drv, "a", ids, [39, 1]), ku.plain_logits(cfg, tensors, ids)) < ku.TOL["float32"]
    with pytest.raises(StepError):
        Executor(model, EngineLimits(max_num_seqs=1, max_model_len=41, max_step_tokens=64, page_size=16, num_pages=4))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("eager", [True, False])
def test_greedy_generation_through_the_engine_and_its_scheduler(eager, dtype):
    """`LLM.generate` (scheduler, chunked prompts, decode graphs, sampling kernel) against greedy decoding with the plain
    model; bfloat16: the ids chosen are among the plain model's best two or three at every step of the engine's own text."""
    from llmgen_b200.engine.api import LLM
    from llmgen_b200.sampling.params import SamplingParams
    cfg = ku.MIXED if dtype == "float32" else ku.TENSOR
    model, tensors = ku.build(cfg, seed=10, dtype=dtype)
    prompts = [ku.ids_for(cfg, n, 60 + n) for n in (9, 21, 4)]
    new = 10
    llm = LLM(model, dtype=dtype, max_model_len=64, max_num_seqs=2, max_batched_tokens=64, pass_tokens=64, block_size=16,
              kv_blocks=8, policy="chunked", chunk=8, eager=eager, capture_at_start=False)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=new, ignore_eos=True))
    for p, o in zip(prompts, outs):
        text = list(p) + list(o["token_ids"])
        logits = ku.plain_logits(cfg, tensors, text)[len(p) - 1:-1]
        best = logits.max(dim=-1).values
        spread = logits.std(dim=-1)
        chosen = logits.gather(1, torch.tensor(o["token_ids"])[:, None])[:, 0]
        assert len(o["token_ids"]) == new
        if dtype == "float32":
            assert o["token_ids"] == logits.argmax(dim=-1).tolist()
        else:
            assert float(((best - chosen) / spread).quantile(0.9)) < 0.3
    assert llm.executor.cache.all_free()
    if not eager:
        assert llm.executor.n_graph_steps > 0


def test_single_tokens_in_the_bfloat16_engine_s_decode_graphs_match_the_plain_model():
    """Decoding by `LLM.generate` takes the graphs of single tokens (attention over key parts in a cluster, the memory's one
    launch); the logits of the text it wrote, fed as portions, are the plain model's."""
    from llmgen_b200.engine.api import LLM
    from llmgen_b200.sampling.params import SamplingParams
    cfg = ku.TENSOR
    model, tensors = ku.build(cfg, seed=12, dtype="bfloat16")
    prompt = ku.ids_for(cfg, 300, 77)
    llm = LLM(model, dtype="bfloat16", max_model_len=384, max_num_seqs=2, max_batched_tokens=384, pass_tokens=384, block_size=16, kv_blocks=48,
              capture_at_start=False)
    out = llm.generate([prompt, prompt[:130]], SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
    for p, o in zip((prompt, prompt[:130]), out):
        text = list(p) + list(o["token_ids"])
        logits = ku.plain_logits(cfg, tensors, text)[len(p) - 1:-1]
        gap = (logits.max(dim=-1).values - logits.gather(1, torch.tensor(o["token_ids"])[:, None])[:, 0]) / logits.std(dim=-1)
        assert float(gap.quantile(0.9)) < 0.3 and float(gap.median()) < 0.05


def test_a_model_folder_through_the_replay_program_and_the_command_line(tmp_path):
    """A Kugisun folder written by the random-weights mode, with the positions left to their table's shape: `bin/trace_run`
    replays a trace of five requests on four state slots and a pool smaller than their sum (float32 logits against the
    plain model), and `python -m llmgen_b200 chat` generates the plain model's greedy tokens."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np
    from safetensors.torch import load_file

    from llmgen_b200.engine.api import write_random_model
    from tests.util import ROOT
    cfg = ku.MIXED
    folder = write_random_model(str(tmp_path / "model"), cfg, seed=13, sigma=0.1, sigma_norm=0.2)
    path = os.path.join(folder, "config.json")
    with open(path) as f:
        written = json.load(f)
    assert written["architecture"] == "Kugisun"
    written.pop("max_positions")
    with open(path, "w") as f:
        json.dump(written, f)
    tensors = load_file(os.path.join(folder, "model.safetensors"))
    lengths = [70, 40, 23, 64, 51]
    ids = [ku.ids_for(cfg, n, 70 + i) for i, n in enumerate(lengths)]
    want = [ku.plain_logits(cfg, tensors, t) for t in ids]
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
        assert ku.relative_error(got, ref) < ku.TOL["float32"], i
    prompt, new = ids[2][:9], 8
    seq = list(prompt)
    for _ in range(new):
        seq.append(int(ku.plain_logits(cfg, tensors, seq)[-1].argmax()))
    proc = subprocess.run([sys.executable, "-m", "llmgen_b200", "chat", ",".join(map(str, prompt)), str(new), "--model", folder, "--dtype", "float32",
                           "--max-model-len", "64", "--max-num-seqs", "2", "--max-batched-tokens", "64", "--kv-blocks", "8"],
                          capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert proc.returncode == 0, proc.stderr[-2000:]
    printed = [l.split() for l in proc.stdout.splitlines() if l.split() and all(t.lstrip("-").isdigit() for t in l.split())]
    assert printed and [int(t) for t in printed[-1]] == seq[len(prompt):], proc.stdout[-2000:]
