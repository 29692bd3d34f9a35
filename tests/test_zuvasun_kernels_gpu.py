"""The kernels that Zuvasun added or widened, each by itself against the plain functions of tests/plain/zuvasun_plain.py (float64
on the CPU): the sum that ends a layer of two sublayers side by side, entries that are key and value at once (their
preparation and both attention kernels), queries straight into the latent space, latent attention under a window, the router's
correction and constants, and experts without a gate."""
import math

import pytest
import torch

from tests.plain import zuvasun_plain as plain

pytestmark = pytest.mark.gpu
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DEV = "cuda:0"


def rnd(shape, seed, scale=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * scale).to(dtype)


def close(got, want, tol):
    err = float((got.double().cpu() - want.double()).abs().max() / want.double().abs().max())
    assert err < tol, err


def ints(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H", [40, 37, 260, 2052])
def test_parallel_add_ends_a_layer_of_two_sublayers(H, dtype):
    """Arrays, float32 slices and routed rows, with and without gains, with and without the next layer's norm."""
    from llmgen_b200.kernels import ops
    dt, n, top, slots = DT[dtype], 7, 3, 30
    resid = rnd((n, H), 1)
    ga, gb, gain = rnd((H,), 2), rnd((H,), 3), 1 + rnd((H,), 4, 0.2)
    y1, s1, y2, s2 = rnd((n, H), 5, 1.0, dt), rnd((4, n, H), 6), rnd((n, H), 7, 1.0, dt), rnd((2, n, H), 8)
    rows, weights = rnd((slots, H), 9), rnd((n * top,), 10).abs()
    pos = torch.randperm(slots, generator=torch.Generator().manual_seed(11))[:n * top].to(torch.int32)
    pos[4] = -1                                                          # a slot nobody computed adds nothing
    routed = lambda w: torch.stack([sum((float(weights[t * top + k]) if w else 1.0) * rows[pos[t * top + k]].double()
                                        for k in range(top) if pos[t * top + k] >= 0) for t in range(n)])
    d = lambda x: x.to(DEV)
    seconds = [(None, None), (d(y2), y2.double()), (ops.Partials(d(s2)), s2.double().sum(0)),
               (ops.RoutedRows(d(rows), d(pos), d(weights), top), routed(True)), (ops.RoutedRows(d(rows), d(pos), None, top), routed(False))]
    for first, f64 in ((d(y1), y1.double()), (ops.Partials(d(s1)), s1.double().sum(0))):
        for second, s64 in seconds:
            for gains in (True, False):
                want = resid.double() + (ga.double() if gains else 1.0) * f64
                if s64 is not None:
                    want = want + (gb.double() if gains else 1.0) * s64
                r, normed = d(resid.clone()), torch.zeros(n, H, dtype=dt, device=DEV)
                ops.parallel_add(r, first, d(ga) if gains else None, second, d(gb) if gains else None, dt, next_gain=d(gain), eps=1e-5, normed=normed)
                close(r, want, 1e-6)
                close(normed, plain.rmsnorm(want, gain.double(), 1e-5), 1e-5 if dtype == "float32" else 1e-2)
                r2 = d(resid.clone())
                ops.parallel_add(r2, first, d(ga) if gains else None, second, d(gb) if gains else None, dt)
                assert torch.equal(r2, r)
    out = torch.zeros(1, n, H, device=DEV)
    close(seconds[3][0].sum(out).tensor[0], seconds[3][1], 1e-6)


def entries(n_keys, nkv, hd, page, dt, seed):
    """Projected keys in shuffled pages with their rows' inverse root mean squares: (keys, factors, cache, k_scale, block table)."""
    k = rnd((n_keys, nkv, hd), seed, 1.0, dt)
    factor = 1.0 / torch.sqrt(k.double().pow(2).mean(dim=(1, 2)) + 1e-5)
    pages = (n_keys + page - 1) // page
    order = torch.randperm(pages + 2, generator=torch.Generator().manual_seed(seed + 1))[:pages]
    kc = torch.full((pages + 2, nkv, page, hd), 9.0, dtype=dt)
    ks = torch.full((pages + 2, page), 9.0)
    for j in range(n_keys):
        kc[order[j // page], :, j % page], ks[order[j // page], j % page] = k[j], float(factor[j])
    return k.double(), factor, kc.to(DEV), ks.to(DEV), order.to(torch.int32).to(DEV)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("form", ["array", "slices"])
@pytest.mark.parametrize("nq,nk,hd", [(4, 2, 16), (3, 1, 9), (6, 6, 8), (20, 1, 24), (8, 4, 128)])
def test_keys_are_cached_once_as_projected_with_their_norm_as_one_number(nq, nk, hd, form, dtype):
    from llmgen_b200.kernels import ops
    dt, n, page, pages, eps, coef, every = DT[dtype], 9, 4, 6, 1e-4, 0.4, 7.0
    C = (nq + nk) * hd
    x = rnd((n, C), 1, 1.0, dt) if form == "array" else rnd((3, n, C), 1)
    x64 = x.double() if form == "array" else x.double().sum(0)
    bias, qg, kg = rnd((C,), 2, 0.5), 1 + rnd((nq * hd,), 3, 0.3), 1 + rnd((nk * hd,), 4, 0.3)
    gains = (qg.view(nk, nq // nk, hd) * kg.view(nk, 1, hd)).reshape(-1)
    pos, slots = [0, 5, 6, 7, 13, 14, 1000, 6999, 6998], [20, 21, 22, 3, -1, 9, 10, 11, 0]
    kc = torch.full((pages, nk, page, hd), 7.0, dtype=dt, device=DEV)
    ks = torch.full((pages, page), 7.0, device=DEV)
    q = torch.zeros(n, nq * hd, dtype=dt, device=DEV)
    src = x.to(DEV) if form == "array" else ops.Partials(x.to(DEV))
    ops.attn_prep_shared_rows(src, bias.to(DEV), q, kc, ks, ints(pos), ints(slots), gains.to(DEV), nq, nk, hd, page, eps, coef, every)
    x64 = x64 + bias.double()
    temp = torch.tensor([plain.query_temperature({"q_temp": {"coef": coef, "every": every}}, p) for p in pos], dtype=torch.float64)
    # the query as the attention uses it against keys as projected: its own norm and gains, and the key's gains
    want_q = plain.rmsnorm(x64[:, :nq * hd], qg.double(), eps) * temp[:, None]
    want_q = (want_q.view(n, nk, nq // nk, hd) * kg.double().view(1, nk, 1, hd)).reshape(n, -1)
    close(q, want_q, 1e-5 if dtype == "float32" else 1e-2)
    used = set()
    for t, s in enumerate(slots):
        if s < 0:
            continue
        used.add(s)
        k64 = x64[t, nq * hd:]
        close(kc[s // page, :, s % page].reshape(-1), k64, 1e-6 if dtype == "float32" else 1e-2)
        assert abs(float(ks[s // page, s % page]) * float(torch.sqrt(k64.pow(2).mean() + eps)) - 1.0) < 1e-5
    for s in range(pages * page):
        if s not in used:
            assert float(kc[s // page, :, s % page].float().min()) == 7.0 and float(ks[s // page, s % page]) == 7.0
    # without a temperature, positions change nothing
    q2, q3 = torch.zeros_like(q), torch.zeros_like(q)
    ops.attn_prep_shared_rows(src, None, q2, kc, ks, ints(pos), ints(slots), gains.to(DEV), nq, nk, hd, page, eps)
    ops.attn_prep_shared_rows(src, None, q3, kc, ks, ints([0] * n), ints(slots), gains.to(DEV), nq, nk, hd, page, eps)
    assert torch.equal(q2, q3)


def shared_attention(q, k, factor, n_keys, nq, nkv, hd, scale):
    """float64: query rows are the last of the n_keys positions."""
    T = q.shape[0]
    out = torch.zeros(T, nq, hd, dtype=torch.float64)
    for i in range(T):
        last = n_keys - T + i
        for h in range(nq):
            g = h // (nq // nkv)
            w = plain.softmax_row((k[:last + 1, g] @ q[i, h * hd:(h + 1) * hd].double()) * factor[:last + 1] * scale)
            out[i, h] = w @ k[:last + 1, g]
    return out.reshape(T, nq * hd)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nq,nkv,hd,page", [(4, 2, 16, 16), (3, 1, 9, 16), (20, 1, 24, 32), (6, 3, 64, 16), (2, 1, 130, 16)])
def test_attention_over_entries_that_are_key_and_value(nq, nkv, hd, page, dtype):
    """The general kernel: a portion of 21 queries, a single token whole and with its keys in parts."""
    from llmgen_b200.kernels import ops
    dt, n_keys, T, scale = DT[dtype], 300, 21, 0.3
    k, factor, kc, ks, bt = entries(n_keys, nkv, hd, page, dt, 5)
    q = rnd((T, nq * hd), 6, 1.0, dt)
    want = shared_attention(q, k, factor, n_keys, nq, nkv, hd, scale)
    tol = 2e-5 if dtype == "float32" else 1e-2
    bq = ops.attention_tile_queries(nq, nkv)
    starts = list(range(0, T, bq))
    out = torch.zeros(T, nq * hd, dtype=dt, device=DEV)
    ops.paged_attention(out, q.to(DEV), nq * hd, kc, None, bt, bt.numel(), ints([n_keys]), ints([0, T]), ints([0] * len(starts)), ints(starts),
                        len(starts), T, nq, nkv, hd, page, 0, scale, k_scale=ks)
    close(out, want, tol)
    for parts in (1, 2, 5):
        one = torch.zeros(1, nq * hd, dtype=dt, device=DEV)
        scratch = torch.zeros(ops.attention_scratch_floats(1, nq, hd, parts), device=DEV) if parts > 1 else None
        ops.paged_attention(one, q[T - 1:].to(DEV), nq * hd, kc, None, bt, bt.numel(), ints([n_keys]), ints([0, 1]), ints([0]), ints([0]), 1, 1, nq,
                            nkv, hd, page, 0, scale, parts, 0, scratch, k_scale=ks)
        close(one, want[T - 1:], tol)


@pytest.mark.parametrize("nq,nkv,hd,page", [(6, 3, 64, 16), (2, 1, 128, 32), (4, 4, 128, 16)])
@pytest.mark.parametrize("T", [64, 150, 5])
def test_tensor_core_attention_over_entries_that_are_key_and_value(nq, nkv, hd, page, T):
    from llmgen_b200.kernels import ops
    n_keys, scale = 290, 0.25
    k, factor, kc, ks, bt = entries(n_keys, nkv, hd, page, torch.bfloat16, 5)
    q = rnd((T, nq * hd), 6, 1.0, torch.bfloat16)
    want = shared_attention(q, k, factor, n_keys, nq, nkv, hd, scale)
    bq = ops.attention_mma_tile_queries(nq, nkv, hd, hd)
    starts = list(range(0, T, bq))
    out = torch.zeros(T, nq * hd, dtype=torch.bfloat16, device=DEV)
    ops.attention_mma(out, q.to(DEV), kc, None, bt, bt.numel(), ints([n_keys]), ints([0, T]), ints([0] * len(starts) + [-1]), ints(starts + [0]),
                      len(starts) + 1, nq, nkv, hd, hd, page, 0, scale, k_scale=ks)
    close(out, want, 1e-2)


@pytest.mark.parametrize("nq,nkv,hd,vd,page,shared", [
    (6, 3, 64, 64, 16, True), (2, 1, 128, 128, 32, True), (4, 4, 128, 128, 16, True), (20, 1, 64, 64, 16, True),
    (6, 3, 64, 64, 48, False), (4, 4, 128, 128, 16, False), (20, 1, 64, 64, 16, False), (4, 2, 64, 128, 16, False), (6, 2, 128, 64, 16, False)])
def test_single_tokens_on_the_tensor_cores_with_their_keys_in_a_cluster_of_parts(nq, nkv, hd, vd, page, shared):
    """Sequences of 1 to 300 keys in one step, one without a token and one of padding, parts beyond the keys there are; windows,
    blocks of positions, a bound on the scores and sinks; entries that are key and value, or two arrays."""
    from llmgen_b200.kernels import ops
    scale, lens = 0.25, [300, 1, 64, 65, 0, 130]
    seqs = [entries(max(n, 1), nkv, hd, page, torch.bfloat16, 5 + 2 * i) for i, n in enumerate(lens)]
    values = [rnd((max(n, 1), nkv, vd), 40 + i, 1.0, torch.bfloat16) for i, n in enumerate(lens)]
    sizes = [s[2].shape[0] for s in seqs]
    base = [sum(sizes[:i]) for i in range(len(sizes))]
    kc, ks = torch.cat([s[2] for s in seqs]), torch.cat([s[3] for s in seqs])
    vc = torch.zeros(kc.shape[0], nkv, page, vd, dtype=torch.bfloat16, device=DEV)
    most = max(s[4].numel() for s in seqs)
    bt = torch.full((len(lens), most), -1, dtype=torch.int32, device=DEV)
    for i, s in enumerate(seqs):
        bt[i, :s[4].numel()] = s[4] + base[i]
        for j in range(values[i].shape[0]):
            vc[int(bt[i, j // page]), :, j % page] = values[i][j].to(DEV)
    cu = [0, 1, 2, 3, 4, 5, 6]
    q = rnd((6, nq * hd), 6, 1.0, torch.bfloat16)
    sinks = rnd((nq,), 7, 2.0)
    forms = [dict(), dict(window=70), dict(chunk=96, softcap=3.0), dict(sink=True), dict(sink=True, sink_values=sinks.to(DEV), window=33)]
    for form in forms:
        window, chunk, cap = form.get("window", 0), form.get("chunk", 0), form.get("softcap", 0.0)
        want = torch.zeros(6, nq, vd, dtype=torch.float64)
        for i, n in enumerate(lens):
            if n == 0:
                continue
            first = max(0, n - window) if window else (n - 1) // chunk * chunk if chunk else 0
            for h in range(nq):
                g = h // (nq // nkv)
                sc = seqs[i][0][first:n, g] @ q[i, h * hd:(h + 1) * hd].double() * scale
                if shared:
                    sc = sc * seqs[i][1][first:n]
                if cap:
                    sc = cap * torch.tanh(sc / cap)
                e = torch.exp(sc - sc.max())
                sink = math.exp((float(sinks[h]) if "sink_values" in form else 0.0) - float(sc.max())) if form.get("sink") else 0.0
                v = seqs[i][0][first:n, g] if shared else values[i][first:n, g].double()
                want[i, h] = (e / (e.sum() + sink)) @ v
        for parts in (1, 3, 8):
            out = torch.full((6, nq * vd), 5.0, dtype=torch.bfloat16, device=DEV)
            ops.attention_mma_parts(out, q.to(DEV), kc, None if shared else vc, bt, most, ints(lens), ints(cu), 6, nq, nkv, hd, vd, page, window, scale,
                                    parts, softcap=cap, sink=form.get("sink", False), chunk=chunk, sink_values=form.get("sink_values"),
                                    k_scale=ks if shared else None)
            for i, n in enumerate(lens):
                if n:
                    close(out[i], want[i].reshape(-1), 1e-2)
                else:
                    assert float(out[i].float().abs().max()) == 0.0


def test_values_and_factors_exclude_each_other():
    from llmgen_b200.kernels import ops
    k, factor, kc, ks, bt = entries(16, 1, 64, 16, torch.bfloat16, 5)
    q, out = rnd((1, 64), 1, 1.0, torch.bfloat16).to(DEV), torch.zeros(1, 64, dtype=torch.bfloat16, device=DEV)
    for v, s in ((None, None), (kc, ks), (None, ks.double()), (None, ks[:1])):
        with pytest.raises(ops.KernelError):
            ops.paged_attention(out, q, 64, kc, v, bt, 1, ints([16]), ints([0, 1]), ints([0]), ints([0]), 1, 1, 1, 1, 64, 16, 0, 0.3, k_scale=s)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,window", [
    (3, 16, 8, 24, 32, 24), (5, 7, 6, 5, 18, 0), (37, 8, 4, 8, 16, 2), (2, 10, 4, 6, 16, 1), (2, 8, 48, 16, 40, 33),
    (5, 24, 16, 40, 64, 50), (34, 16, 16, 8, 64, 33), (2, 32, 32, 64, 128, 0), (6, 8, 64, 16, 512, 40), (3, 16, 16, 24, 192, 130)])
def test_latent_attention_with_direct_queries_under_a_window(heads, dim, rot, vdim, rank, window, dtype):
    """Queries into the latent space with the entries written in the same launch (`latent_absorb`; in bfloat16, sizes that fit:
    `latent_split` and the grouped product), attention whole and as a step of single tokens in key parts, and the expansion,
    against keys and values expanded per head; shuffled pages, a table whose passed pages are gone."""
    from llmgen_b200.kernels import ops
    dt = DT[dtype]
    T, page, eps = 77, 16, 1e-5
    za, hd = rank + rot, dim + rot
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": 0.8 / (dim + rot) ** 0.5,
         "rot": {"base": 200.0, "dims": rot, "scaling": {"factor": 3.0, "original": 100, "fast": 8.0, "slow": 1.0}}}
    if window:
        m["mask"] = {"size": window}
    w = {"q": rnd((heads * hd, 32), 1, 0.3, dt), "dkv": rnd((za, 32), 4, 0.3, dt), "dkv.norm": 1 + rnd((rank,), 5, 0.2),
         "uk": rnd((heads * dim, rank), 6, 0.5 / rank ** 0.5 * 2, dt), "uv": rnd((heads * vdim, rank), 7, 0.3, dt), "o": torch.eye(heads * vdim)}
    h = rnd((T, 32), 9, 1.0, dt)
    p64 = {k: v.double() for k, v in w.items()}
    want = plain.latent_attention(h.double(), p64, m, plain.latent_entries(h.double(), p64, m, eps))
    pad = 8 - (heads * hd + za) % 8
    packed = torch.cat([h.float() @ w["q"].float().t(), h.float() @ w["dkv"].float().t(), torch.zeros(T, pad)], dim=1).to(dt).to(DEV)
    table = [4, 0, 3, 1, 2]
    pos = torch.arange(T, dtype=torch.int32, device=DEV)
    slots = ints([table[p // page] * page + p % page for p in range(T)])
    speeds, factor = plain.turning_speeds(m["rot"])
    ang = torch.arange(T, dtype=torch.float64)[:, None] * torch.tensor(speeds, dtype=torch.float64)[None, :]
    cos, sin = (factor * ang.cos()).float().to(DEV).contiguous(), (factor * ang.sin()).float().to(DEV).contiguous()
    cache = torch.zeros(5, 1, page, za, dtype=dt, device=DEV)
    kg, uk = w["dkv.norm"].to(DEV), w["uk"].to(DEV)
    qa = torch.empty(T, heads * za, device=DEV)
    ops.latent_absorb(qa, packed, uk, pos, cos, sin, heads, dim, rot, rank, "interleaved", dkv=packed[:, heads * hd:], kv_gain=kg, eps=eps,
                      cache=cache, slots=slots)
    bq = ops.latent_attention_tile_queries(heads)
    starts = list(range(0, T, bq))
    tiles = (ints([0] * len(starts)), ints(starts))
    oa = torch.empty(T, heads * rank, device=DEV)
    scale = m["scale"]
    ops.latent_attention(oa, qa, cache, ints(table), 5, ints([T]), ints([0, T]), *tiles, T, heads, rank, rot, page, scale, window=window)
    y = torch.empty(T, heads * vdim, dtype=dt, device=DEV)
    ops.latent_expand(y, oa, w["uv"].to(DEV), None, heads, rank, vdim)
    tol = 3e-5 if dtype == "float32" else 3e-2
    close(y, want, tol)
    # the last token alone, its visible keys cut into parts (more than it has keys for, too); pages behind the window are gone
    passed = max(0, T - window) // page if window else 0
    gone = [-1] * passed + table[passed:]
    for parts in (1, 3, 9):
        scratch = torch.empty(ops.latent_attention_scratch_floats(1, heads, rank, parts), device=DEV) if parts > 1 else None
        o1 = torch.empty(1, heads * rank, device=DEV)
        ops.latent_attention(o1, qa[T - 1:], cache, ints(gone), 5, ints([T]), ints([0, 1]), ints([0]), ints([0]), 1, heads, rank, rot, page,
                             scale, parts, scratch, window=window)
        close(o1, oa[T - 1:].cpu(), 2e-5)
    if dtype == "bfloat16" and ops.latent_attention_on_tensor_cores(dt, rank, rot) and dim % 8 == 0 and rot % 8 == 0:
        # whole portions: unrotated parts head-major through the grouped product, queries head-major in bfloat16
        t_pad = 128
        qn = torch.zeros(heads * t_pad, dim, dtype=dt, device=DEV)
        hm = torch.zeros(heads * t_pad, za, dtype=dt, device=DEV)
        cache2 = torch.zeros_like(cache)
        ops.latent_split(packed, heads * hd, qn.view(heads, t_pad, dim), hm.view(heads, t_pad, za), pos, cos, sin, heads, dim, rot, rank,
                         "interleaved", kv_gain=kg, eps=eps, cache=cache2, slots=slots)
        assert torch.equal(cache2, cache)
        ukt = uk.view(heads, dim, rank).transpose(1, 2).contiguous()
        ops.gemm_tc_grouped(hm[:, :rank], qn, ukt, torch.arange(heads, dtype=torch.int32, device=DEV))
        close(hm.view(heads, t_pad, za)[:, :T].permute(1, 0, 2).reshape(T, heads * za).float(), qa.cpu(), 1e-2)
        out = torch.zeros(heads, t_pad, rank, dtype=dt, device=DEV)
        ops.latent_attention(None, None, cache, ints(table), 5, ints([T]), ints([0, T]), *tiles, T, heads, rank, rot, page, scale,
                             out_head_major=out, window=window, q_head_major=hm.view(heads, t_pad, za))
        close(out[:, :T].permute(1, 0, 2).reshape(T, heads * rank).float(), oa.cpu(), 2e-2)


@pytest.mark.parametrize("T", [5, 90, 700])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,E,F,top", [(40, 7, 24, 2), (36, 5, 10, 3), (64, 33, 16, 4), (48, 1, 8, 1), (72, 80, 8, 6)])
def test_experts_without_a_gate_chosen_by_corrected_scores(H, E, F, top, dtype, T):
    """The part itself on rows of its own: the choice by score plus correction, the weights, both products, the sum; and the
    same rows handed over before their sum."""
    from llmgen_b200.engine.context import Workspace
    from llmgen_b200.kernels import ops
    from llmgen_b200.parts.moe import RoutedMLP
    from llmgen_b200.parts.registry import model_weight_decls  # noqa: F401  (registers the parts)
    from llmgen_b200.parts.spec import PlainExpertSpec, RoutedMLPSpec
    from llmgen_b200.weights import random_tensors, weights_from_dict
    dev, dt = torch.device(DEV), DT[dtype]
    spec = RoutedMLPSpec(H, "router", tuple(PlainExpertSpec(F, f"e{j}.up", f"e{j}.down") for j in range(E)), top, scoring="softmax",
                         renormalize=True, weight_on_input=False, choice_bias="correction", weight_scale=1.6, sum_eps=1e-20)
    decls = RoutedMLP.weight_decls(spec)
    tensors = random_tensors(decls, 5, 0.3, 0.1, torch.bfloat16)
    tensors["correction"][0] += 0.3                                     # the first expert is chosen by most rows: more than one tile
    part = RoutedMLP(spec, weights_from_dict(tensors, decls), dt, dev)

    class Ctx:
        workspace = Workspace(dev, max(T, 128))
    x = rnd((T, H), 9, 1.0, dt)
    got = part.forward(Ctx, x.to(dev)).sum()
    p64 = {k: v.double() for k, v in tensors.items()}
    want = plain.routed_ff(x.double(), p64, {"router": {"experts": E, "top": top, "scale": 1.6}})
    close(got, want, 2e-5 if dtype == "float32" else 2e-2)
    rows = part.forward(Ctx, x.to(dev), combine=False)
    assert isinstance(rows, ops.RoutedRows)
    assert torch.equal(rows.sum(torch.zeros(1, T, H, device=DEV)).tensor[0], got)


def test_the_chosen_scores_sum_may_vanish():
    """Corrections that choose experts whose scores are far below float32's smallest beside the largest: the sum's own 1e-20
    keeps the weights finite, as in the plain model."""
    from llmgen_b200.kernels import ops
    E, K = 4, 8
    router = torch.zeros(E, K)
    router[0, 0] = 200.0
    h = torch.zeros(2, K)
    h[:, 0] = torch.tensor([1.0, 0.3])
    corr = torch.tensor([-9.0, 1.0, 2.0, 0.0])
    expert, weight = torch.zeros(4, dtype=torch.int32, device=DEV), torch.zeros(4, device=DEV)
    ops.moe_route(h.to(DEV), router.to(DEV), expert, weight, 2, "softmax", True, choice_bias=corr.to(DEV), weight_scale=2.0, sum_eps=1e-20)
    assert expert.tolist() == [2, 1, 2, 1]
    for t in range(2):
        _, w = plain.choose((router @ h[t]).double(), corr.double(), 2, 2.0)
        for k in range(2):
            assert abs(float(weight[2 * t + k]) - w[k]) < 1e-5 + 1e-4 * abs(w[k]) and math.isfinite(float(weight[2 * t + k]))


@pytest.mark.parametrize("N", [40, 64, 136, 320])
def test_the_grouped_product_squares_its_relu_in_the_epilogue(N):
    from llmgen_b200.kernels import ops
    K, groups, tiles = 72, 3, [2, 0, -1, 1]
    a, w = rnd((128 * len(tiles), K), 1, 1.0, torch.bfloat16), rnd((groups, N, K), 2, 0.3, torch.bfloat16)
    out = torch.full((128 * len(tiles), N), 3.0, dtype=torch.bfloat16, device=DEV)
    ops.gemm_tc_grouped(out, a.to(DEV), w.to(DEV), ints(tiles), activation="relu2")
    for i, g in enumerate(tiles):
        rows = slice(128 * i, 128 * (i + 1))
        if g < 0:
            assert float(out[rows].float().min()) == 3.0
        else:
            close(out[rows], torch.relu(a[rows].double() @ w[g].double().t()) ** 2, 1e-2)
    with pytest.raises(ops.KernelError):
        ops.gemm_tc_grouped(torch.zeros(128, N, device=DEV), a[:128].to(DEV), w.to(DEV), ints([0]), activation="relu2")
