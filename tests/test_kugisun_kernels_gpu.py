"""The kernels that Kugisun added or widened, each by itself against the plain functions of tests/plain/kugisun_plain.py (float64
on the CPU): learned positions, biases and turned neighbours in front of the attention, the memory with one decay per head in its
three forms and what precedes it, the router's groups, identities and gate, and the streams' step for rows of vectors."""
import pytest
import torch

from tests.plain import kugisun_plain as plain

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


def cumulative(lens):
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    return cu


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H", [37, 64, 1024])
def test_learned_positions_join_the_embedding(H, dtype):
    from llmgen_b200.kernels import ops
    dt = DT[dtype]
    table, pos = rnd((20, H), 1, 1.0, dt), rnd((9, H), 2, 1.0, dt)
    ids, places = [3, 19, 0, 3, 7], [0, 8, 4, 4, 1]
    out = torch.zeros(5, H, device=DEV)
    ops.embed_rows(out, table.to(DEV), ints(ids), scale=1.5, position_table=pos.to(DEV), positions=ints(places))
    close(out, 1.5 * table.double()[ids] + pos.double()[places], 1e-6)
    # a sampled id takes the place of a row's own
    ops.embed_rows(out, table.to(DEV), ints(ids), ids_from=ints([-1, 1, -1, -1, 0]), sampled=ints([11, 12]), position_table=pos.to(DEV), positions=ints(places))
    close(out, table.double()[[3, 12, 0, 3, 11]] + pos.double()[places], 1e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nq,nk,hd,vd,rot", [(4, 2, 64, 128, 16), (3, 3, 16, 8, 16), (8, 1, 32, 40, 8), (2, 1, 128, 64, 64), (2, 2, 24, 24, 0), (5, 1, 10, 6, 4),
                                             (1, 1, 256, 16, 8)])
def test_biases_norms_and_turned_neighbours_in_front_of_the_attention(nq, nk, hd, vd, rot, dtype):
    """Rows inside a wider packed array; q to its place, k and v to the cache; whole vectors and sizes that are none."""
    from llmgen_b200.kernels import ops
    dt, n, page = DT[dtype], 37, 16
    cols = (nq + nk) * hd + nk * vd
    x = rnd((n, cols + 8), 1, 1.0, dt)
    bias, gq, gk = rnd((cols,), 2), 1 + rnd((hd,), 3, 0.2), 1 + rnd((hd,), 4, 0.2)
    places = torch.randperm(200, generator=torch.Generator().manual_seed(5))[:n]
    slots = torch.randperm(4 * page, generator=torch.Generator().manual_seed(6))[:n].to(torch.int32)
    slots[3] = -1
    half = rot // 2
    freq = torch.tensor([50.0 ** (-2.0 * i / rot) for i in range(half)], dtype=torch.float64) if rot else None
    angles = torch.arange(200, dtype=torch.float64)[:, None] * freq if rot else None
    kc, vc = torch.full((4, nk, page, hd), 9.0, dtype=dt, device=DEV), torch.full((4, nk, page, vd), 9.0, dtype=dt, device=DEV)
    q = torch.zeros(n, nq * hd, dtype=dt, device=DEV)
    ops.attn_prep(x.to(DEV)[:, :cols], kc, vc, ints(places.tolist()), slots.to(DEV), angles.cos().float().to(DEV) if rot else None,
                  angles.sin().float().to(DEV) if rot else None, gq.to(DEV), gk.to(DEV), nq, nk, hd, rot, page, 1e-5, q_out=q, pairing="interleaved",
                  bias=bias.to(DEV), vd=vd)
    y = x[:, :cols].double() + bias.double()
    turn = lambda h, t: plain.turn_neighbours(h, int(places[t]), {"base": 50.0, "dims": rot})
    wq = plain.rmsnorm(y[:, :nq * hd].view(n, nq, hd), gq.double(), 1e-5)
    wk = plain.rmsnorm(y[:, nq * hd:(nq + nk) * hd].view(n, nk, hd), gk.double(), 1e-5)
    tol = 1e-5 if dtype == "float32" else 1e-2
    close(q, torch.stack([turn(wq[t], t) for t in range(n)]).reshape(n, -1), tol)
    want_k, want_v = torch.full((4, nk, page, hd), 9.0, dtype=torch.float64), torch.full((4, nk, page, vd), 9.0, dtype=torch.float64)
    for t in range(n):
        s = int(slots[t])
        if s >= 0:
            want_k[s // page, :, s % page] = turn(wk[t], t)
            want_v[s // page, :, s % page] = y[t, (nq + nk) * hd:].view(nk, vd)
    close(kc, want_k, tol)
    close(vc, want_v, tol)


SIZES = [(2, 1, 32, 48), (6, 3, 32, 16), (4, 2, 128, 128), (3, 3, 20, 12), (4, 4, 48, 72), (2, 1, 64, 40), (4, 1, 10, 7), (20, 10, 128, 136)]


def memory_case(lens, H, G, D, E, seed, log_decay=0.03):
    """Prepared rows of sequences of the given lengths (a common part in all keys, so that they overlap), and their states."""
    n, C = sum(lens), 2 * G * D + H * E
    q = plain.unit(rnd((n, G, D), seed)) * D ** -0.5
    k = plain.unit(rnd((n, G, D), seed + 1) + rnd((1, G, D), seed + 2))
    v, beta = rnd((n, H, E), seed + 3), torch.rand((n, H), generator=torch.Generator().manual_seed(seed + 4))
    log_g = -log_decay * torch.rand((n, H), generator=torch.Generator().manual_seed(seed + 5))
    qkv = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], dim=1).contiguous()
    gates = torch.cat([beta, log_g, (q * k).sum(-1)], dim=1).contiguous()
    state = rnd((len(lens) + 1, H * D * E + 5), seed + 6)
    return (q, k, v, beta, log_g), qkv, gates, state, cumulative(lens), list(range(len(lens)))[::-1]


def run_memory(form, qkv, gates, state, cu, slots, H, G, D, E):
    from llmgen_b200.kernels import ops
    n = qkv.shape[0]
    out, st = torch.full((n, H * E), 7.0, device=DEV), state.to(DEV)
    args = (out, qkv.to(DEV), gates.to(DEV), st, ints(cu), ints(slots))
    if form == "tokens":
        ops.delta_scan_heads(*args, len(slots), H, G, D, E)
    else:
        floats = ops.head_delta_chunk_floats(n, len(slots), H, G, D, E)
        assert floats > 0
        ops.head_delta_chunks(*args, torch.full((floats,), float("nan"), device=DEV), len(slots), H, G, D, E)
    return out, st


@pytest.mark.parametrize("form", ["tokens", "chunks"])
@pytest.mark.parametrize("H,G,D,E", SIZES)
def test_the_memory_token_by_token_and_chunk_by_chunk(H, G, D, E, form):
    """Sequences of one token, of less than, exactly and just beyond a chunk of 64, and of none, from states that hold
    something; columns behind the state and a slot nobody owns stay as they are."""
    lens = [1, 0, 63, 64, 65, 130] if H * D * E < 100000 else [1, 70]
    (q, k, v, beta, log_g), qkv, gates, state, cu, slots = memory_case(lens, H, G, D, E, 10)
    out, st = run_memory(form, qkv, gates, state, cu, slots, H, G, D, E)
    for i, n in enumerate(lens):
        a, b = cu[i], cu[i + 1]
        S = state[slots[i], :H * D * E].view(H, D, E).double()
        if n:
            o, S = plain.delta_memory(q[a:b].double(), k[a:b].double(), v[a:b].double(), beta[a:b].double(), log_g[a:b].double().exp(), S)
            close(out[a:b].view(n, H, E), o, 3e-6)
        close(st[slots[i], :H * D * E].view(H, D, E), S, 3e-6)
    assert torch.equal(st[:, H * D * E:].cpu(), state[:, H * D * E:]) and torch.equal(st[len(lens)].cpu(), state[len(lens)])


@pytest.mark.parametrize("form", ["tokens", "chunks"])
def test_a_memory_that_keeps_its_state_over_thousands_of_tokens(form):
    """Decays just below one: what a float32 holds of 1 - g must not be lost at every token (or chunk)."""
    H, G, D, E = 1, 1, 16, 8
    (q, k, v, beta, log_g), qkv, gates, state, cu, slots = memory_case([3000], H, G, D, E, 30, log_decay=1e-4)
    beta *= 0.01
    gates[:, :H] = beta
    out, st = run_memory(form, qkv, gates, state, cu, slots, H, G, D, E)
    o, S = plain.delta_memory(q.double(), k.double(), v.double(), beta.double(), log_g.double().exp(), state[0, :H * D * E].view(H, D, E).double())
    close(st[0, :H * D * E].view(H, D, E), S, 3e-6)
    close(out.view(3000, H, E), o, 3e-6)


@pytest.mark.parametrize("form", ["tokens", "chunks"])
def test_the_memory_does_not_depend_on_where_a_sequence_is_cut(form):
    H, G, D, E = 4, 2, 32, 24
    _, qkv, gates, state, _, _ = memory_case([200], H, G, D, E, 50)
    whole, st = run_memory(form, qkv, gates, state, [0, 200], [0], H, G, D, E)
    held, parts, at = state.clone(), [], 0
    for n in (2, 61, 1, 64, 72):
        o, held = run_memory(form, qkv[at:at + n].contiguous(), gates[at:at + n].contiguous(), held.cpu(), [0, n], [0], H, G, D, E)
        parts.append(o)
        at += n
    close(torch.cat(parts), whole.cpu(), 2e-6)
    close(held[0], st[0].cpu(), 2e-6)


def projected(lens, H, G, D, E, K, dt, seed, extra=0):
    """Packed projections [q | k | v | gate | beta | decay] of the given sequences and what the layer holds beside them."""
    n, C = sum(lens) + 3, 2 * G * D + H * E
    x = rnd((n, C + H * E + 2 * H + extra), seed, 1.0, dt)
    w = dict(taps=rnd((C, K), seed + 1), dt_bias=rnd((H,), seed + 2), a_log=rnd((H,), seed + 3), gain=1 + rnd((E,), seed + 4, 0.2))
    state = rnd((len(lens) + 1, H * D * E + (K - 1) * C), seed + 5)
    return x, w, state, cumulative(lens), list(range(len(lens)))[::-1]


def plain_branch(x, w, S, hist, H, G, D, E, eps):
    """One sequence of packed rows from a state: (prepared rows, gates, gated rows, last S, last inputs of the convolution)."""
    C, K = w["taps"].shape
    n = x.shape[0]
    seq = torch.cat([hist, x[:, :C]])
    y = plain.silu(plain.short_conv(seq, w["taps"].double())[K - 1:])
    q, k = plain.unit(y[:, :G * D].view(n, G, D)) * D ** -0.5, plain.unit(y[:, G * D:2 * G * D].view(n, G, D))
    v = y[:, 2 * G * D:].view(n, H, E)
    beta = torch.sigmoid(x[:, C + H * E:C + H * E + H])
    log_g = -torch.exp(w["a_log"].double()) * plain.softplus(x[:, C + H * E + H:C + H * E + 2 * H] + w["dt_bias"].double())
    o, S = plain.delta_memory(q, k, v, beta, log_g.exp(), S)
    rows = plain.rmsnorm(o, w["gain"].double(), eps).reshape(n, -1) * plain.silu(x[:, C:C + H * E])
    prepared = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], dim=1)
    return prepared, torch.cat([beta, log_g, (q * k).sum(-1)], dim=1), rows, S, seq[seq.shape[0] - (K - 1):]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,E,K", [(4, 2, 128, 128, 4), (6, 3, 32, 16, 4), (4, 4, 20, 12, 1), (8, 1, 48, 72, 3), (2, 1, 256, 64, 2), (3, 1, 64, 200, 8), (2, 2, 10, 6, 3)])
def test_what_precedes_the_memory(H, G, D, E, K, dtype):
    """Convolution with its history from and to the state, unit vectors, beta, decays and q . k; sequences shorter than the
    convolution, and a tile of token rows with several of them."""
    from llmgen_b200.kernels import ops
    dt, lens = DT[dtype], [20, 1, 0, 9, 2]
    x, w, state, cu, slots = projected(lens, H, G, D, E, K, dt, 60, extra=3)
    C, n, size = 2 * G * D + H * E, x.shape[0], H * D * E
    qkv, gates, st = torch.full((n, C), 7.0, device=DEV), torch.full((n, 2 * H + G), 7.0, device=DEV), state.to(DEV)
    ops.head_delta_prep(qkv, gates, x.to(DEV), C + H * E, C + H * E + H, w["taps"].to(DEV), w["dt_bias"].to(DEV), w["a_log"].to(DEV),
                        st[:, size:] if K > 1 else None, ints(cu), ints(slots), len(lens), H, G, D, E, 1e-6)
    for i, m in enumerate(lens):
        if m == 0:
            continue
        a, b = cu[i], cu[i + 1]
        hist = state[slots[i], size:].view(K - 1, C).double()
        prepared, g, _, _, last = plain_branch(x[a:b].double(), w, torch.zeros(H, D, E, dtype=torch.float64), hist, H, G, D, E, 1e-5)
        close(qkv[a:b], prepared, 3e-6)
        close(gates[a:b], g, 3e-6)
        if K > 1:
            close(st[slots[i], size:].view(K - 1, C), last, 1e-6)
    assert float((qkv[cu[-1]:] - 7.0).abs().max()) == 0.0 and torch.equal(st[:, :size].cpu(), state[:, :size])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("lens,H,G,D,E,K", [([1] * 5, 8, 4, 128, 128, 4), ([1, 0, 3, 2], 6, 3, 32, 16, 4), ([5, 1], 4, 4, 20, 12, 1), ([16], 8, 1, 48, 72, 3),
                                            ([1, 1], 2, 1, 256, 64, 2), ([7, 2, 1], 3, 1, 64, 200, 8), ([2, 1], 2, 2, 10, 6, 3), ([1], 1, 1, 136, 33, 4)])
def test_a_few_tokens_in_one_launch(lens, H, G, D, E, K, dtype):
    """From the packed projection to the gated rows, written into a wider array, with both parts of the state; heads that share
    a key head read one history."""
    from llmgen_b200.kernels import ops
    assert ops.head_delta_step_usable(H, G, D, E)
    dt = DT[dtype]
    x, w, state, cu, slots = projected(lens, H, G, D, E, K, dt, 80, extra=5)
    C, n, size = 2 * G * D + H * E, x.shape[0], H * D * E
    wide, st = torch.full((n, H * E + 8), 7.0, dtype=dt, device=DEV), state.to(DEV)
    y = wide[:, :H * E]
    for _ in range(2):                          # the second step goes on from the state the first one left
        before = st.clone().cpu()
        ops.head_delta_step(y, x.to(DEV), C + H * E, C + H * E + H, C, w["taps"].to(DEV), w["dt_bias"].to(DEV), w["a_log"].to(DEV), w["gain"].to(DEV), 1e-5,
                            st, ints(cu), ints(slots), len(lens), H, G, D, E, 1e-6)
        for i, m in enumerate(lens):
            if m == 0:
                continue
            a, b = cu[i], cu[i + 1]
            row = before[slots[i]].double()
            _, _, rows, S, last = plain_branch(x[a:b].double(), w, row[:size].view(H, D, E), row[size:].view(K - 1, C), H, G, D, E, 1e-5)
            close(y[a:b], rows, 2e-5 if dtype == "float32" else 1e-2)
            close(st[slots[i], :size].view(H, D, E), S, 3e-6)
            if K > 1:
                close(st[slots[i], size:].view(K - 1, C), last, 1e-6)
    assert float((wide[:, H * E:].float() - 7.0).abs().max()) == 0.0 and torch.equal(st[len(lens)].cpu(), state[len(lens)])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [5, 700])
@pytest.mark.parametrize("E,groups,keep,top,K", [(8, 4, 2, 3, 48), (6, 1, 1, 6, 36), (40, 5, 1, 8, 64), (16, 8, 8, 2, 33), (66, 33, 2, 4, 40)])
def test_the_router_s_groups_correction_and_gate(E, groups, keep, top, K, n, dtype):
    """Corrections far below zero: an output outside the groups kept must count as minus infinity, not as zero."""
    from llmgen_b200.kernels import ops
    h = rnd((n, K), 1, 1.0, DT[dtype])
    router = rnd((E + 1, K), 2, 0.5)
    for shift in (0.0, -3.0):
        corr = rnd((E,), 3, 0.2) + shift
        se, sw, gate = torch.zeros(n * top, dtype=torch.int32, device=DEV), torch.zeros(n * top, device=DEV), torch.zeros(n, device=DEV)
        ops.moe_route(h.to(DEV), router.to(DEV), se, sw, top, "softmax", False, choice_bias=corr.to(DEV), weight_scale=1.7, groups=groups, keep_groups=keep,
                      gate_out=gate)
        z = h.double() @ router.double().T
        close(gate, torch.sigmoid(z[:, E]), 1e-5)
        r = {"groups": {"count": groups, "keep": keep}, "top": top, "scale": 1.7}
        experts, weights = se.view(n, top).cpu().tolist(), sw.view(n, top).cpu().double()
        for t in range(0, n, 1 if n < 50 else 23):
            best, w = plain.choose(z[t, :E], corr.double(), r)
            s = torch.softmax(z[t, :E], 0) + corr.double()
            order = s.sort(descending=True).values
            if float((order[:-1] - order[1:]).min()) < 1e-6:
                continue                        # a close call
            assert experts[t] == best, (t, experts[t], best)
            assert float((weights[t] - torch.tensor(w, dtype=torch.float64)).abs().max()) < 1e-5
    with pytest.raises(ops.KernelError):
        ops.moe_route(h.to(DEV), router.to(DEV), se, sw, E, "softmax", groups=groups, keep_groups=keep, gate_out=gate, choice_bias=corr.to(DEV)) \
            if E > E // groups * keep else ops.moe_route(h.to(DEV), router.to(DEV), se, sw, top, "softmax", groups=groups, keep_groups=groups + 1, gate_out=gate)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H", [48, 37, 1024])
def test_the_sum_over_experts_identities_and_the_gated_shared_expert(H, dtype):
    from llmgen_b200.kernels import ops
    dt, n, top, E = DT[dtype], 9, 3, 4
    h, shared, rows = rnd((n, H + 4), 1, 1.0, dt)[:, :H], rnd((n, H), 2, 1.0, dt), rnd((30, H), 3)
    weights, gate = rnd((n * top,), 4).abs(), rnd((n,), 5).abs()
    experts = torch.randint(0, 7, (n * top,), generator=torch.Generator().manual_seed(6)).to(torch.int32)
    pos = torch.randperm(30, generator=torch.Generator().manual_seed(7))[:n * top].to(torch.int32)
    pos[experts >= E] = -1
    for with_shared in (True, False):
        for weighted in (True, False):
            out = torch.zeros(n, H, device=DEV)
            wide = rnd((n, H + 4), 1, 1.0, dt).to(DEV)
            ops.moe_combine(out, rows.to(DEV), pos.to(DEV), shared.to(DEV) if with_shared else None, top, slot_weight=weights.to(DEV) if weighted else None,
                            shared_gate=gate.to(DEV) if with_shared else None, identity=(wide[:, :H], experts.to(DEV), weights.to(DEV), E))
            want = gate.double()[:, None] * shared.double() if with_shared else torch.zeros(n, H, dtype=torch.float64)
            for s in range(n * top):
                t = s // top
                if int(experts[s]) >= E:
                    want[t] += float(weights[s]) * h[t].double()
                else:
                    want[t] += (float(weights[s]) if weighted else 1.0) * rows[int(pos[s])].double()
            close(out, want, 1e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("S,H", [(1, 64), (2, 1024), (4, 2048), (5, 36), (8, 4096), (4, 4100), (4, 50), (9, 64)])
def test_the_streams_step_for_rows_of_vectors_and_others(S, H, dtype):
    from llmgen_b200.kernels import ops
    dt, n = DT[dtype], 5
    xs = rnd((n, S, H), 1)
    mix, out, read, gain = rnd((S, S), 2, 0.5), rnd((S,), 3), rnd((S,), 4), 1 + rnd((H,), 5, 0.2)
    y1, y2 = rnd((n, H), 6, 1.0, dt), rnd((3, n, H), 7)
    d = lambda t: t.to(DEV)
    forms = [(d(y1), y1.double()), (ops.Partials(d(y2)), y2.double().sum(0)), (ops.WeightedPair(d(y1), 0.6, None, 0.0), 0.6 * y1.double()),
             (ops.WeightedPair(ops.Partials(d(y2)), -0.4, d(y1), 1.1), -0.4 * y2.double().sum(0) + 1.1 * y1.double())]
    for y, y64 in forms:
        streams, normed = d(xs.clone()), torch.zeros(n, H, dtype=dt, device=DEV)
        ops.stream_step(streams, y, d(mix), d(out), d(read), d(gain), 1e-5, normed, dt)
        new = torch.einsum("st,nsh->nth", mix.double(), xs.double()) + out.double()[None, :, None] * y64[:, None, :]
        close(streams, new, 1e-6)
        close(normed, plain.rmsnorm(torch.einsum("t,nth->nh", read.double(), new), gain.double(), 1e-5), 1e-5 if dtype == "float32" else 1e-2)
        streams2 = d(xs.clone())
        ops.stream_step(streams2, y, d(mix), d(out), None, None, 0.0, None, dt)
        assert torch.equal(streams2, streams)
    streams, normed = d(xs.clone()), torch.zeros(n, H, dtype=dt, device=DEV)
    ops.stream_step(streams, None, None, None, d(read), d(gain), 1e-5, normed, dt)
    assert torch.equal(streams.cpu(), xs)
    close(normed, plain.rmsnorm(torch.einsum("t,nth->nh", read.double(), xs.double()), gain.double(), 1e-5), 1e-5 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("heads,H", [(3, 40), (8, 128), (2, 300)])
def test_the_gated_norm_writes_rows_inside_a_wider_array(heads, H):
    from llmgen_b200.kernels import ops
    n = 30
    o, gate, gain = rnd((n * heads, H), 1), rnd((n, heads * H), 2), 1 + rnd((H,), 3, 0.2)
    wide = torch.full((n, heads * H + 16), 7.0, device=DEV)
    ops.gated_rmsnorm(wide[:, 8:8 + heads * H], o.to(DEV), gate.to(DEV), gain.to(DEV), 1e-5, gate_form="silu", heads=heads)
    close(wide[:, 8:8 + heads * H], plain.rmsnorm(o.double().view(n, heads, H), gain.double(), 1e-5).reshape(n, -1) * plain.silu(gate.double()), 1e-5)
    assert float((wide[:, :8] - 7.0).abs().max()) == 0.0 and float((wide[:, 8 + heads * H:] - 7.0).abs().max()) == 0.0
