"""Small Kugisun configurations with random weights, for the tests: the engine's model and the tensors the plain
implementation reads, made from one seed."""
from __future__ import annotations

import copy
from typing import Dict, List, Sequence

import torch

from tests.derupel_util import TOL, driver, ids_for, relative_error, row_errors, run_in_portions  # noqa: F401
from tests.nasozen_util import assert_close, draw  # noqa: F401


def left(heads, kv_heads, dim, vdim, scale, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return m


def right(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def layer(left_m, right_m, mlp, scales=(0.7, 1.2)):
    return {"type": "parallel", "mixer": {"left": left_m, "right": right_m, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale=1.0, identity=0, groups=None, shared=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if identity:
        router["identity"] = identity
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def config(layers, width=48, vocab=97, eps=1e-5, streams=3, max_positions=512, shares=()) -> dict:
    """`shares`: (i, j) pairs: layer j's entry is put in at place i, with `weights_of` j."""
    layers = copy.deepcopy(list(layers))
    for i, j in shares:
        layers.insert(i, dict(copy.deepcopy(layers[j]), weights_of=j))
    cfg = {"architecture": "Kugisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "max_positions": max_positions, "layers": layers}
    if streams is not None:
        cfg["streams"] = streams
    return cfg


# Every kind of feed-forward, sizes that differ from one another wherever they can: key width != value width in both
# branches, grouped heads, half a head rotated, groups of outputs of which the last are identities, three streams, a layer that
# uses the routed layer's weights right behind it and one that uses the first layer's at the end.
MIXED = config([
    layer(left(4, 2, 16, 24, 0.3, rot=(300.0, 8)), right(4, 2, 8, 16, 3), dense(40)),
    layer(left(6, 2, 8, 16, 0.4, rot=(5000.0, 8)), right(2, 1, 16, 24, 4), moe(6, 3, 24, 1.7, identity=2, groups=(4, 2), shared=40), scales=(1.1, 0.6)),
    layer(left(2, 1, 24, 8, 0.25, rot=(77.0, 4)), right(3, 3, 12, 8, 2), None),
], shares=((2, 1), (4, 0)))
# Sizes that are multiples of little, and values that a usual model makes equal or one: one stream (with coefficients of its
# own), one head, as many key heads as heads, one expert chosen, a convolution of one tap, no rotation, both scales 1, no groups, no
# identities, no shared expert, a chain of layers that use another's weights.
ODD = config([
    layer(left(3, 3, 10, 6, 0.4), right(3, 1, 10, 7, 1), moe(3, 1, 20), scales=(1.0, 1.0)),
    layer(left(1, 1, 12, 20, 0.2, rot=(77.0, 12)), right(1, 1, 6, 9, 2), moe(2, 4, 30, 0.5, identity=3, groups=(1, 1), shared=18)),
    dict(layer(left(1, 1, 12, 20, 0.2, rot=(77.0, 12)), right(1, 1, 6, 9, 2), moe(2, 4, 30, 0.5, identity=3, groups=(1, 1), shared=18)), weights_of=1),
    dict(layer(left(1, 1, 12, 20, 0.2, rot=(77.0, 12)), right(1, 1, 6, 9, 2), moe(2, 4, 30, 0.5, identity=3, groups=(1, 1), shared=18)), weights_of=2),
], width=36, vocab=50, eps=1e-4, streams=1, max_positions=128)
# No streams at all (a plain pre-norm layer), eight heads on one key head, eight taps, more identities than experts.
PLAIN = config([
    layer(left(8, 1, 8, 8, 0.35, rot=(50.0, 8)), right(8, 1, 8, 8, 8), moe(2, 2, 16, 2.5, identity=6, groups=(4, 1), shared=24), scales=(1.3, 0.4)),
    layer(left(2, 2, 12, 10, 0.3, rot=(1000.0, 4)), right(2, 2, 20, 12, 2), None),
    layer(left(2, 1, 8, 16, 0.3), right(4, 4, 4, 8, 4), dense(24)),
], width=24, vocab=61, streams=None, max_positions=128)
# Key widths beyond 64 and 128 in the memory (the kernels' wider forms, and the one that only the walk token by token takes),
# value widths that are no multiples of 8 or 16, five streams.
WIDE = config([
    layer(left(8, 4, 32, 40, 0.18, rot=(100.0, 32)), right(2, 1, 72, 40, 4), dense(32)),
    layer(left(4, 1, 16, 16, 0.3, rot=(100.0, 2)), right(2, 2, 136, 24, 3), moe(4, 2, 48, 1.2, shared=16)),
], width=48, vocab=61, eps=1e-6, streams=5, max_positions=128)
# Key and value widths that the tensor-core attention of the bfloat16 engine takes, and prompts long enough for the memory's
# chunks: several tiles of keys and queries, chunks that end inside a portion.
TENSOR = config([
    layer(left(4, 2, 64, 64, 0.11, rot=(10000.0, 32)), right(4, 2, 16, 32, 4), moe(4, 2, 64, 1.5, identity=4, groups=(2, 1), shared=32)),
    layer(left(2, 1, 128, 64, 0.09, rot=(500.0, 128)), right(2, 1, 64, 48, 2), None),
], width=64, vocab=97, streams=2, max_positions=1024)
# One layer whose weights `plant_needle` rewrites so that one token's query finds one other token's key.
NEEDLE = config([layer(left(2, 1, 64, 16, 0.25, rot=(30.0, 8)), right(1, 1, 8, 8, 2), dense(16), scales=(1.0, 0.1))],
                width=32, vocab=53, streams=2, max_positions=2048)
NEEDLE_ID, PROBE_ID, FILLER_ID = 5, 9, 11
# A memory that keeps (nearly) everything and nothing else to carry information over more than one token: losing a state, or a
# token of it, shows at every later position.
KEEPING = config([layer(left(1, 1, 8, 8, 0.3), right(2, 1, 16, 8, 3), None, scales=(0.0, 1.0))], width=32, vocab=53, streams=2, max_positions=1024)


def build(cfg: dict, seed: int, dtype: str = "float32", sigma: float = 0.1, sigma_norm: float = 0.2, prepare=None):
    """(the engine's model on the GPU, tensors by name on the CPU).  Router and correction are drawn wider than the other
    matrices, so that chosen scores, groups and corrections lie apart; for the bfloat16 engine the corrections lie far apart: there
    a close call says nothing about a kernel."""
    from llmgen_b200.engine.api import require_cuda, resolve_dtype
    from llmgen_b200.engine.model import DecoderModel
    from llmgen_b200.weights import weights_from_dict
    spec, decls, tensors = draw(cfg, seed, sigma, sigma_norm)
    for name, t in tensors.items():
        if name.endswith(".router"):
            t.mul_(4.0)
        elif name.endswith(".correction"):
            t.mul_(2.0 if dtype == "float32" else 12.0)
    if prepare is not None:
        prepare(cfg, tensors)
    model = DecoderModel(spec, weights_from_dict(tensors, decls), resolve_dtype(dtype), require_cuda())
    return model, tensors


def keep_long(cfg: dict, tensors: Dict[str, torch.Tensor]) -> None:
    """Makes the one-layer KEEPING model remember: decays near one, and writes small enough for hundreds of tokens (the first
    value of every normed row is positive and far from zero, and beta's projection reads it with a minus)."""
    tensors["l0.mix.right.A_log"].fill_(-9.0)
    tensors["embed"][:, 0] = 1.0
    tensors["pos"].mul_(0.1)
    tensors["l0.norm1"].zero_()
    b = tensors["l0.mix.right.b"]
    b.mul_(0.1)
    b[:, 0] = -1.2


def plant_needle(cfg: dict, tensors: Dict[str, torch.Tensor]) -> None:
    """Rewrites the tensors of the one-layer NEEDLE model in place so that the query of token PROBE_ID points where the key
    of token NEEDLE_ID points: queries read the first half of the normed row, keys the second half, through the same matrix
    rows; the probe's first half is the needle's second half; biases are zero and gains one, positions and rotated rows
    small.  The score of that pair is then about scale * dim = 16 against a few for random directions: the probe's output is
    nearly the needle's value wherever the needle lies, and a key or value that is not the one written for it shows far
    beyond rounding."""
    m = cfg["layers"][0]["mixer"]["left"]
    heads, kv, dim, width = m["heads"], m["kv_heads"], m["dim"], cfg["width"]
    half = width // 2
    p = "l0.mix.left."
    wq, wk = tensors[p + "q"], tensors[p + "k"]
    wk[:, :half] = 0
    for g in range(kv):
        wk[g * dim:g * dim + m["rot"]["dims"]] *= 0.1
    for h in range(heads):
        g = h // (heads // kv)
        wq[h * dim:(h + 1) * dim, :half] = wk[g * dim:(g + 1) * dim, half:]
    wq[:, half:] = 0
    for n in ("q.b", "k.b"):
        tensors[p + n].zero_()
    for n in ("q.norm", "k.norm"):
        tensors[p + n].fill_(1.0)
    tensors["l0.norm1"].zero_()
    tensors["pos"].mul_(0.02)
    emb = tensors["embed"]
    emb[PROBE_ID, :half] = emb[NEEDLE_ID, half:]


def needle_ids(cfg: dict, n: int, needle_at: int, seed: int) -> List[int]:
    """`n` random ids with the needle token at `needle_at` only and the probe token last only."""
    ids = [t if t not in (NEEDLE_ID, PROBE_ID) else FILLER_ID for t in ids_for(cfg, n, seed)]
    ids[needle_at] = NEEDLE_ID
    ids[-1] = PROBE_ID
    return ids


def plain_logits(cfg: dict, tensors: Dict[str, torch.Tensor], ids: Sequence[int]) -> torch.Tensor:
    from tests.plain import kugisun_plain
    return kugisun_plain.forward(cfg, tensors, ids)
