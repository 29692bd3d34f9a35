"""Small Zuvasun configurations with random weights, for the tests: the engine's model and the tensors the plain
implementation reads, made from one seed."""
from __future__ import annotations

import copy
from typing import Dict, List, Sequence

import torch

from tests.derupel_util import TOL, driver, ids_for, relative_error, row_errors, run_in_portions  # noqa: F401
from tests.nasozen_util import assert_close  # noqa: F401


def attention(heads, kv_heads, dim, scale, mlp, q_temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if q_temp is not None:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, mlp, window=None, yarn=None, kv_from=None):
    rot = {"base": base, "dims": rot_dim}
    if yarn is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": rot}
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def moe(experts, top, ff, scale):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}}


def config(layers, width=48, vocab=97, eps=1e-5) -> dict:
    return {"architecture": "Zuvasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": copy.deepcopy(list(layers))}


# Every kind of layer, sizes that differ from one another wherever they can: key width != value width in the latent layers,
# grouped heads and as many key heads as heads, a layer that reads another's entries through a wider window (the pages must
# outlive the owner's window) and with heads of other widths, frequencies inside the blended stretch, temperatures that step
# every 10 positions and none, windows that are no multiple of a page (16), a layer without a feed-forward, every expert chosen.
YARN = (4.0, 64, 8.0, 1.0)
MIXED = config([
    latent(3, 16, 8, 24, 32, 0.3, 100.0, moe(6, 2, 24, 1.7), window=24, yarn=YARN),
    attention(4, 2, 16, 0.4, moe(5, 3, 16, 0.8), q_temp=(0.25, 10)),
    latent(2, 12, 8, 10, 32, 0.4, 100.0, None, window=41, yarn=YARN, kv_from=0),
    attention(6, 6, 8, 0.5, moe(3, 3, 20, 2.2)),
])
# Sizes that are multiples of little (odd widths too), values that a usual model makes equal or one: no window at all, a
# reader whose window is narrower than the owner's (which has none), one head, one expert of one, a scale and a temperature of one.
ODD = config([
    attention(3, 1, 9, 0.3, moe(4, 1, 12, 1.0), q_temp=(1.0, 1)),
    latent(1, 7, 6, 5, 18, 0.45, 77.0, moe(1, 1, 30, 0.6)),
    latent(5, 6, 6, 11, 18, 1.0, 77.0, moe(7, 2, 10, 1.3), window=5, kv_from=1),
    attention(1, 1, 14, 0.35, None, q_temp=(-0.2, 7.5)),
], width=36, vocab=50, eps=1e-4)
# More query heads than one block of the latent attention takes rows (32), of which the last chunk is partial; a window of one
# position and of two; more heads on a key head than one block of the general attention takes (16); a long rotated part.
WIDE = config([
    latent(37, 8, 4, 8, 16, 0.3, 50.0, moe(3, 2, 16, 1.1), window=2),
    latent(2, 10, 4, 6, 16, 0.5, 50.0, None, window=1, kv_from=0),
    attention(20, 1, 24, 0.2, moe(9, 4, 8, 3.0), q_temp=(0.4, 16)),
    latent(2, 8, 48, 16, 40, 0.2, 1000.0, None, window=33, yarn=(2.5, 300, 20.0, 2.0)),
], width=40, vocab=61, eps=1e-6)
# Widths that the tensor-core kernels of the bfloat16 engine take (latents of 64 and 128 and key widths of 64 and 128, unrotated
# widths that are multiples of 8, experts' rows likewise), with windows that are no multiple of their tiles.
TENSOR = config([
    attention(6, 3, 64, 0.14, moe(4, 2, 64, 1.4), q_temp=(0.3, 50)),
    latent(5, 24, 16, 40, 64, 0.17, 10000.0, moe(5, 2, 40, 0.9), window=90, yarn=(3.0, 500, 16.0, 1.0)),
    latent(34, 16, 16, 8, 64, 0.2, 10000.0, None, window=130, yarn=(3.0, 500, 16.0, 1.0), kv_from=1),
    attention(2, 1, 128, 0.1, None),
    latent(2, 32, 32, 64, 128, 0.15, 300.0, moe(3, 1, 24, 2.0)),
], width=64, vocab=97)
# One layer (or two) whose weights `plant_*` rewrite so that one token's query finds one other token's key.
NEEDLE_WINDOW = 40
NEEDLE_ID, PROBE_ID, FILLER_ID = 5, 9, 11
FAR = config([attention(4, 2, 64, 0.25, moe(3, 1, 32, 0.3), q_temp=(0.05, 64))], width=32, vocab=53)
NEAR = config([latent(2, 64, 8, 24, 64, 0.25, 30.0, moe(3, 1, 32, 0.3), window=NEEDLE_WINDOW)], width=32, vocab=53)
# the second layer reads the first one's entries through a wider window; the first adds nothing to the stream
BORROWED = config([
    latent(2, 16, 8, 24, 64, 0.25, 30.0, None, window=7),
    latent(2, 64, 8, 24, 64, 0.25, 30.0, moe(3, 1, 32, 0.3), window=NEEDLE_WINDOW, kv_from=0),
], width=32, vocab=53)


def draw(cfg: dict, seed: int, sigma: float = 0.1, sigma_norm: float = 0.2):
    from llmgen_b200.parts.registry import model_weight_decls
    from llmgen_b200.registry import config_from_dict
    from llmgen_b200.weights import random_tensors
    arch, typed = config_from_dict(cfg)
    spec = arch.build_spec(typed)
    decls = model_weight_decls(spec)
    return spec, decls, random_tensors(decls, seed, sigma, sigma_norm, torch.bfloat16)     # stored as a model folder stores them


def build(cfg: dict, seed: int, dtype: str = "float32", sigma: float = 0.1, sigma_norm: float = 0.2, prepare=None):
    """(the engine's model on the GPU, tensors by name on the CPU)."""
    from llmgen_b200.engine.api import require_cuda, resolve_dtype
    from llmgen_b200.engine.model import DecoderModel
    from llmgen_b200.weights import weights_from_dict
    spec, decls, tensors = draw(cfg, seed, sigma, sigma_norm)
    if prepare is not None:
        prepare(cfg, tensors)
    model = DecoderModel(spec, weights_from_dict(tensors, decls), resolve_dtype(dtype), require_cuda())
    return model, tensors


def plant_far(cfg: dict, tensors: Dict[str, torch.Tensor]) -> None:
    """FAR: queries read the first half of the normed row, keys the second half, through the same matrix rows; the probe's first
    half is the needle's second half; no biases, gains of one.  Both projections have a root mean square of one, so the score of
    that pair is about scale * dim = 16 and all others are those of random directions: the probe's output is nearly the needle's
    value, which is its key as projected."""
    m = cfg["layers"][0]["mixer"]
    heads, kv, dim, half = m["heads"], m["kv_heads"], m["dim"], cfg["width"] // 2
    wq, wk = tensors["l0.mix.q"], tensors["l0.mix.k"]
    wk[:, :half] = 0
    for h in range(heads):
        g = h // (heads // kv)
        wq[h * dim:(h + 1) * dim, :half] = wk[g * dim:(g + 1) * dim, half:]
    wq[:, half:] = 0
    for n in ("l0.mix.q.b", "l0.mix.k.b"):
        tensors[n].zero_()
    for n in ("l0.norm1", "l0.mix.q.norm", "l0.mix.k.norm"):
        tensors[n].fill_(1.0)
    emb = tensors["embed"]
    emb[PROBE_ID, :half] = emb[NEEDLE_ID, half:]


def plant_latent(cfg: dict, tensors: Dict[str, torch.Tensor]) -> None:
    """NEAR and BORROWED: the latent reads the second half of the normed row; a head's unrotated query is its key matrix on the
    latent that the first half would give, and the probe's first half is the needle's second half, so its query points where the
    needle's key points, with a length that makes the score of that pair 25; the rotated parts decide nothing."""
    last = len(cfg["layers"]) - 1
    m, half = cfg["layers"][last]["mixer"], cfg["width"] // 2
    heads, dim, rot, rank = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    dkv, wq, uk = tensors["l0.mix.dkv"], tensors[f"l{last}.mix.q"], tensors[f"l{last}.mix.uk"]
    dkv[:rank, :half] = 0
    for i in range(last + 1):
        tensors[f"l{i}.norm1"].fill_(1.0)
    if last:
        tensors["l0.ls1"].zero_()                     # the stream the second layer reads is the embedding's
    emb = tensors["embed"]
    emb[PROBE_ID, :half] = emb[NEEDLE_ID, half:]
    norm = lambda x: x.double() / (x.double().pow(2).mean() + cfg["norm"]["eps"]).sqrt()
    gain = tensors["l0.mix.dkv.norm"].double()
    raw = dkv[:rank, half:].double()
    c = norm(raw @ norm(emb[NEEDLE_ID])[half:]) * gain                       # the needle's latent
    for h in range(heads):
        u = uk[h * dim:(h + 1) * dim].double()
        to_query = u @ (gain[:, None] * raw)                                  # [dim, half]
        score = float((to_query @ norm(emb[PROBE_ID])[:half]) @ (u @ c)) * m["scale"]
        rows = wq[h * (dim + rot):(h + 1) * (dim + rot)]
        rows.zero_()
        rows[:dim, :half] = (to_query * (25.0 / score)).to(wq.dtype)


def needle_ids(cfg: dict, n: int, needle_at: int, seed: int) -> List[int]:
    """`n` random ids with the needle token at `needle_at` only and the probe token last only."""
    ids = [t if t not in (NEEDLE_ID, PROBE_ID) else FILLER_ID for t in ids_for(cfg, n, seed)]
    ids[needle_at] = NEEDLE_ID
    ids[-1] = PROBE_ID
    return ids


def plain_logits(cfg: dict, tensors: Dict[str, torch.Tensor], ids: Sequence[int]) -> torch.Tensor:
    from tests.plain import zuvasun_plain
    return zuvasun_plain.forward(cfg, tensors, ids)
