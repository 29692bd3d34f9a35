"""Zuvasun: from its typed configuration to a `ModelSpec`.

A decoder whose layers run their mixer and their feed-forward side by side off one norm (`ParallelBlockSpec`, with a
gain vector on each result as it joins the stream), and pick one of two mixers:

    mixer "attention"         `AttentionSpec`: grouped-query attention over every earlier key, without positions; q and k with
                              biases and normed over their whole projections, queries scaled by a temperature that grows
                              with the position, and values that are the projected keys (one cached entry a token)
    mixer "latent_attention"  `LatentAttentionSpec`: attention over cached latents with queries projected straight from
                              the stream, a sliding window, and rotary frequencies scaled by YaRN; a layer with `kv_from`
                              keeps nothing and reads the entries another layer cached (a run item with
                              `writes_cache=False` on that layer's cache number)
    mlp null | moe            none | `RoutedMLPSpec`: softmax over all experts, chosen by score plus a correction per
                              expert, weighed by the chosen scores over their sum times a constant; experts without a
                              gate, relu squared

Tensor names of a model folder (layer i):

    embed, head [vocab, width]; final.norm [width]
    l<i>.norm1, l<i>.ls1, l<i>.ls2 [width]
    l<i>.mix.{q,k,o}, .{q,k}.b, .{q,k}.norm                      attention
    l<i>.mix.{q,uk,uv,o}, and .dkv, .dkv.norm without `kv_from`  latent_attention
    l<i>.mlp.router, .correction, .e<j>.{up,down}

Fixed by the architecture, not by its config.json: pairs (2i, 2i + 1) of the rotated part, the 1e-20 beside the sum of
the chosen scores.
"""
from __future__ import annotations

from ..config.zuvasun import ATTENTION, ZuvasunConfig
from ..parts.spec import (AttentionSpec, LatentAttentionSpec, ModelSpec, ParallelBlockSpec, PlainExpertSpec, RMSNormSpec, RopeSpec,
                          RoutedMLPSpec, RunItem)
from ..registry import register_architecture

ROUTER_SUM_EPS = 1e-20


def build_zuvasun_spec(cfg: ZuvasunConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    layers, order, ignorable = [], [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.mix.", layer.mixer
        cache, writes = i, True
        if layer.type == ATTENTION:
            mixer = AttentionSpec(
                hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, scale=m.scale,
                q_proj=p + "q", k_proj=p + "k", v_proj="", o_proj=p + "o", q_bias=p + "q.b", k_bias=p + "k.b",
                q_norm=RMSNormSpec(m.heads * m.dim, eps, p + "q.norm"), k_norm=RMSNormSpec(m.kv_heads * m.dim, eps, p + "k.norm"),
                row_norms=True, values_from_keys=True, query_temperature=m.q_temp)
        else:
            rope = RopeSpec(rotary_dim=m.rot_dim, theta=m.rot.base, max_positions=cfg.max_positions, pairing="interleaved",
                            yarn=m.rot.scaling)
            own = m.kv_from is None
            if not own:
                cache, writes = m.kv_from, False
            mixer = LatentAttentionSpec(
                hidden_size=W, num_heads=m.heads, nope_dim=m.dim, rope_dim=m.rot_dim, value_dim=m.vdim, q_rank=0, kv_rank=m.kv_rank,
                scale=m.scale, dq_proj=None, uq_proj=None, dkv_proj=p + "dkv" if own else None, uk_proj=p + "uk", uv_proj=p + "uv",
                o_proj=p + "o", q_norm=None, kv_norm=RMSNormSpec(m.kv_rank, eps, p + "dkv.norm") if own else None, position=rope,
                q_proj=p + "q", window=m.window or None, absorb_at_load=False)
        ffn = None
        if layer.mlp is not None:
            q, f = f"l{i}.mlp.", layer.mlp
            ffn = RoutedMLPSpec(
                hidden_size=W, router=q + "router", top_k=f.top, scoring="softmax", renormalize=True, weight_on_input=False,
                experts=tuple(PlainExpertSpec(f.ff, f"{q}e{j}.up", f"{q}e{j}.down") for j in range(f.experts)),
                choice_bias=q + "correction", weight_scale=f.scale, sum_eps=ROUTER_SUM_EPS)
        else:
            ignorable.append(f"l{i}.ls2")        # no use for a gain of its feed-forward; a folder may carry it
        layers.append(ParallelBlockSpec(mixer_norm=RMSNormSpec(W, eps, f"l{i}.norm1"), mixer=mixer, ffn=ffn, mixer_gain=f"l{i}.ls1",
                                        ffn_gain=f"l{i}.ls2" if ffn is not None else None))
        order.append(RunItem(layer=i, cache=cache, writes_cache=writes))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=W, embedding="embed", layers=tuple(layers),
        run_order=tuple(order), final_norm=RMSNormSpec(W, eps, "final.norm"), lm_head="head", max_positions=cfg.max_positions,
        ignorable_tensors=tuple(ignorable))


register_architecture("Zuvasun", ZuvasunConfig, build_zuvasun_spec, aliases=("zuvasun",))
