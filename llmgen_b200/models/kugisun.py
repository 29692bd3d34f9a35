"""Kugisun: from its typed configuration to a `ModelSpec`.

A pre-norm decoder over several residual streams per token (`MultiStreamBlockSpec`: hyper-connections; its norms' gains are
stored around zero), with a learned vector per position added to the embedding (`ModelSpec.position_table`), whose table of
embeddings is also its output matrix.  Every layer has one mixer, and some layers run with another layer's weights:

    mixer "parallel"        `ParallelMixerSpec` of two branches on the same input, added with a scale each:
                            left   `AttentionSpec`: grouped-query attention over every earlier key with biases on q, k, v, a norm
                                   per head of q and k, the first `rot.dims` values of a head turned in pairs (2i, 2i + 1), and
                                   values of a width of their own
                            right  `HeadDecayDeltaSpec`: the gated delta rule with one decay per head
    mlp null | dense | moe  none | `GatedMLPSpec` (silu) | `RoutedMLPSpec`: softmax over all outputs of the router, chosen by score
                            plus a correction inside the best groups, weighed by the chosen scores times a constant; the last
                            outputs return the input itself; a shared expert behind a gate per token
    weights_of              the run list names layer j once more with a cache and state number of its own

Tensor names of a model folder (layer i without `weights_of`):

    embed [vocab, width], pos [max_positions, width]; final.norm [width]
    l<i>.norm1, l<i>.norm2 [width]; l<i>.hc1.{in,out} [streams], l<i>.hc1.mix [streams, streams], l<i>.hc2.* the same
    l<i>.mix.left.{q,k,v,o}, .{q,k,v}.b, .{q,k}.norm
    l<i>.mix.right.{q,k,v,b,a,g,o}, .{q,k,v}.conv, .A_log, .dt_bias, .norm
    l<i>.mlp.{gate,up,down} | l<i>.mlp.router, .correction, .e<j>.{gate,up,down}, .shared.{gate,up,down,sg}

Fixed by the architecture, not by its config.json: the 1e-6 beside the squares of a unit vector.
"""
from __future__ import annotations

from ..config.kugisun import DENSE, KugisunConfig, weight_owner
from ..parts.spec import (AttentionSpec, GatedExpertSpec, GatedMLPSpec, HeadDecayDeltaSpec, ModelSpec, MultiStreamBlockSpec,
                          ParallelMixerSpec, RMSNormSpec, RopeSpec, RoutedMLPSpec, RunItem, ShortConvSpec, StreamCoefficients)
from ..registry import register_architecture

UNIT_EPS = 1e-6


def build_kugisun_spec(cfg: KugisunConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name: RMSNormSpec(W, eps, name, weight_offset=1.0)
    layers, place, ignorable = [], {}, []
    for i, layer in enumerate(cfg.layers):
        if weight_owner(cfg.layers, i) != i:
            continue
        p, a, d = f"l{i}.mix.left.", layer.mixer.left, layer.mixer.right
        rope = RopeSpec(rotary_dim=a.rot_dims, theta=a.rot_base, max_positions=cfg.max_positions, pairing="interleaved") if a.rot_dims else None
        left = AttentionSpec(
            hidden_size=W, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, scale=a.scale, q_proj=p + "q", k_proj=p + "k",
            v_proj=p + "v", o_proj=p + "o", q_norm=RMSNormSpec(a.dim, eps, p + "q.norm"), k_norm=RMSNormSpec(a.dim, eps, p + "k.norm"),
            position=rope, v_head_dim=a.vdim, q_bias=p + "q.b", k_bias=p + "k.b", v_bias=p + "v.b")
        p = f"l{i}.mix.right."
        right = HeadDecayDeltaSpec(
            hidden_size=W, num_heads=d.heads, num_kv_heads=d.kv_heads, key_dim=d.dim, value_dim=d.vdim,
            conv=ShortConvSpec(2 * d.kv_heads * d.dim + d.heads * d.vdim, d.conv, p + "qkv.conv"),
            conv_weights=(p + "q.conv", p + "k.conv", p + "v.conv"), q_proj=p + "q", k_proj=p + "k", v_proj=p + "v", beta_proj=p + "b",
            decay_proj=p + "a", decay_bias=p + "dt_bias", decay_log=p + "A_log", gate_proj=p + "g", o_proj=p + "o",
            out_norm=RMSNormSpec(d.vdim, eps, p + "norm"), unit_eps=UNIT_EPS)
        ffn = None
        if layer.mlp is None:
            # a layer without a feed-forward has no use for its second norm and coefficients; a folder may carry them
            ignorable += [f"l{i}.norm2", f"l{i}.hc2.*"]
        else:
            q, f = f"l{i}.mlp.", layer.mlp
            expert = lambda name, ff: GatedExpertSpec(ff, f"{q}{name}.gate", f"{q}{name}.up", f"{q}{name}.down")
            if f.kind == DENSE:
                ffn = GatedMLPSpec(W, f.ff, q + "gate", q + "up", q + "down")
            else:
                ffn = RoutedMLPSpec(
                    hidden_size=W, router=q + "router", top_k=f.top, scoring="softmax", renormalize=False, weight_on_input=False,
                    experts=tuple(expert(f"e{j}", f.ff) for j in range(f.experts)), choice_bias=q + "correction", weight_scale=f.scale,
                    shared=expert("shared", f.shared_ff) if f.shared_ff else None, shared_gate=q + "shared.sg" if f.shared_ff else None,
                    identity_outputs=f.identity, groups=f.groups, keep_groups=f.keep)
        coefficients = (lambda n: StreamCoefficients(f"l{i}.hc{n}.in", f"l{i}.hc{n}.out", f"l{i}.hc{n}.mix")) if cfg.streams else (lambda n: None)
        place[i] = len(layers)
        layers.append(MultiStreamBlockSpec(
            mixer_norm=norm(f"l{i}.norm1"),
            mixer=ParallelMixerSpec(branches=(left, right), scales=(layer.mixer.left_scale, layer.mixer.right_scale)),
            ffn_norm=norm(f"l{i}.norm2") if ffn is not None else None, ffn=ffn, streams=cfg.streams or 1,
            mixer_streams=coefficients(1), ffn_streams=coefficients(2) if ffn is not None else None))
    order = tuple(RunItem(layer=place[weight_owner(cfg.layers, i)], cache=i) for i in range(len(cfg.layers)))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=W, embedding="embed", layers=tuple(layers), run_order=order,
        final_norm=norm("final.norm"), lm_head="embed", max_positions=cfg.max_positions, residual_streams=cfg.streams or 1,
        position_table="pos", ignorable_tensors=tuple(ignorable))


register_architecture("Kugisun", KugisunConfig, build_kugisun_spec, aliases=("kugisun",))
