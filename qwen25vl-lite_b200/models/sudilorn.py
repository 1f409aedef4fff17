"""The Sudilorn decoder as a ``ModelSpec``: a token embedding; pre-norm layers whose sublayers' results are scaled per channel
on their way into the stream (``scaled_residual`` blocks: ``rmsnorm`` with a weight stored around zero before a sublayer, a
learned vector times a constant behind it, ``channel_scale``); a mixer that is either differential attention with a short
convolution, query/key norm, rotation in halves, a sliding window and an output gate (``differential_attention``), or window
attention with biases, interleaved rotation and kept first tokens beside a gated delta rule (``summed_mixers`` of
``sink_attention`` without a sink and ``gated_delta_rule``); routed experts without gates (``grouped_routed_mlp``) or no
feed-forward; a final norm and an untied head.  Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.ls1|ls2``,
``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..config.sudilorn_config import SudilornConfig

ARCHITECTURE = "Sudilorn"


def _rotary(rot, layout: str) -> PartSpec:
    if rot is None:
        return PartSpec("rotary", dict(dims=0, base=1.0, layout=layout))
    return PartSpec("rotary", dict(dims=rot.dims, base=rot.base, layout=layout, scaling=rot.scaling_dict()))


def build_spec(cfg: SudilornConfig) -> ModelSpec:
    w, eps = cfg.hidden_size, cfg.norm_eps
    norm = lambda name, optional=False: PartSpec("rmsnorm", dict(dim=w, eps=eps, name=name, optional=optional, offset=1.0))
    scale = lambda name, gain=1.0, optional=False: PartSpec("channel_scale", dict(dim=w, name=name, gain=cfg.residual_mult * gain, optional=optional))
    layers = []
    for i, layer in enumerate(cfg.layers):
        m, common = layer.mixer, 1.0
        if layer.type == "attention":
            mixer = PartSpec("differential_attention", dict(hidden_size=w, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                                                            scale=m.scale, diff=m.diff, norm_eps=eps, window=m.window, conv=m.conv), "mix.")
            position = _rotary(m.rot, "halves")
        else:
            l, r = m.left, m.right
            # the left branch's constant belongs to the layer's scale, the right branch's is taken relative to it
            common = m.left_scale if m.left_scale != 0.0 else 1.0
            left = PartSpec("sink_attention", dict(hidden_size=w, num_heads=l.heads, num_kv_heads=l.kv_heads, head_dim=l.dim, value_dim=l.vdim,
                                                   scale=l.scale, window=l.window, keep_first=l.keep_first, qkv_bias=True))
            right = PartSpec("gated_delta_rule", dict(hidden_size=w, num_heads=r.heads, num_kv_heads=r.kv_heads, head_dim=r.dim, value_dim=r.vdim,
                                                      conv=r.conv, norm_eps=eps))
            mixer = PartSpec("summed_mixers", dict(hidden_size=w, branches=(("left", left, m.left_scale / common),
                                                                            ("right", right, m.right_scale / common))), "mix.")
            position = _rotary(l.rot, "interleaved")
        ffn, f = None, layer.mlp
        if f is not None:
            ffn = PartSpec("grouped_routed_mlp", dict(hidden_size=w, experts=f.experts, top=f.top, expert_size=f.ff, groups=f.groups, keep=f.keep), "mlp.")
        # a layer without a feed-forward never runs its second norm and scale; a file that holds them all the same is accepted
        norms = (norm("norm1"), scale("ls1", common), norm("norm2", ffn is None), scale("ls2", optional=ffn is None))
        layers.append(LayerSpec(block="scaled_residual", mixer=mixer, feed_forward=ffn, norms=norms, prefix=f"l{i}.", position=position))
    return ModelSpec(
        embedding=PartSpec("token_embedding", dict(vocab_size=cfg.vocab_size, hidden_size=w, name="embed")),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", dict(vocab_size=cfg.vocab_size, hidden_size=w, tied=False, name="head")),
        position=PartSpec("token_index", dict()),
    )


register_architecture(ARCHITECTURE, SudilornConfig.from_dict, build_spec, replace=True)
