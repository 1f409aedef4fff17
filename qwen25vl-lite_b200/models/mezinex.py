"""The Mezinex decoder as a ``ModelSpec``: a token embedding to which a hashed table of token pairs is added
(``pair_embedding``); a residual stream of several rows per token whose sublayers read and write it through
hyper-connections (``hyper_residual`` blocks with ``hyper_rmsnorm``; without ``streams`` in the configuration a plain
pre-norm residual); three mixers -- a state space with a step size per head (``mamba2``), latent attention with a query
latent and a gated output (``latent_attention``), a gated linear recurrence (``rglru``) -- and a dense feed-forward
(``swiglu``) or none; a stretch of layers that runs several times in a row, each pass with caches and states of its
own; a final norm over the sum of the rows and a head whose logits are scaled (the constant is folded into the final
norm's weight).  Tensor names: ``embed``, ``bigram``, ``l<i>.norm1|norm2``, ``l<i>.hc1|hc2.in|out|mix``, ``l<i>.mix.*``,
``l<i>.mlp.gate|up|down``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.mezinex_config import MezinexConfig
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Mezinex"
DECAY_GAIN = 8.0            # log a = -8 r softplus(lam) in the gated linear recurrence


def build_spec(cfg: MezinexConfig) -> ModelSpec:
    w, eps = cfg.hidden_size, cfg.norm_eps

    def norm(name, connection=None, optional=False, gain=1.0):
        if cfg.streams is None:
            return PartSpec("rmsnorm", dict(dim=w, eps=eps, name=name, optional=optional, gain=gain))
        return PartSpec("hyper_rmsnorm", dict(dim=w, eps=eps, streams=cfg.streams, name=name, connection=connection, optional=optional, gain=gain))

    layers = []
    for i, layer in enumerate(cfg.layers):
        m, position = layer.mixer, None
        if layer.type == "mamba2":
            mixer = PartSpec("mamba2", dict(hidden_size=w, num_heads=m.heads, value_dim=m.vdim, state_dim=m.state, groups=m.groups, conv=m.conv,
                                            norm_groups=m.norm_groups, norm_eps=eps), "mix.")
        elif layer.type == "latent_attention":
            mixer = PartSpec("latent_attention", dict(hidden_size=w, num_heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim, value_dim=m.vdim,
                                                      kv_rank=m.kv_rank, scale=m.scale, norm_eps=eps, sink=None, q_rank=m.q_rank, out_gate=True), "mix.")
            dims, base = (0, 1.0) if m.rot is None else (m.rot.dims, m.rot.base)
            position = PartSpec("rotary", dict(dims=dims, base=base, layout="interleaved"))
        else:
            mixer = PartSpec("rglru", dict(hidden_size=w, width=m.width, blocks=m.blocks, conv=m.conv, gain=DECAY_GAIN), "mix.")
        ffn = None
        if layer.mlp is not None:
            ffn = PartSpec("swiglu", dict(hidden_size=w, intermediate_size=layer.mlp.ff, names=("gate", "up", "down")), "mlp.")
        # a layer without a feed-forward never runs its second norm and connection; a file that holds them is accepted
        norms = (norm("norm1", "hc1"), norm("norm2", "hc2", optional=ffn is None))
        layers.append(LayerSpec(block="prenorm_residual" if cfg.streams is None else "hyper_residual", mixer=mixer, feed_forward=ffn, norms=norms,
                                prefix=f"l{i}.", position=position))
    pairs = {} if cfg.pairs is None else dict(buckets=cfg.pairs.buckets, mul_prev=cfg.pairs.mul_prev, mul_cur=cfg.pairs.mul_cur)
    return ModelSpec(
        embedding=PartSpec("pair_embedding", dict(vocab_size=cfg.vocab_size, hidden_size=w, streams=cfg.streams, names=("embed", "bigram"), **pairs)),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in cfg.layer_runs()),
        final_norm=norm("final.norm", gain=cfg.logit_scale),
        head=PartSpec("linear_head", dict(vocab_size=cfg.vocab_size, hidden_size=w, tied=False, name="head")),
        position=PartSpec("token_index", dict()),
    )


register_architecture(ARCHITECTURE, MezinexConfig.from_dict, build_spec, replace=True)
