"""The Dubodra decoder as a list of parts.

x = embed[token] * embedding.scale.  A layer is pre-norm with layer norms, x += mixer(norm1(x)); x += ff(norm2(x)), and ends
with the token's side input, x += rms(proj (gelu(gate x) * e)) w with e the layer's part of the token's row of a second table
(the ``layernormed`` block; a layer may have no feed-forward, a model no side input).  The mixer is, layer by layer,

  "attention"  grouped-query softmax attention over all earlier positions (``gqa_attention``): q and k heads RMS-normed with a
               weight each before the rotation of their first ``rot.dims`` elements (rotate-half pairs), capped scores, values
               of a size of their own;
  "lightning"  linear attention with one fixed decay per head whose q, k and v pass silu (``retention`` with ``activation``),
               the heads of a token normed together, a sigmoid gate;
  "delta"      the gated delta rule with one decay per head and token and a full silu gate (``gated_delta``).

The feed-forward is a gated gelu unit (``gated_mlp``), or a mixture of clamped gated units (``sum`` of ``routed_experts`` and
``gated_mlp``): softmax scores with a correction for the choice, which is limited to the best groups of experts, identity
experts among the router's outputs, and a shared unit gated by one number per token.  Final layer norm, an untied head, a tanh
cap on the logits.

Tensor names: ``embed``, ``side.embed``; ``l<i>.norm1|norm2`` with ``.b``; attention: ``l<i>.mix.q|k|v|q.norm|k.norm|o``; lightning:
``l<i>.mix.q|k|v|g|norm|o``; delta: ``l<i>.mix.q|q.conv|k|k.conv|v|v.conv|b|a|A_log|dt_bias|norm|g|o``; ``l<i>.mlp.gate|up|down``
or ``l<i>.mlp.router|correction``, ``.e<j>.gate|up|down``, ``.shared.gate|up|down|sg``; ``l<i>.side.gate|proj|norm``; ``final.norm``
with ``.b``; ``head``.
"""
from __future__ import annotations

from ..config.dubodra import DubodraConfig
from ..config.registry import register_architecture
from ..engine.model import ModelSpec, ScheduleEntry
from ..parts import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITIONS
from ..parts.embedding import OutputHead, TokenEmbedding
from ..parts.side import SideTable, TokenSideInput

NO_POSITION_LIMIT = 1 << 20      # the design has no longest sequence; the cache's size is the only limit
UNIT_VECTOR_EPS = 1e-6           # inside the root that makes the delta rule's q and k unit vectors: fixed by the design
GLU_ALPHA = 1.702                # the clamped unit's factor inside the sigmoid: fixed by the design
UNIT_NAMES = {"gate": "gate", "up": "up", "down": "down"}


def build_dubodra(cfg: DubodraConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.eps

    def norm():
        return NORMS.build("layernorm", size=W, eps=eps, param_name="")

    def attention(m):
        position = (POSITIONS.build("rope_neox", head_dim=m.dim, theta=m.rot_base, rotary_dim=m.rot_dims)
                    if m.rot_dims else None)
        return MIXERS.build("gqa_attention", hidden=W, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, v_head_dim=m.vdim,
                            qkv_bias=False, position=position, scale=m.scale, softcap=m.softcap, qk_norm_eps=eps,
                            qk_norm_weight=True, names={"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"})

    def lightning(m):
        return MIXERS.build("retention", hidden=W, n_heads=m.heads, dim=m.dim, vdim=m.vdim, decay=m.decay, eps=eps, k_scale=1.0,
                            activation="silu", joint_norm=True, gate_fn="sigmoid",
                            names={"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm"})

    def delta(m):
        return MIXERS.build("gated_delta", hidden=W, n_heads=m.heads, qk_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, taps=m.taps,
                            decay_rank=None, gate_rank=None, eps=eps, unit_eps=UNIT_VECTOR_EPS, gate_fn="silu",
                            names={"q": "q", "k": "k", "v": "v", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "b": "b",
                                   "a": "a", "a_log": "A_log", "dt_bias": "dt_bias", "norm": "norm", "g": "g", "o": "o"})

    def feed_forward(f):
        if f is None:
            return None
        if f.kind == "dense":
            return FEED_FORWARDS.build("gated_mlp", hidden=W, intermediate=f.ff, activation="gelu_tanh", names=UNIT_NAMES)
        routed = FEED_FORWARDS.build("routed_experts", hidden=W, intermediate=f.expert.ff, n_experts=f.experts, top=f.top,
                                     router_bias=False, activation="clamped_glu", limit=f.expert.limit, glu_alpha=GLU_ALPHA,
                                     grouped=dict(groups=f.groups, keep=f.keep, scale=f.scale), identity=f.identity,
                                     token_gate="shared.sg" if f.shared is not None else None)
        if f.shared is None:
            return routed
        shared = FEED_FORWARDS.build("gated_mlp", hidden=W, intermediate=f.shared.ff, activation="clamped_glu", limit=f.shared.limit,
                                     glu_alpha=GLU_ALPHA, names=UNIT_NAMES)
        return FEED_FORWARDS.build("sum", branches={"": routed, "shared.": shared}, token_gates={"shared.": routed})

    table = SideTable(cfg.vocab, len(cfg.layers), cfg.side_dim, param_name="embed") if cfg.side_dim is not None else None
    mixers = {"attention": attention, "lightning": lightning, "delta": delta}
    blocks, prefixes = [], []
    for i, L in enumerate(cfg.layers):
        ffn = feed_forward(L.mlp)
        side = (TokenSideInput(W, table, i, eps, names={"gate": "gate", "proj": "proj", "norm": "norm"})
                if table is not None else None)
        blocks.append(BLOCKS.build("layernormed", norm1=norm(), mixer=mixers[L.type](L.mixer),
                                   norm2=norm() if ffn is not None else None, ffn=ffn, side=side,
                                   names={"norm1": "norm1", "mixer": "mix.", "norm2": "norm2", "ffn": "mlp.", "side": "side."}))
        prefixes.append(f"l{i}.")
    return ModelSpec(
        config=cfg, embedding=TokenEmbedding(cfg.vocab, W, param_name="", scale=cfg.embedding_scale), embedding_prefix="embed",
        blocks=blocks, block_prefixes=prefixes, final_norm=norm(), final_norm_prefix="final.norm",
        head=OutputHead(cfg.vocab, W, param_name="", softcap=cfg.logit_softcap), head_prefix="head",
        schedule=[ScheduleEntry(layer=i) for i in range(len(cfg.layers))], vocab_size=cfg.vocab, hidden_size=W,
        max_position=NO_POSITION_LIMIT, stop_token_ids=[], shared={"side.": table} if table is not None else {})


register_architecture(DubodraConfig.ARCHITECTURE, DubodraConfig, build_dubodra)
