"""The Gedilorn decoder as a list of parts.

x = embed[token] * embedding.scale plus a row of a second table chosen by the previous and the current token, then an RMS
norm (``PairEmbedding``).  The residual is ``streams`` copies of x (``hyper_connected`` blocks): a sub-layer reads a weighted
sum of them through its norm, and its result and a matrix over the streams make the new ones; without ``streams`` the block is
the ordinary ``prenorm``.  The mixer is attention over a cached latent with one rotated key part for all heads
(``latent_cache_attention``), of type "latent_attention_2" with an element-wise sigmoid gate on the concatenated heads;
neighbouring pairs turn, with YaRN-stretched frequencies.  The feed-forward is a gated unit with relu (``gated_mlp``).  The sum
of the streams goes through the final norm and the head, and the logits are multiplied by a number.

A layer with ``weights_of`` is one more execution of that layer's block in the schedule, with a cache of its own.

Tensor names: ``embed``, ``bigram``, ``embed.norm``; ``l<i>.norm1|norm2``; ``l<i>.mix.q|dkv|dkv.norm|uk|uv|g|o``;
``l<i>.mlp.gate|up|down``; ``l<i>.hc1|hc2.in|out|mix``; ``final.norm``; ``head``.
"""
from __future__ import annotations

from ..config.gedilorn import GedilornConfig
from ..config.registry import register_architecture
from ..engine.model import ModelSpec, ScheduleEntry
from ..parts import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITIONS
from ..parts.embedding import OutputHead, PairEmbedding
from ..parts.streams import StreamsNorm

NO_POSITION_LIMIT = 1 << 20      # the design has no longest sequence; the cache's size is the only limit


def build_gedilorn(cfg: GedilornConfig) -> ModelSpec:
    W, eps, S = cfg.width, cfg.eps, cfg.streams

    def norm():
        return NORMS.build("rmsnorm", size=W, eps=eps, param_name="")

    def mixer(m):
        position = None
        if m.rot_dim and m.rot_scaling is not None:
            position = POSITIONS.build("rope_yarn", head_dim=m.rot_dim, theta=m.rot_base, interleaved=True, **m.rot_scaling)
        elif m.rot_dim:
            position = POSITIONS.build("rope_neox", head_dim=m.rot_dim, theta=m.rot_base, interleaved=True)
        return MIXERS.build("latent_cache_attention", hidden=W, n_heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim,
                            v_head_dim=m.vdim, kv_rank=m.kv_rank, eps=eps, scale=m.scale, position=position,
                            gate="sigmoid" if m.gated else None,
                            names={"q": "q", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "g": "g", "o": "o"})

    names = {"norm1": "norm1", "mixer": "mix.", "norm2": "norm2", "ffn": "mlp."}
    blocks, prefixes, index_of = [], [], {}
    for i, L in enumerate(cfg.layers):
        if L.weights_of is not None:
            continue
        ffn = (FEED_FORWARDS.build("gated_mlp", hidden=W, intermediate=L.ff, activation="relu",
                                   names={"gate": "gate", "up": "up", "down": "down"}) if L.ff is not None else None)
        parts = dict(norm1=norm(), mixer=mixer(L.mixer), norm2=norm() if ffn is not None else None, ffn=ffn)
        if S is None:
            block = BLOCKS.build("prenorm", names=names, **parts)
        else:
            block = BLOCKS.build("hyper_connected", streams=S, names=dict(names, conn1="hc1.", conn2="hc2."), **parts)
        index_of[i] = len(blocks)
        blocks.append(block)
        prefixes.append(f"l{i}.")
    schedule = [ScheduleEntry(layer=index_of[i if L.weights_of is None else L.weights_of]) for i, L in enumerate(cfg.layers)]
    pairs = cfg.pairs
    embedding = PairEmbedding(cfg.vocab, W, scale=cfg.embedding_scale, eps=eps,
                              buckets=pairs.buckets if pairs else None, mul_prev=pairs.mul_prev if pairs else 0,
                              mul_cur=pairs.mul_cur if pairs else 0,
                              names={"table": "embed", "pairs": "bigram", "norm": "embed.norm"})
    return ModelSpec(
        config=cfg, embedding=embedding, embedding_prefix="", blocks=blocks, block_prefixes=prefixes,
        final_norm=norm() if S is None else StreamsNorm(norm(), S), final_norm_prefix="final.norm",
        head=OutputHead(cfg.vocab, W, param_name="", scale=cfg.logit_scale), head_prefix="head",
        schedule=schedule, vocab_size=cfg.vocab, hidden_size=W, max_position=NO_POSITION_LIMIT, stop_token_ids=[], streams=S)


register_architecture(GedilornConfig.ARCHITECTURE, GedilornConfig, build_gedilorn)
