"""Layered models: the trunk is a list of layer specs (``YvConfig.layer_specs``), each naming a mixer and a
feed-forward from the tables below, around an fp32 residual stream.  ``YvConfig.layer_block`` says how a layer joins its
branches to the stream; n(x) = rms(x) * (offset + w):

    sandwich    x += n1b(mixer(n1(x)))
                x += n2b(ff(n2(x)))                                       (layers with a feed-forward)
                x += ns(P (gelu_tanh(G x) * e_layer[token]))              (models with a per-layer token input)
    parallel    x += mixer(n1(x)) + ff(n2(x))                             (both of the same x)

The stream starts as n(embed[token]) or scale * embed[token].  ``YvConfig.layer_loop`` runs some layers several times;
before every pass but the first the start of the stream is added to it again, and before every pass a learned vector.
The model ends with logits = head nf(x).

Every ``x +=`` and the norms in front of the next branch are one kernel: the stream is read and written once per join.
A parallel block forms both branches' sum in one product, [heads | activations] against [W_o | W_down], that adds to the
stream itself.  The classes keep the contracts that generation, the engine, the captured decode step and the loader
rely on, so a layered model is served by the same code as the Yv trunk.  They are serving models: no backward."""
from __future__ import annotations

from typing import Any, Callable, Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..config import YvConfig
from ..ops import latent as L
from .attention import AttnContext
from .grouped_attention import YvGroupedAttention
from .latent_attention import YvWindowedLatentAttention, rotary_for
from .model import YvModelForCausalLM, YvModelOutput, YvPackedTrunk


class YvDenseGELU(nn.Module):
    """Two products around the exact GELU."""

    def __init__(self, hidden: int, spec: Dict[str, Any], init_std: float = 0.02):
        super().__init__()
        mk = lambda *s: nn.Parameter(torch.empty(*s).normal_(std=init_std), requires_grad=False)
        self.up, self.down = mk(spec["ff"], hidden), mk(hidden, spec["ff"])

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return L.project(L.gelu(L.project(h, self.up)), self.down)

    def checkpoint_slices(self) -> Dict[str, torch.Tensor]:
        return {"up": self.up, "down": self.down}


class YvDenseSwiGLU(nn.Module):
    """``W_down (silu(W_gate h) * (W_up h))``; gate and up are one product."""

    def __init__(self, hidden: int, spec: Dict[str, Any], init_std: float = 0.02, own_output: bool = True):
        super().__init__()
        mk = lambda *s: nn.Parameter(torch.empty(*s).normal_(std=init_std), requires_grad=False)
        self.out_width = spec["ff"]
        self.gate_up = mk(2 * spec["ff"], hidden)
        self.down = mk(hidden, spec["ff"]) if own_output else None

    def activate(self, h: torch.Tensor, out: torch.Tensor) -> None:
        L.swiglu(L.project(h, self.gate_up), out)

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        out = torch.empty(h.shape[0], self.out_width, dtype=h.dtype, device=h.device)
        self.activate(h, out)
        return L.project(out, self.down)

    def checkpoint_slices(self) -> Dict[str, torch.Tensor]:
        out = {"gate": self.gate_up[:self.out_width], "up": self.gate_up[self.out_width:]}
        if self.down is not None:
            out["down"] = self.down
        return out


MIXERS: Dict[str, Callable[..., nn.Module]] = {"latent_attention": YvWindowedLatentAttention,
                                               "grouped_attention": YvGroupedAttention}
FEED_FORWARDS: Dict[str, Callable[..., nn.Module]] = {"dense_gelu": YvDenseGELU, "dense_swiglu": YvDenseSwiGLU}


class YvTokenSide(nn.Module):
    """Per-layer token input: ``P (gelu_tanh(G x) * e)`` with e this layer's slice of the token's side embedding."""

    def __init__(self, hidden: int, dim: int, layer_idx: int, init_std: float = 0.02):
        super().__init__()
        mk = lambda *s: nn.Parameter(torch.empty(*s).normal_(std=init_std), requires_grad=False)
        self.gate, self.proj, self.offset = mk(dim, hidden), mk(hidden, dim), layer_idx * dim

    def forward(self, x: torch.Tensor, tokens: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
        return L.project(L.token_gate(L.project(x, self.gate), table, self.offset, tokens), self.proj)


class YvJoin:
    """What happens to the stream between a layer run's branches and the norms of the next one (or the final norm): the
    branches' sum, and in front of a pass of the loop the start of the stream and the pass's vector, are added."""

    def __init__(self, cfg: YvConfig, norms: List[torch.Tensor], table: Optional[torch.Tensor] = None,
                 vec: Optional[torch.Tensor] = None):
        self.norms, self.table, self.vec = norms, table, vec
        self.eps, self.offset, self.scale = cfg.layer_norm_eps, cfg.norm_offset, cfg.embedding_scale

    @property
    def plain(self) -> bool:
        """Only one norm, nothing to add: the sandwich block's own kernel covers it."""
        return self.table is None and self.vec is None and self.offset == 0.0 and len(self.norms) == 1

    def __call__(self, x: torch.Tensor, parts: Optional[torch.Tensor], tokens: torch.Tensor, dtype: torch.dtype,
                 start: bool = False) -> Tuple[torch.Tensor, ...]:
        return L.stream_add(x, parts, self.norms, self.offset, self.eps, dtype, table=self.table, rows=tokens,
                            table_scale=self.scale, vec=self.vec, start=start)


class YvLayeredBlock(nn.Module):
    """Norms before and after every branch; ``forward`` takes the stream and the already normed mixer input and returns
    the next run's."""

    def __init__(self, cfg: YvConfig, layer_idx: int, rotary: Optional[nn.Module]):
        super().__init__()
        spec, C, std = cfg.layer_specs[layer_idx], cfg.hidden_size, cfg.initializer_range
        if cfg.norm_offset:
            raise ValueError("sandwich blocks store their norm weights as they are")
        self.layer_idx, self.eps = layer_idx, cfg.layer_norm_eps
        norm = lambda: nn.Parameter(torch.ones(C), requires_grad=False)
        self.norm1, self.norm1b = norm(), norm()
        self.mixer = MIXERS[spec["mixer"]["kind"]](C, spec["mixer"], layer_idx, self.eps, rotary, std)
        self.ff = self.side = None
        if spec["mlp"]:
            self.norm2, self.norm2b = norm(), norm()
            self.ff = FEED_FORWARDS[spec["mlp"]["kind"]](C, spec["mlp"], std)
        if cfg.token_side_dim:
            self.side = YvTokenSide(C, cfg.token_side_dim, layer_idx, std)
            self.side_norm = norm()

    def entry_norms(self) -> List[torch.Tensor]:
        return [self.norm1]

    def forward(self, x: torch.Tensor, hs: Tuple[torch.Tensor, ...], ctx: AttnContext, run: int, tokens: torch.Tensor,
                side_table: Optional[torch.Tensor], join: YvJoin,
                tap: Optional[Callable[[torch.Tensor], None]] = None) -> Tuple[torch.Tensor, ...]:
        h, dt = hs[0], hs[0].dtype
        y, w = self.mixer(h, ctx, run), self.norm1b
        if self.ff is not None:
            h = L.stream_norm(x, y, w, self.norm2, self.eps, dt)
            y, w = self.ff(h), self.norm2b
        if self.side is not None:
            h = L.stream_norm(x, y, w, None, self.eps, dt)           # the token gate reads the stream itself
            y, w = self.side(h, tokens, side_table), self.side_norm
        if join.plain:
            hs = (L.stream_norm(x, y, w, join.norms[0], self.eps, dt),)
            if tap is not None:
                tap(x)
            return hs
        L.stream_norm(x, y, w, None, self.eps, dt, want_h=False)
        if tap is not None:
            tap(x)
        return join(x, None, tokens, dt)

    def checkpoint_slices(self) -> Dict[str, torch.Tensor]:
        out = {"norm1": self.norm1, "norm1b": self.norm1b}
        out.update({"mix." + k: v for k, v in self.mixer.checkpoint_slices().items()})
        if self.ff is not None:
            out.update({"norm2": self.norm2, "norm2b": self.norm2b})
            out.update({"mlp." + k: v for k, v in self.ff.checkpoint_slices().items()})
        if self.side is not None:
            out.update({"side.gate": self.side.gate, "side.proj": self.side.proj, "side.norm": self.side_norm})
        return out


class YvParallelBlock(nn.Module):
    """Mixer and feed-forward of the same stream, each behind its own norm.  Their output weights lie side by side in
    ``out_proj`` and their results in one buffer, so that one product forms the sum."""

    def __init__(self, cfg: YvConfig, layer_idx: int, rotary: Optional[nn.Module]):
        super().__init__()
        spec, C, std = cfg.layer_specs[layer_idx], cfg.hidden_size, cfg.initializer_range
        if cfg.token_side_dim:
            raise ValueError("parallel blocks take no per-layer token input")
        self.layer_idx, self.eps = layer_idx, cfg.layer_norm_eps
        norm = lambda: nn.Parameter(torch.full((C,), 1.0 - cfg.norm_offset), requires_grad=False)
        self.norm1 = norm()
        self.mixer = MIXERS[spec["mixer"]["kind"]](C, spec["mixer"], layer_idx, self.eps, rotary, std, own_output=False)
        self.ff = self.norm2 = None
        a = self.mixer.out_width
        self.ff_col = width = -(-a // 8) * 8
        if spec["mlp"]:
            self.norm2 = norm()
            self.ff = FEED_FORWARDS[spec["mlp"]["kind"]](C, spec["mlp"], std, own_output=False)
            width += -(-self.ff.out_width // 8) * 8
        f = self.ff.out_width if self.ff is not None else 0
        self.filled = a == self.ff_col and self.ff_col + f == width          # no padding columns
        self.out_proj = nn.Parameter(torch.empty(C, width).normal_(std=std), requires_grad=False)
        self.out_proj.data[:, a:self.ff_col].zero_()
        self.out_proj.data[:, self.ff_col + f:].zero_()

    def entry_norms(self) -> List[torch.Tensor]:
        return [self.norm1] if self.ff is None else [self.norm1, self.norm2]

    def forward(self, x: torch.Tensor, hs: Tuple[torch.Tensor, ...], ctx: AttnContext, run: int, tokens: torch.Tensor,
                side_table: Optional[torch.Tensor], join: YvJoin,
                tap: Optional[Callable[[torch.Tensor], None]] = None) -> Tuple[torch.Tensor, ...]:
        h, a = hs[0], self.mixer.out_width
        make = torch.empty if self.filled else torch.zeros
        z = make(h.shape[0], self.out_proj.shape[1], dtype=h.dtype, device=h.device)
        self.mixer.attend(h, ctx, run, z[:, :a])
        if self.ff is not None:
            self.ff.activate(hs[1], z[:, self.ff_col:self.ff_col + self.ff.out_width])
        parts = L.project_onto(x, z, self.out_proj)
        if tap is not None:
            if parts is not None:
                L.stream_add(x, parts, (), 0.0, self.eps, h.dtype)
                parts = None
            tap(x)
        return join(x, parts, tokens, h.dtype)

    def checkpoint_slices(self) -> Dict[str, torch.Tensor]:
        out = {"norm1": self.norm1, "mix.o": self.out_proj[:, :self.mixer.out_width]}
        out.update({"mix." + k: v for k, v in self.mixer.checkpoint_slices().items()})
        if self.ff is not None:
            out.update({"norm2": self.norm2, "mlp.down": self.out_proj[:, self.ff_col:self.ff_col + self.ff.out_width]})
            out.update({"mlp." + k: v for k, v in self.ff.checkpoint_slices().items()})
        return out


BLOCKS: Dict[str, Callable[..., nn.Module]] = {"sandwich": YvLayeredBlock, "parallel": YvParallelBlock}


class YvLayeredModel(YvPackedTrunk):
    def __init__(self, cfg: YvConfig, parallel=None):
        super().__init__()
        if parallel is not None and getattr(parallel, "world_size", 1) > 1:
            raise ValueError("layered models run on one GPU per replica")
        self.cfg, self.parallel, self.rotary = cfg, None, None
        self.layer_lo, self.layer_hi = 0, cfg.n_layer
        self.is_first_stage = self.is_last_stage = True
        C = cfg.hidden_size
        self.embed = nn.Embedding(cfg.vocab_size, C)
        nn.init.normal_(self.embed.weight, std=cfg.initializer_range)
        self.embed.weight.requires_grad_(False)
        self.embed_norm = nn.Parameter(torch.ones(C), requires_grad=False) if cfg.embedding_norm else None
        self.final_norm = nn.Parameter(torch.full((C,), 1.0 - cfg.norm_offset), requires_grad=False)
        self.side_embed = None
        if cfg.token_side_dim:
            self.side_embed = nn.Parameter(torch.empty(cfg.vocab_size, cfg.n_layer * cfg.token_side_dim).normal_(
                std=cfg.initializer_range), requires_grad=False)
        self.loop_step = None
        if cfg.layer_loop:
            if cfg.embedding_norm:
                raise ValueError("a loop adds the scaled embedding again: models with an embedding norm have none")
            self.loop_step = nn.Parameter(torch.empty(cfg.layer_loop["times"], C).normal_(std=cfg.initializer_range),
                                          requires_grad=False)
        rotaries: Dict[str, nn.Module] = {}                          # layers with the same rotation share its tables
        layers: List[nn.Module] = []
        for i in range(cfg.n_layer):
            rot = cfg.layer_specs[i]["mixer"]["rotation"]
            key = repr(sorted(rot.items())) if rot else ""
            if rot and key not in rotaries:
                rotaries[key] = rotary_for(rot)
            layers.append(BLOCKS[cfg.layer_block](cfg, i, rotaries.get(key)))
        self.layers = nn.ModuleList(layers)
        self.runs = cfg.layer_runs()
        self.subconscious = self.block_field = self.vision_encoder = self.modal_fusion = None
        self.materialized_components: List[str] = []
        # called with the number of the run and the stream after every layer run
        self.layer_tap: Optional[Callable[[int, torch.Tensor], None]] = None

    def join_before(self, run: int) -> YvJoin:
        """The step that prepares the stream for a run (one past the last: for the head)."""
        if run == len(self.runs):
            return YvJoin(self.cfg, [self.final_norm])
        layer, number, first = self.runs[run]
        opening = run == 0 and self.embed_norm is None
        return YvJoin(self.cfg, self.layers[layer].entry_norms(),
                      self.embed.weight if opening or (first and number > 0) else None,
                      self.loop_step[number] if first else None)

    def forward(self, input_ids: torch.Tensor, ctx: Optional[AttnContext] = None) -> YvModelOutput:
        B, S = input_ids.shape
        dev, dt = input_ids.device, self.final_norm.dtype
        if ctx is None:
            ctx = self.build_context(B, S, dev)
        tokens = input_ids.reshape(-1).long()
        x = torch.empty(B * S, self.cfg.hidden_size, dtype=torch.float32, device=dev)
        join = self.join_before(0)
        if self.embed_norm is not None:
            hs = (L.stream_norm(x, self.embed.weight, self.embed_norm, join.norms[0], self.cfg.layer_norm_eps, dt,
                                rows=tokens, start=True),)
        else:
            hs = join(x, None, tokens, dt, start=True)
        for run, (layer, _, _) in enumerate(self.runs):
            tap = None if self.layer_tap is None else lambda s, r=run: self.layer_tap(r, s)
            hs = self.layers[layer](x, hs, ctx, run, tokens, self.side_embed, self.join_before(run + 1), tap)
        return YvModelOutput(hidden_states=hs[0].view(B, S, -1), aux_loss=None)


class YvLayeredForCausalLM(YvModelForCausalLM):
    trunk_class = YvLayeredModel
    supports_portions = True          # a prompt may be continued from the cache at any position

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """hidden [..., H] -> fp32 logits [..., V]."""
        return L.project(hidden.reshape(-1, hidden.shape[-1]), self.head_weight, out_fp32=True).view(
            *hidden.shape[:-1], -1)

    @torch.no_grad()
    def forward(self, input_ids: Optional[torch.Tensor] = None, labels: Optional[torch.Tensor] = None,
                ctx: Optional[AttnContext] = None, return_logits: Optional[bool] = None, return_hidden: bool = False,
                **unused: Any) -> YvModelOutput:
        given = [k for k, v in unused.items() if v is not None]
        if labels is not None or given:
            raise NotImplementedError(f"layered models serve token ids; not supported: {given or ['labels']}")
        hidden = self.model(input_ids, ctx)["hidden_states"]
        res = YvModelOutput(aux_loss=None, loss=None, lm_loss=None, mtp_loss=None, logits=None)
        if return_hidden:
            res["hidden_states"] = hidden
        if return_logits or return_logits is None:
            res["logits"] = self.logits(hidden)
        return res

    # ---- checkpoint names --------------------------------------------------------------------------------------------
    def checkpoint_slices(self) -> Dict[str, torch.Tensor]:
        """Checkpoint tensor name -> view of the parameter that holds it."""
        m = self.model
        out = {"embed": m.embed.weight, "final.norm": m.final_norm, "head": self.lm_head}
        if m.embed_norm is not None:
            out["embed.norm"] = m.embed_norm
        if m.loop_step is not None:
            out["loop.step"] = m.loop_step
        if m.side_embed is not None:
            out["side.embed"] = m.side_embed
        for blk in m.layers:
            out.update({f"l{blk.layer_idx}.{k}": v for k, v in blk.checkpoint_slices().items()})
        return out

    def to_reference_state_dict(self) -> Dict[str, torch.Tensor]:
        return {k: v.detach().clone() for k, v in self.checkpoint_slices().items()}

    @torch.no_grad()
    def load_reference_state_dict(self, sd: Dict[str, torch.Tensor], strict: bool = True) -> List[str]:
        """Load a checkpoint by tensor name; returns the names that were not consumed."""
        slots = self.checkpoint_slices()
        missing = [k for k in slots if k not in sd]
        if missing and strict:
            raise KeyError(f"checkpoint lacks {len(missing)} tensors, e.g. {missing[:4]}")
        for k, dst in slots.items():
            if k in sd:
                if tuple(sd[k].shape) != tuple(dst.shape):
                    raise ValueError(f"{k}: checkpoint has {tuple(sd[k].shape)}, the configuration asks for {tuple(dst.shape)}")
                dst.copy_(sd[k])
        for blk in self.model.layers:
            getattr(blk.mixer, "weights_changed", lambda: None)()
        return [k for k in sd if k not in slots]
