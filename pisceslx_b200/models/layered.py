"""Layered models: the trunk is a list of layer specs (``YvConfig.layer_specs``), each naming a mixer and a
feed-forward from the tables below, around an fp32 residual stream.

    x = rms(embed[token]) * w_e
    per layer:  x += rms(mixer(rms(x) * w1)) * w1b
                x += rms(ff(rms(x) * w2)) * w2b                          (layers with a feed-forward)
                x += rms(P (gelu_tanh(G x) * e_layer[token])) * w_s       (models with a per-layer token input)
    logits = head (rms(x) * w_f)

Every ``x +=`` and the norm in front of the next branch are one kernel (``ops.latent.stream_norm``): the stream is
read and written once per branch.  The classes keep the contracts that generation, the engine, the captured decode
step and the loader rely on, so a layered model is served by the same code as the Yv trunk.  They are serving models:
no backward."""
from __future__ import annotations

from typing import Any, Callable, Dict, List, Optional

import torch
import torch.nn as nn

from ..config import YvConfig
from ..ops import latent as L
from .attention import AttnContext
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


MIXERS: Dict[str, Callable[..., nn.Module]] = {"latent_attention": YvWindowedLatentAttention}
FEED_FORWARDS: Dict[str, Callable[..., nn.Module]] = {"dense_gelu": YvDenseGELU}


class YvTokenSide(nn.Module):
    """Per-layer token input: ``P (gelu_tanh(G x) * e)`` with e this layer's slice of the token's side embedding."""

    def __init__(self, hidden: int, dim: int, layer_idx: int, init_std: float = 0.02):
        super().__init__()
        mk = lambda *s: nn.Parameter(torch.empty(*s).normal_(std=init_std), requires_grad=False)
        self.gate, self.proj, self.offset = mk(dim, hidden), mk(hidden, dim), layer_idx * dim

    def forward(self, x: torch.Tensor, tokens: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
        return L.project(L.token_gate(L.project(x, self.gate), table, self.offset, tokens), self.proj)


class YvLayeredBlock(nn.Module):
    """One layer; ``forward`` takes the stream and the already normed mixer input and returns the next layer's."""

    def __init__(self, cfg: YvConfig, layer_idx: int, rotary: nn.Module):
        super().__init__()
        spec, C, std = cfg.layer_specs[layer_idx], cfg.hidden_size, cfg.initializer_range
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

    def forward(self, x: torch.Tensor, h: torch.Tensor, ctx: AttnContext, tokens: torch.Tensor,
                side_table: Optional[torch.Tensor], next_norm: torch.Tensor) -> torch.Tensor:
        y, w, dt = self.mixer(h, ctx), self.norm1b, h.dtype
        if self.ff is not None:
            h = L.stream_norm(x, y, w, self.norm2, self.eps, dt)
            y, w = self.ff(h), self.norm2b
        if self.side is not None:
            h = L.stream_norm(x, y, w, None, self.eps, dt)           # the token gate reads the stream itself
            y, w = self.side(h, tokens, side_table), self.side_norm
        return L.stream_norm(x, y, w, next_norm, self.eps, dt)

    def checkpoint_slices(self) -> Dict[str, torch.Tensor]:
        out = {"norm1": self.norm1, "norm1b": self.norm1b}
        out.update({"mix." + k: v for k, v in self.mixer.checkpoint_slices().items()})
        if self.ff is not None:
            out.update({"norm2": self.norm2, "norm2b": self.norm2b})
            out.update({"mlp." + k: v for k, v in self.ff.checkpoint_slices().items()})
        if self.side is not None:
            out.update({"side.gate": self.side.gate, "side.proj": self.side.proj, "side.norm": self.side_norm})
        return out


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
        self.embed_norm = nn.Parameter(torch.ones(C), requires_grad=False)
        self.final_norm = nn.Parameter(torch.ones(C), requires_grad=False)
        self.side_embed = None
        if cfg.token_side_dim:
            self.side_embed = nn.Parameter(torch.empty(cfg.vocab_size, cfg.n_layer * cfg.token_side_dim).normal_(
                std=cfg.initializer_range), requires_grad=False)
        rotaries: Dict[str, nn.Module] = {}                          # layers with the same rotation share its tables
        layers: List[nn.Module] = []
        for i in range(cfg.n_layer):
            rot = cfg.layer_specs[i]["mixer"]["rotation"]
            key = repr(sorted(rot.items()))
            if key not in rotaries:
                rotaries[key] = rotary_for(rot)
            layers.append(YvLayeredBlock(cfg, i, rotaries[key]))
        self.layers = nn.ModuleList(layers)
        self.subconscious = self.block_field = self.vision_encoder = self.modal_fusion = None
        self.materialized_components: List[str] = []
        self.layer_tap: Optional[Callable[[int, torch.Tensor], None]] = None   # called with the stream after every layer

    def forward(self, input_ids: torch.Tensor, ctx: Optional[AttnContext] = None) -> YvModelOutput:
        B, S = input_ids.shape
        dev, dt = input_ids.device, self.embed_norm.dtype
        if ctx is None:
            ctx = self.build_context(B, S, dev)
        tokens = input_ids.reshape(-1).long()
        x = torch.empty(B * S, self.cfg.hidden_size, dtype=torch.float32, device=dev)
        norms = [blk.norm1 for blk in self.layers[1:]] + [self.final_norm]
        h = L.stream_norm(x, self.embed.weight, self.embed_norm, self.layers[0].norm1, self.cfg.layer_norm_eps, dt,
                          rows=tokens, start=True)
        for blk, nxt in zip(self.layers, norms):
            h = blk(x, h, ctx, tokens, self.side_embed, nxt)
            if self.layer_tap is not None:
                self.layer_tap(blk.layer_idx, x)
        return YvModelOutput(hidden_states=h.view(B, S, -1), aux_loss=None)


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
        out = {"embed": m.embed.weight, "embed.norm": m.embed_norm, "final.norm": m.final_norm, "head": self.lm_head}
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
