"""What decoders made of mixers and feed-forwards of several kinds have in common: embedding, head, checkpoint tensors,
caches, positions, and the rows whose logits are wanted. A design brings its layers and the walk over them (`hidden`)."""
from __future__ import annotations

import torch
import torch.nn as nn

from . import _lib
from .generation import GenerationMixin, InferenceParams
from .gpt import CausalLMOutput, _randn_big, _stable_hash
from .mixers import Linear, _empty


class HybridDecoder(nn.Module, GenerationMixin):
    """Same calls as the other models: forward(input_ids, position_ids, inference_params).logits, generate(...).

    `config` has vocab_size and hidden_size. Subclasses fill self.layers (each with `mixer` and `checkpoint_slots`) and
    self.runs (layer number of every layer run; each run has a cache of its own), and define `hidden` and, for tensors
    that are not N(0, std) at random initialisation, `init_constant`."""

    selects_logit_rows = True  # forward(logit_rows=...) computes logits at those tokens only
    takes_portions = True      # a prompt may arrive in portions of any size
    load_kernels = staticmethod(_lib.load_hybrid)  # the library that has the design's kernels

    def __init__(self, config, device=None, dtype=torch.bfloat16):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"this model runs in bfloat16 or float32, not {dtype}")
        self.config, self.dtype = config, dtype
        f = {"device": device, "dtype": dtype}
        self.embed = _empty(config.vocab_size, config.hidden_size, **f)
        self.layers = nn.ModuleList()
        self.final_norm = _empty(config.hidden_size, device=device, dtype=torch.float32)
        self.lm_head = Linear(config.hidden_size, config.vocab_size, **f)
        self.runs: list = []
        # bf16 products accumulate in fp32 to the end, fp32 products are true fp32
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        if dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False

    # ---- weights ------------------------------------------------------------------------------------------
    def checkpoint_slots(self) -> dict:
        """Checkpoint tensor name -> the parameter (or slice of a fused one) that holds it."""
        out = {"embed": self.embed, "final.norm": self.final_norm, "head": self.lm_head.weight}
        for i, layer in enumerate(self.layers):
            out.update({f"l{i}.{k}": v for k, v in layer.checkpoint_slots().items()})
        return out

    def _zero_padding(self):
        for layer in self.layers:
            if hasattr(layer.mixer, "zero_padding"):
                layer.mixer.zero_padding()

    @torch.no_grad()
    def load_tensors(self, tensors: dict):
        """Fills the model from checkpoint tensors; a missing, unknown or misshapen one is an error."""
        slots = self.checkpoint_slots()
        missing, unknown = sorted(set(slots) - set(tensors)), sorted(set(tensors) - set(slots))
        if missing or unknown:
            raise ValueError(f"checkpoint does not fit the configuration: missing {missing}, unknown {unknown}")
        for name, dst in slots.items():
            src = tensors[name]
            if tuple(src.shape) != tuple(dst.shape):
                raise ValueError(f"{name}: shape {tuple(src.shape)}, expected {tuple(dst.shape)}")
            dst.copy_(src)
        self._zero_padding()
        return self

    def init_constant(self, name: str):
        """Value of a tensor that random initialisation leaves constant, None for the others."""
        return None

    @torch.no_grad()
    def init_random(self, seed: int = 0, std: float = 0.02):
        """Random weights from seeds derived from tensor names: N(0, std), and the constants of `init_constant`."""
        gen = torch.Generator(device=self.embed.device)
        for name, dst in self.checkpoint_slots().items():
            value = self.init_constant(name)
            if value is not None:
                dst.copy_(torch.as_tensor(value, dtype=dst.dtype, device=dst.device).expand_as(dst))
            else:
                gen.manual_seed((seed * 1000003 + _stable_hash(name)) % (2 ** 63))
                dst.copy_(_randn_big(tuple(dst.shape), gen, dst.device, std, dst.dtype))
        self._zero_padding()
        return self

    # ---- caches -------------------------------------------------------------------------------------------
    def allocate_cache(self, batch_size: int, max_seqlen: int, device) -> dict:
        """Per layer run: the window's rings or the recurrent state. Nothing needs clearing between requests: a sequence
        that starts at position 0 reads neither."""
        if torch.device(device).type == "cuda":
            self.load_kernels()
        return {r: self.layers[i].mixer.new_cache(batch_size, max_seqlen, device, self.dtype)
                for r, i in enumerate(self.runs)}

    def reset_decode_state(self, prompt_len: int, device, max_seqlen: int, batch: int = 1):
        """All decode state is in the caches and in the positions."""

    # ---- forward ------------------------------------------------------------------------------------------
    def hidden(self, ids, caches, pos, n: int, past: int, rows, collect):
        """Final-normed activations (R, width) of the rows asked for (None: all, an empty tensor: none are computed)."""
        raise NotImplementedError

    def head(self, h, decode: bool):
        return self.lm_head.rows(h, decode, torch.float32)

    def forward(self, input_ids, position_ids=None, inference_params=None, logit_rows=None, collect=None):
        """input_ids (B, n): the next n tokens of every sequence; the caches of `inference_params` hold what came
        before. position_ids (B, n) or (B, 1): only the first column is read; without it the position is the caches'
        offset, and for n > 1 no sequence is further than that. logit_rows: places among the n tokens whose logits are
        wanted (default all). collect: a list that receives the residual after every layer run (for inspection).
        -> logits (B, len(logit_rows), vocab) fp32."""
        B, n = input_ids.shape
        dev = input_ids.device
        if inference_params is None:
            inference_params = InferenceParams(max_sequence_len=n, max_batch_size=B,
                                               key_value_memory_dict=self.allocate_cache(B, n, dev))
        past = inference_params.sequence_len_offset
        if position_ids is None:
            pos = torch.full((B,), past, dtype=torch.int64, device=dev)
        else:
            pos = position_ids[:, 0].contiguous()
        if logit_rows is None or list(logit_rows) == list(range(n)):
            rows, R = None, n
        else:
            R = len(logit_rows)
            rows = torch.tensor([b * n + t for b in range(B) for t in logit_rows], dtype=torch.int32, device=dev)
        h = self.hidden(input_ids.reshape(-1).contiguous(), inference_params.key_value_memory_dict, pos, n, past, rows,
                        collect)
        if R == 0:
            return CausalLMOutput(logits=torch.empty(B, 0, self.config.vocab_size, device=dev))
        return CausalLMOutput(logits=self.head(h, n == 1).view(B, R, self.config.vocab_size))
