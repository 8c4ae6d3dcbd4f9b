from .channel_delta import DSChannelDeltaRule
from .matrix_memory import DSMatrixMemory
from .min_gru import DSMinGRU
from .state_space import DSStateSpace
from .tied_gate_linear import DSTiedGateLinearAttention
