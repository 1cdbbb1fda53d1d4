from .gpt import GPT, GPTConfig
from .llama import Llama, LlamaConfig
from .registry import architecture, load_config
from .resnet import ResNet50, Bottleneck
from .zidalix import ZidalixConfig
