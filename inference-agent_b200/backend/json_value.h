// A small JSON reader for model configurations, safetensors headers and replayed traces (recursive descent, UTF-8 passed
// through, \uXXXX escapes of the basic plane decoded). Errors are std::runtime_error with the byte offset.
#pragma once

#include <cstdint>
#include <cstdlib>
#include <map>
#include <memory>
#include <stdexcept>
#include <string>
#include <utility>
#include <vector>

class Json {
public:
    enum class Kind { Null, Bool, Number, String, Array, Object };

    static Json parse(const std::string& text) {
        Parser p{text, 0};
        Json v = p.value(0);
        p.space();
        if (p.at != text.size()) p.fail("trailing characters");
        return v;
    }

    Kind kind() const { return kind_; }
    bool is_null() const { return kind_ == Kind::Null; }
    bool is_object() const { return kind_ == Kind::Object; }
    bool has(const std::string& key) const { return kind_ == Kind::Object && members_.count(key) > 0; }
    // Member of an object; throws with `key` in the text if it is missing.
    const Json& at(const std::string& key) const {
        if (kind_ != Kind::Object) throw std::runtime_error("json: not an object while looking for \"" + key + "\"");
        auto it = members_.find(key);
        if (it == members_.end()) throw std::runtime_error("json: key \"" + key + "\" is missing");
        return it->second;
    }
    const std::map<std::string, Json>& members() const { need(Kind::Object, "an object"); return members_; }
    const std::vector<Json>& items() const { need(Kind::Array, "an array"); return items_; }
    double number() const { need(Kind::Number, "a number"); return number_; }
    int64_t integer() const {
        need(Kind::Number, "a number");
        const int64_t v = static_cast<int64_t>(number_);
        if (double(v) != number_) throw std::runtime_error("json: not an integer");
        return v;
    }
    bool boolean() const { need(Kind::Bool, "a boolean"); return number_ != 0; }
    const std::string& str() const { need(Kind::String, "a string"); return string_; }

private:
    void need(Kind k, const char* what) const {
        if (kind_ != k) throw std::runtime_error(std::string("json: expected ") + what);
    }
    struct Parser {
        const std::string& s;
        size_t at;
        [[noreturn]] void fail(const char* why) const { throw std::runtime_error("json: " + std::string(why) + " at byte " + std::to_string(at)); }
        void space() {
            while (at < s.size() && (s[at] == ' ' || s[at] == '\t' || s[at] == '\n' || s[at] == '\r')) at++;
        }
        bool eat(char c) {
            space();
            if (at < s.size() && s[at] == c) { at++; return true; }
            return false;
        }
        void expect(char c) {
            if (!eat(c)) fail("unexpected character");
        }
        void word(const char* w) {
            for (; *w; w++, at++)
                if (at >= s.size() || s[at] != *w) fail("bad literal");
        }
        Json value(int depth) {
            if (depth > 64) fail("nested too deeply");
            space();
            if (at >= s.size()) fail("unexpected end");
            Json v;
            switch (s[at]) {
                case '{':
                    at++;
                    v.kind_ = Kind::Object;
                    if (eat('}')) return v;
                    do {
                        space();
                        std::string key = string();
                        expect(':');
                        v.members_[std::move(key)] = value(depth + 1);
                    } while (eat(','));
                    expect('}');
                    return v;
                case '[':
                    at++;
                    v.kind_ = Kind::Array;
                    if (eat(']')) return v;
                    do v.items_.push_back(value(depth + 1));
                    while (eat(','));
                    expect(']');
                    return v;
                case '"': v.kind_ = Kind::String; v.string_ = string(); return v;
                case 't': word("true"); v.kind_ = Kind::Bool; v.number_ = 1; return v;
                case 'f': word("false"); v.kind_ = Kind::Bool; return v;
                case 'n': word("null"); return v;
                default: {
                    const char* begin = s.c_str() + at;
                    char* end = nullptr;
                    v.number_ = std::strtod(begin, &end);
                    if (end == begin) fail("unexpected character");
                    at += size_t(end - begin);
                    v.kind_ = Kind::Number;
                    return v;
                }
            }
        }
        std::string string() {
            if (at >= s.size() || s[at] != '"') fail("expected a string");
            at++;
            std::string out;
            while (at < s.size() && s[at] != '"') {
                char c = s[at++];
                if (c != '\\') { out.push_back(c); continue; }
                if (at >= s.size()) fail("unterminated escape");
                c = s[at++];
                switch (c) {
                    case 'b': out.push_back('\b'); break;
                    case 'f': out.push_back('\f'); break;
                    case 'n': out.push_back('\n'); break;
                    case 'r': out.push_back('\r'); break;
                    case 't': out.push_back('\t'); break;
                    case 'u': {
                        if (at + 4 > s.size()) fail("short \\u escape");
                        const unsigned u = unsigned(std::strtoul(s.substr(at, 4).c_str(), nullptr, 16));
                        at += 4;
                        if (u < 0x80) out.push_back(char(u));
                        else if (u < 0x800) { out.push_back(char(0xC0 | (u >> 6))); out.push_back(char(0x80 | (u & 63))); }
                        else { out.push_back(char(0xE0 | (u >> 12))); out.push_back(char(0x80 | ((u >> 6) & 63))); out.push_back(char(0x80 | (u & 63))); }
                        break;
                    }
                    default: out.push_back(c);
                }
            }
            if (at >= s.size()) fail("unterminated string");
            at++;
            return out;
        }
    };

    Kind kind_ = Kind::Null;
    double number_ = 0;
    std::string string_;
    std::vector<Json> items_;
    std::map<std::string, Json> members_;
};
